"""The two ends of the model: token embedding and the output head."""
from __future__ import annotations

from typing import List, Mapping

import torch

from ..config.spec import PartSpec
from ..csrc import ops
from ..weights.loader import TensorNeed
from .base import EMBEDDINGS, HEADS, OPENERS, CacheNeed, Embedding, Head, Opener
from .linear import Linear
from .norm import PostNormed

EMBEDDING_OUTPUT = "embedding.output"      # the workspace buffer an embedding with `keep` leaves its rows in


class TokenEmbedding(Embedding):
    """resid[r] = float32(table[token[r]]); an id outside the table gives a zero row
    (x0ne-core/kernels/cuda/embedding.cu:5-17).  With `scale` the row is multiplied by it in float32
    on its way into the residual.  Parameters: vocab_size, hidden_size, scale (default 1), names.weight."""
    replayable = True

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.table = None
        self.scale = float(spec.get("scale", 1.0) or 1.0)

    @staticmethod
    def tensor_needs(spec: PartSpec) -> List[TensorNeed]:
        return [TensorNeed(spec["names"]["weight"], (int(spec["vocab_size"]), int(spec["hidden_size"])),
                           init="embedding")]

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        self.table = tensors[self.spec["names"]["weight"]]

    def forward(self, ctx, resid, n_rows):
        ops.embedding(self.table, ctx.tokens, resid, n_rows, self.scale)


class SumEmbedding(Embedding):
    """resid[r] = table[token] + pairs[(previous token * mul_prev + token * mul_cur) mod buckets] + positions[pos], added in
    float32 in this order.  `pairs` has one row more than `buckets`: the last one stands for a sequence's first token, which
    has no previous one.  A sequence keeps its last token.  Without `buckets` there is no pair term, without `positions` (the
    number of learned position rows) no position term.  `keep` leaves the rows in the workspace as well
    (`EMBEDDING_OUTPUT`), for parts further on that read the embedding output again.
    Parameters: vocab_size, hidden_size, buckets, mul_prev, mul_cur, positions, keep, names.{weight, pairs, positions}."""
    replayable = True
    TAG = "previous token"

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.hidden = int(spec["hidden_size"])
        self.buckets = int(spec.get("buckets") or 0)
        self.mul_prev, self.mul_cur = (int(spec["mul_prev"]), int(spec["mul_cur"])) if self.buckets else (0, 0)
        self.keep = bool(spec.get("keep"))
        self.table = self.pairs = self.positions = None

    @classmethod
    def cache_needs(cls, spec: PartSpec) -> List[CacheNeed]:
        return [CacheNeed("state", state_shape=(1,), tag=cls.TAG)] if spec.get("buckets") else []

    @staticmethod
    def tensor_needs(spec: PartSpec) -> List[TensorNeed]:
        h, n = int(spec["hidden_size"]), spec["names"]
        needs = [TensorNeed(n["weight"], (int(spec["vocab_size"]), h), init="embedding")]
        if spec.get("buckets"):
            needs.append(TensorNeed(n["pairs"], (int(spec["buckets"]) + 1, h), init="embedding"))
        if spec.get("positions"):
            needs.append(TensorNeed(n["positions"], (int(spec["positions"]), h), init="embedding"))
        return needs

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        n = self.spec["names"]
        self.table = tensors[n["weight"]]
        self.pairs = tensors[n["pairs"]] if self.buckets else None
        self.positions = tensors[n["positions"]] if self.spec.get("positions") else None

    def forward(self, ctx, resid, n_rows):
        copy = ctx.ws.buffer(EMBEDDING_OUTPUT, (ctx.ws.max_rows, self.hidden), torch.float32) if self.keep else None
        last = ctx.cache.model_state(self.TAG) if self.buckets else None
        ops.embed_sum(self.table, self.pairs, self.positions, ctx.tokens, resid, copy, last, self.mul_prev, self.mul_cur, ctx.row_slot,
                      ctx.row_pos, ctx.seq_first_row, ctx.n_seqs, n_rows)


class ConcatOpener(Opener):
    """The start of a pass over a repeated stretch of layers: the residual becomes W [x; x0], x being the residual with the
    pending result of the layer before and x0 the embedding output (`EMBEDDING_OUTPUT`, left there by the embedding).  The
    product's operand is built by one launch (which also norms and adds the pending result), its float32 result is the new
    residual.
    Parameters: hidden_size, names.weight ([hidden_size, 2 hidden_size])."""
    replayable = True

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.hidden = int(spec["hidden_size"])
        self.w = None

    @staticmethod
    def tensor_needs(spec: PartSpec) -> List[TensorNeed]:
        h = int(spec["hidden_size"])
        return [TensorNeed(spec["names"]["weight"], (h, 2 * h))]

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        self.w = Linear(tensors[self.spec["names"]["weight"]])

    def weight_bytes(self) -> int:
        return self.w.weight_bytes()

    def forward(self, ctx, resid, delta, n_rows):
        ws, h, dt = ctx.ws, self.hidden, self.env.dtype
        norm = bias = None
        if isinstance(delta, PostNormed):
            norm, bias, delta = delta.norm, delta.bias, delta.delta
        elif delta is not None and not isinstance(delta, torch.Tensor):
            raise ValueError("a concatenating opener takes the pending result of a layer as one tensor")
        if norm is not None and (norm.groups != 1 or norm.centred):
            raise ValueError("a concatenating opener takes a result that is still to be normed by one root mean square only")
        x0 = ws.buffer(EMBEDDING_OUTPUT, (ws.max_rows, h), torch.float32)
        cat = ws.buffer("opener.rows", (ws.max_rows, 2 * h), dt)
        ops.concat_rows(resid, delta, bias, None if norm is None else norm.weight, 0.0 if norm is None else norm.eps, x0, cat, n_rows)
        self.w(cat, resid, n_rows)
        return None


class PassOpener(Opener):
    """The start of a pass over a stretch of layers that a model repeats:
    resid = ((resid + pending delta) + scale * table[token]) + step[step_row], one float32 add after the other.  The
    embedding term is the model's embedding output over again (`add_embedding`; a first pass leaves it out); `step` is a
    [step_rows, hidden_size] tensor of which every pass has a row of its own.
    Parameters: hidden_size, vocab_size, scale, add_embedding, step_row, step_rows, names.{table, step}."""
    replayable = True

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.scale = float(spec.get("scale", 1.0) or 1.0)
        self.add_embedding = bool(spec.get("add_embedding"))
        self.row = int(spec["step_row"])
        if not 0 <= self.row < int(spec["step_rows"]):
            raise ValueError("a pass opener names a row of its step tensor that does not exist")
        self.table = self.step = None

    @staticmethod
    def tensor_needs(spec: PartSpec) -> List[TensorNeed]:
        h, n = int(spec["hidden_size"]), spec["names"]
        needs = [TensorNeed(n["step"], (int(spec["step_rows"]), h), role="vector", init="linear")]
        if spec.get("add_embedding"):
            needs.append(TensorNeed(n["table"], (int(spec["vocab_size"]), h), init="embedding"))
        return needs

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        n = self.spec["names"]
        self.step = tensors[n["step"]][self.row].contiguous()
        self.table = tensors[n["table"]] if self.add_embedding else None

    def forward(self, ctx, resid, delta, n_rows):
        if delta is not None and not isinstance(delta, torch.Tensor):
            raise ValueError("a pass opener takes the pending result of a layer as one tensor")
        ops.open_pass(resid, delta, self.table, ctx.tokens if self.add_embedding else None, self.scale, self.step, n_rows)
        return None


class LMHead(Head):
    """logits = normed W^T in float32 for the wanted rows only; W is the embedding table when the
    model is tied (x0ne-core/runtime/src/engine.rs:823-835).  With `softcap` they become softcap * tanh(logits / softcap).
    Parameters: vocab_size, hidden_size, tied, softcap (default: none), names.weight."""
    replayable = True

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.linear = None
        self.act = (ops.OUT_SOFT_CAP, float(spec["softcap"])) if spec.get("softcap") else None

    @staticmethod
    def tensor_needs(spec: PartSpec) -> List[TensorNeed]:
        return [TensorNeed(spec["names"]["weight"], (int(spec["vocab_size"]), int(spec["hidden_size"])),
                           init="embedding")]

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        self.linear = Linear(tensors[self.spec["names"]["weight"]])

    @staticmethod
    def optional_duplicates(spec: PartSpec):
        # a tied checkpoint may also store lm_head.weight, equal to the table (x0ne-core/runtime/src/weights.rs:154-159)
        return {"lm_head.weight": spec["names"]["weight"]} if spec.get("tied") else {}

    def weight_bytes(self) -> int:
        return self.linear.weight_bytes()

    def forward(self, normed, logits, n_rows):
        return self.linear(normed, logits, n_rows, act=self.act)


EMBEDDINGS.register("token_embedding", TokenEmbedding)
EMBEDDINGS.register("sum_embedding", SumEmbedding)
HEADS.register("lm_head", LMHead)
OPENERS.register("pass_opener", PassOpener)
OPENERS.register("concat_opener", ConcatOpener)
