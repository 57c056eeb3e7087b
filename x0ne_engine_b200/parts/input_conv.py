"""A short causal convolution on the rows a mixer reads."""
from __future__ import annotations

from typing import List, Mapping

import torch

from ..config.spec import PartSpec
from ..csrc import ops
from ..weights.loader import TensorNeed
from .base import INPUT_TRANSFORMS, CacheNeed, InputTransform
from .norm import PostNormed, RMSNorm


class CausalInputConv(InputTransform):
    """The mixer reads h + conv(h), h being the normed rows: conv(h)_t = sum_j w[:, j] h_(t - taps + 1 + j) per channel, zeros
    before the sequence's first token, no bias.  A sequence keeps its last taps - 1 inputs (float32).  Sums are float32; the
    result is rounded once.  Passes of one row per sequence do the residual add, the norm and the convolution in one launch
    (bfloat16 runs; a 32-bit run keeps the two launches of a prompt, so that a row's bits do not depend on the cut).
    Parameters: hidden_size, taps, names.weight ([hidden_size, taps])."""
    replayable = True
    TAG = "input conv"

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.hidden = int(spec["hidden_size"])
        self.taps = int(spec["taps"])
        if not 1 <= self.taps <= ops.INPUT_CONV_MAX_TAPS:
            raise ValueError(f"an input convolution of {self.taps} taps; 1 to {ops.INPUT_CONV_MAX_TAPS} are served")
        self.w = None

    @classmethod
    def cache_needs(cls, spec: PartSpec) -> List[CacheNeed]:
        kept = int(spec["taps"]) - 1
        return [CacheNeed("state", state_shape=(-(-kept * int(spec["hidden_size"]) // 4) * 4,), tag=cls.TAG)] if kept else []

    @staticmethod
    def tensor_needs(spec: PartSpec) -> List[TensorNeed]:
        return [TensorNeed(spec["names"]["weight"], (int(spec["hidden_size"]), int(spec["taps"])), role="vector", init="linear")]

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        self.w = tensors[self.spec["names"]["weight"]].to(torch.float32).t().contiguous()       # [taps, hidden]

    def forward(self, ctx, entry, norm, resid, delta, n_rows):
        ws, dt = ctx.ws, self.env.dtype
        out = ws.buffer("conv.out", (ws.max_rows, self.hidden), dt)
        state = ctx.cache.state(entry, self.TAG) if self.taps > 1 else None
        if ctx.decode and dt == torch.bfloat16 and self._fuses(norm, delta):
            pending = (delta.delta, delta.bias, delta.norm.weight, delta.norm.eps) if delta is not None else (None, None, None, 0.0)
            ops.norm_conv_step(resid, *pending, norm.weight, norm.eps, self.w, state, out, ctx.row_slot, n_rows)
            return out
        normed = ws.buffer("normed", (ws.max_rows, self.hidden), dt)
        norm.add_norm(ctx, resid, delta, normed, n_rows)
        ops.input_conv(normed, self.w, state, out, ctx.seq_first_row, ctx.seq_slot, ctx.n_seqs, ctx.max_seq_rows)
        return out

    def _fuses(self, norm, delta) -> bool:
        return type(norm) is RMSNorm and norm.groups == 1 and ops.norm_conv_step_takes(self.hidden) and \
            (delta is None or isinstance(delta, PostNormed) and delta.norm.groups == 1 and not delta.norm.centred)


INPUT_TRANSFORMS.register("causal_input_conv", CausalInputConv)
