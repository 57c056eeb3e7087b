"""Attention whose weights are sigmoids: every visible key counts by its own score, nothing is normalised over keys."""
from __future__ import annotations

from typing import List, Mapping

import torch

from ..config.spec import PartSpec
from ..csrc import ops
from ..weights.loader import TensorNeed
from .attention import run_attention_ex
from .base import MIXERS, CacheNeed
from .side_by_side import ProjectedMixer


class SigmoidAttention(ProjectedMixer):
    """q = W_q h, k = W_k h, v = W_v h; q head h reads kv head h // (q_heads // kv_heads).  Each query and key head is divided by
    its root mean square (`qk_norm_eps`) and multiplied by a weight of head_dim values shared by all heads, then rotated by
    the model's position encoding (`position`, pairs i and i + rotary_dim / 2).  The weight of key j for query i is
    sigmoid(q_i . k_j * scale + b_h), b a number per q head, where j <= i and, with `chunk` = c, floor(j / c) = floor(i / c)
    (chunks are counted from the sequence's first position); or, with `window`, i - j < window.  The heads' sums of weighted
    values are projected by W_o.  Scores, weights, norms and angles are float32.

    Parameters: hidden_size, q_heads, kv_heads, head_dim, v_dim, scale, chunk, window, qk_norm_eps (None: no norms), position,
    names.{q, k, v, o, q_norm, k_norm, score_bias}."""

    def __init__(self, spec, env):
        super().__init__(spec, env)
        g = spec.get
        self.q_heads = int(spec["q_heads"])
        self.kv_heads = int(spec["kv_heads"])
        self.head_dim = int(spec["head_dim"])
        self.v_dim = int(g("v_dim") or self.head_dim)
        if self.q_heads % self.kv_heads:
            raise ValueError("q heads are not a multiple of kv heads")
        self.scale = float(spec["scale"])
        self.chunk = int(g("chunk") or 0)
        self.window = int(g("window") or 0)
        self.eps = g("qk_norm_eps")
        pos = g("position")
        self.position = env.positions[pos] if pos is not None else None
        if self.position is not None and getattr(self.position, "layout", "half") != "half":
            raise ValueError("this attention rotates value i with value i + rotary_dim / 2; its position encoding has another layout")
        self.q_norm = self.k_norm = self.bias = None
        self.cols = [0, 0, 0]

    @property
    def out_dim(self) -> int:
        return self.q_heads * self.v_dim

    @staticmethod
    def cache_need(spec: PartSpec) -> CacheNeed:
        hd = int(spec["head_dim"])
        vd = int(spec.get("v_dim") or hd)
        return CacheNeed("kv", int(spec["kv_heads"]), hd, spec.get("window"), v_dim=None if vd == hd else vd)

    @staticmethod
    def tensor_needs(spec: PartSpec) -> List[TensorNeed]:
        h, hd, n = int(spec["hidden_size"]), int(spec["head_dim"]), spec["names"]
        vd, qh, kvh = int(spec.get("v_dim") or hd), int(spec["q_heads"]), int(spec["kv_heads"])
        needs = [TensorNeed(n["q"], (qh * hd, h)), TensorNeed(n["k"], (kvh * hd, h)), TensorNeed(n["v"], (kvh * vd, h)),
                 TensorNeed(n["score_bias"], (qh,), role="vector", init="linear"), TensorNeed(n["o"], (h, qh * vd))]
        if spec.get("qk_norm_eps") is not None:
            needs += [TensorNeed(n["q_norm"], (hd,), role="vector", init="norm"), TensorNeed(n["k_norm"], (hd,), role="vector", init="norm")]
        return needs

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        n = self.spec["names"]
        self.cols = self.take([tensors[n["q"]], tensors[n["k"]], tensors[n["v"]]], tensors[n["o"]])
        self.bias = tensors[n["score_bias"]]
        if self.eps is not None:
            self.q_norm, self.k_norm = tensors[n["q_norm"]], tensors[n["k_norm"]]

    def mix(self, ctx, entry, proj, col, act, act_col, scale, n_rows):
        view = ctx.cache.kv_view(entry)
        q = ctx.ws.buffer("sigattn.q", (ctx.ws.max_rows, self.q_heads * self.head_dim), self.env.dtype)
        freq, rot = self.position.rotary() if self.position is not None else (None, 0)
        table = self.position.cos_sin_table(self.env.max_positions) if rot and self.env.max_positions else None
        ops.head_norm_rope_kv_write(proj, col + self.cols[0], col + self.cols[1], col + self.cols[2], self.q_norm, self.k_norm,
                                    float(self.eps or 0.0), freq, table, rot, q, self.q_heads, view, ctx.row_slot, ctx.row_pos, n_rows)
        extra = ops.attn_extra(chunk=self.chunk, sig_bias=self.bias, out_ld=act.shape[-1], out_col=act_col, out_scale=scale)
        run_attention_ex(ctx, q, act, view, n_rows, self.q_heads, self.scale, self.window, extra)


MIXERS.register("sigmoid_attention", SigmoidAttention)
