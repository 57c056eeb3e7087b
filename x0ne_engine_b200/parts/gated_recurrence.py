"""Recurrent mixers with a matrix state per head that is decayed and written through gates."""
from __future__ import annotations

from typing import List, Mapping

import torch

from ..config.spec import PartSpec
from ..csrc import ops
from ..weights.loader import TensorNeed
from .base import MIXERS, CacheNeed
from .side_by_side import ProjectedMixer


class ChannelGatedRecurrence(ProjectedMixer):
    """HGRN2: a forget gate per channel that also decides what is written.  Per head of `head_dim` channels and `v_dim` values:
    q = silu(W_q h), v = W_v h, f = l + (1 - l) sigmoid(W_f h + b) with the stored lower bounds l;
        S = diag(f) S + (1 - f) v^T,    o = S^T q        (S zero at a sequence's start).
    Each head's o over its root mean square (`eps`) times a weight of v_dim values shared by the heads; the heads are
    concatenated and projected by W_o.  1 - f is worked out as (1 - l) sigmoid(-(W_f h + b)), so that gates near one keep their
    digits.  Everything between the projections' float32 results and the normed heads is float32.  A sequence's result
    depends on its own rows and state only.
    Parameters: hidden_size, heads, head_dim, v_dim, eps, names.{q, f, f_bias, lower, v, norm, o}."""

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.heads, self.head_dim, self.v_dim = int(spec["heads"]), int(spec["head_dim"]), int(spec["v_dim"])
        self.eps = float(spec["eps"])
        self.geometry = ops.GatedState(self.heads, self.head_dim, self.v_dim, False)
        self.f_bias = self.lower = self.norm = None
        self.cols = [0, 0, 0]

    @property
    def out_dim(self) -> int:
        return self.heads * self.v_dim

    @staticmethod
    def cache_need(spec: PartSpec) -> CacheNeed:
        return CacheNeed("state", state_shape=(ops.GatedState(int(spec["heads"]), int(spec["head_dim"]), int(spec["v_dim"]), False).floats,))

    @staticmethod
    def tensor_needs(spec: PartSpec) -> List[TensorNeed]:
        h, n = int(spec["hidden_size"]), spec["names"]
        hd, hv = int(spec["heads"]) * int(spec["head_dim"]), int(spec["heads"]) * int(spec["v_dim"])
        return [TensorNeed(n["q"], (hd, h)), TensorNeed(n["f"], (hd, h)), TensorNeed(n["f_bias"], (hd,), role="vector", init="linear"),
                TensorNeed(n["lower"], (hd,), role="vector", init="linear"), TensorNeed(n["v"], (hv, h)),
                TensorNeed(n["norm"], (int(spec["v_dim"]),), role="vector", init="norm"), TensorNeed(n["o"], (h, hv))]

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        n = self.spec["names"]
        self.cols = self.take([tensors[n["q"]], tensors[n["f"]], tensors[n["v"]]], tensors[n["o"]])
        self.f_bias, self.lower, self.norm = (tensors[n[s]].contiguous() for s in ("f_bias", "lower", "norm"))

    def mix(self, ctx, entry, proj, col, act, act_col, scale, n_rows):
        ws, rows, g = ctx.ws, ctx.ws.max_rows, self.geometry
        state = ctx.cache.state(entry, self.tag)
        hd, hv = self.heads * self.head_dim, self.heads * self.v_dim
        o = ws.buffer("gscan.o", (rows, hv), torch.float32)
        q_col, f_col, v_col = (col + c for c in self.cols)
        raw = ops.gated_raw(proj, q_col, f_col, v_col, self.f_bias, lower=self.lower)
        if ctx.decode and self.head_dim <= ops.GATED_STEP_MAX_DIM:
            ops.gated_step(g, raw, o, None, state, ctx.seq_first_row, ctx.seq_slot, ctx.n_seqs)
        else:
            gates = ws.buffer("gscan.channel_gates", (rows, 3 * hd), torch.float32)
            ops.channel_gates(raw, gates, n_rows, hd)
            ops.gated_scan(g, gates[:, :hd], gates[:, hd:2 * hd], gates[:, 2 * hd:], proj[:, v_col:v_col + hv], None, o, None, state,
                           ctx.seq_first_row, ctx.seq_slot, ctx.n_seqs)
        ops.scan_head_norm(o, self.norm, act, act_col, n_rows, self.heads, self.v_dim, self.eps, post=scale)


class MatrixMemory(ProjectedMixer):
    """The matrix memory of xLSTM.  Per head: q = W_q h / sqrt(head_dim), k = W_k h, v = W_v h, a log input gate
    i = cap tanh((W_i h + b_i) / cap) and a log forget gate f = logsigmoid(cap tanh((W_f h + b_f) / cap)).  With a running
    maximum m (zero at a sequence's start, as S and n are):
        m' = max(f + m, i);  S = exp(f + m - m') S + exp(i - m') k v^T;  n = exp(f + m - m') n + exp(i - m') k;
        o = S^T q / (max(|n . q|, exp(-m')) + 1e-6).
    Each head's o over its root mean square (`eps`); the concatenated heads times a weight, times sigmoid(W_g h), projected by
    W_o.  Everything between the projections' float32 results and the gated heads is float32.
    Parameters: hidden_size, heads, head_dim, v_dim, gate_cap, eps, names.{q, k, v, g, o, norm, i, i_bias, f, f_bias}."""
    TINY = 1e-6

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.heads, self.head_dim, self.v_dim = int(spec["heads"]), int(spec["head_dim"]), int(spec["v_dim"])
        self.eps, self.cap = float(spec["eps"]), float(spec["gate_cap"])
        self.geometry = ops.GatedState(self.heads, self.head_dim, self.v_dim, True)
        self.i_bias = self.f_bias = self.norm = None
        self.cols = [0] * 6

    @property
    def out_dim(self) -> int:
        return self.heads * self.v_dim

    @staticmethod
    def cache_need(spec: PartSpec) -> CacheNeed:
        return CacheNeed("state", state_shape=(ops.GatedState(int(spec["heads"]), int(spec["head_dim"]), int(spec["v_dim"]), True).floats,))

    @staticmethod
    def tensor_needs(spec: PartSpec) -> List[TensorNeed]:
        h, n, heads = int(spec["hidden_size"]), spec["names"], int(spec["heads"])
        hd, hv = heads * int(spec["head_dim"]), heads * int(spec["v_dim"])
        return [TensorNeed(n["q"], (hd, h)), TensorNeed(n["k"], (hd, h)), TensorNeed(n["v"], (hv, h)), TensorNeed(n["g"], (hv, h)),
                TensorNeed(n["o"], (h, hv)), TensorNeed(n["norm"], (hv,), role="vector", init="norm"),
                TensorNeed(n["i"], (heads, h)), TensorNeed(n["i_bias"], (heads,), role="vector", init="linear"),
                TensorNeed(n["f"], (heads, h)), TensorNeed(n["f_bias"], (heads,), role="vector", init="linear")]

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        n = self.spec["names"]
        self.cols = self.take([tensors[n[s]] for s in ("q", "k", "v", "g", "i", "f")], tensors[n["o"]])
        self.i_bias, self.f_bias, self.norm = (tensors[n[s]].contiguous() for s in ("i_bias", "f_bias", "norm"))

    def mix(self, ctx, entry, proj, col, act, act_col, scale, n_rows):
        ws, rows, g = ctx.ws, ctx.ws.max_rows, self.geometry
        state = ctx.cache.state(entry, self.tag)
        hd, hv = self.heads * self.head_dim, self.heads * self.v_dim
        o = ws.buffer("gscan.o", (rows, hv), torch.float32)
        nq, em = (ws.buffer("gscan." + s, (rows, self.heads), torch.float32) for s in ("nq", "em"))
        q_col, k_col, v_col, g_col, i_col, f_col = (col + c for c in self.cols)
        raw = ops.gated_raw(proj, q_col, k_col, v_col, self.f_bias, i_col=i_col, f_col=f_col, i_bias=self.i_bias, cap=self.cap, geometry=g, em=em,
                            seq_pos0=ctx.seq_pos0)
        if ctx.decode and self.head_dim <= ops.GATED_STEP_MAX_DIM:
            ops.gated_step(g, raw, o, nq, state, ctx.seq_first_row, ctx.seq_slot, ctx.n_seqs)
        else:
            gates = ws.buffer("gscan.head_gates", (rows, self.heads, 2), torch.float32)
            ops.head_gates(g, raw, gates, state, ctx.seq_first_row, ctx.seq_slot, ctx.n_seqs)
            ops.gated_scan(g, proj[:, q_col:q_col + hd], proj[:, k_col:k_col + hd], None, proj[:, v_col:v_col + hv], gates, o, nq, state,
                           ctx.seq_first_row, ctx.seq_slot, ctx.n_seqs)
        ops.scan_head_norm(o, self.norm, act, act_col, n_rows, self.heads, self.v_dim, self.eps, nq=nq, em=em, q_scale=self.head_dim ** -0.5,
                           tiny=self.TINY, gate=proj[:, g_col:g_col + hv], post=scale)


MIXERS.register("channel_gated_recurrence", ChannelGatedRecurrence)
MIXERS.register("matrix_memory", MatrixMemory)
