"""A recurrent mixer with a matrix state per head whose every write corrects what the state already answers for its key."""
from __future__ import annotations

from typing import List, Mapping

import torch

from ..config.spec import PartSpec
from ..csrc import ops
from ..weights.loader import TensorNeed
from .base import MIXERS, CacheNeed
from .side_by_side import ProjectedMixer

CONVOLVED = ("q", "k", "v")


class GatedDeltaRule(ProjectedMixer):
    """The gated delta rule.  q and k of `kv_heads` heads of `head_dim` channels, v of `heads` heads of `v_dim` values (head h
    uses q and k of head h // (heads / kv_heads)): each a projection, a causal convolution of `taps` taps per channel (the last
    one meets the current token, zeros before a sequence's first) and silu; q and k are then divided by sqrt(sum(x^2) + 1e-6)
    per head, q by sqrt(head_dim) besides.  Per head, with beta = sigmoid(W_b h) and g = exp(-exp(A_log) softplus(W_a h +
    dt_bias)), and the state S [channel, value] zero at a sequence's start:
        S = g S;   u = beta (v - S^T k);   S = S + k u^T;   o = S^T q.
    Each head's o over its root mean square (`eps`), times a weight of v_dim values shared by the heads, times silu(W_g h); the
    heads are concatenated and projected by W_o.

    What a sequence keeps is one float32 row: the heads' states and the last inputs of the convolutions.  Everything between the
    projections' float32 results and the gated heads is float32; passes of one token per sequence do it in one launch.  A
    sequence's result depends on its own rows and state only.
    Parameters: hidden_size, heads, kv_heads, head_dim, v_dim, taps, eps, names.{q, k, v, q_conv, k_conv, v_conv, a, b, A_log,
    dt_bias, norm, g, o}."""

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.geometry = self.geometry_of(spec)
        self.eps = float(spec["eps"])
        self.conv = self.A = self.dt_bias = self.norm = None
        self.cols = [0] * 6

    @staticmethod
    def geometry_of(spec: PartSpec) -> ops.DeltaState:
        return ops.DeltaState(int(spec["heads"]), int(spec["kv_heads"]), int(spec["head_dim"]), int(spec["v_dim"]), int(spec["taps"]))

    @property
    def out_dim(self) -> int:
        return self.geometry.heads * self.geometry.v_dim

    @staticmethod
    def cache_need(spec: PartSpec) -> CacheNeed:
        return CacheNeed("state", state_shape=(GatedDeltaRule.geometry_of(spec).floats,))

    @staticmethod
    def tensor_needs(spec: PartSpec) -> List[TensorNeed]:
        h, n, g = int(spec["hidden_size"]), spec["names"], GatedDeltaRule.geometry_of(spec)
        rows = {"q": g.kv_heads * g.dim, "k": g.kv_heads * g.dim, "v": g.heads * g.v_dim}
        needs = []
        for s in CONVOLVED:
            needs += [TensorNeed(n[s], (rows[s], h)), TensorNeed(n[s + "_conv"], (rows[s], g.taps), role="vector", init="linear")]
        return needs + [TensorNeed(n["a"], (g.heads, h)), TensorNeed(n["b"], (g.heads, h)), TensorNeed(n["A_log"], (g.heads,), role="vector", init="linear"),
                        TensorNeed(n["dt_bias"], (g.heads,), role="vector", init="linear"), TensorNeed(n["norm"], (g.v_dim,), role="vector", init="norm"),
                        TensorNeed(n["g"], (rows["v"], h)), TensorNeed(n["o"], (h, rows["v"]))]

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        n = self.spec["names"]
        self.cols = self.take([tensors[n[s]] for s in ("q", "k", "v", "a", "b", "g")], tensors[n["o"]])
        f32 = lambda s: tensors[n[s]].to(torch.float32).contiguous()
        self.conv = torch.cat([f32(s + "_conv") for s in CONVOLVED], dim=0).contiguous()
        self.A = torch.exp(tensors[n["A_log"]].to(torch.float64)).to(torch.float32).contiguous()
        self.dt_bias, self.norm = f32("dt_bias"), f32("norm")

    def mix(self, ctx, entry, proj, col, act, act_col, scale, n_rows):
        if act_col or act.shape[-1] != self.out_dim or scale != 1.0:
            raise ValueError("a delta rule does not run beside another mixer")
        ws, rows, g = ctx.ws, ctx.ws.max_rows, self.geometry
        state = ctx.cache.state(entry, self.tag)
        one = ctx.decode and g.step_takes()
        buffers = {} if one else dict(planes=ws.buffer("delta.planes", (rows, g.plane_floats), torch.float32), gates=ws.buffer("delta.gates", (rows, 4 * g.heads), torch.float32),
                                      o=ws.buffer("delta.o", (rows, self.out_dim), torch.float32))
        a = ops.delta_arg(g, proj, [col + c for c in self.cols], self.conv, self.A, self.dt_bias, self.norm, g.dim ** -0.5, self.eps, state, ctx.row_slot,
                          ctx.row_pos, ctx.seq_first_row, ctx.seq_slot, ctx.seq_pos0, n_rows, **buffers)
        if one:
            ops.delta_step(a, act, ctx.n_seqs)
        else:
            ops.delta_prepare(a)
            # 32-bit runs walk token by token, so that a token's bits do not depend on where its pass began
            if self.env.dtype == torch.bfloat16 and ctx.max_seq_rows >= ops.DELTA_CHUNK and g.chunks_take():
                ops.delta_chunk_scan(a, ws.buffer("delta.coef", (rows, g.heads * ops.DELTA_COEF), torch.float32), ctx.n_seqs, ctx.max_seq_rows)
            else:
                ops.delta_scan(a, ctx.n_seqs)
            ops.delta_head_norm(a, act)


MIXERS.register("gated_delta_rule", GatedDeltaRule)
