"""Mixers that are one projection, a core and one output product, and two of them side by side over the same rows."""
from __future__ import annotations

from dataclasses import replace
from typing import List, Mapping, Optional, Tuple

import torch

from ..config.spec import ConfigError, PartSpec
from ..weights.loader import TensorNeed
from .base import MIXERS, CacheNeed, Mixer
from .linear import Linear

COLUMN_ALIGN = 8


def pack_rows(parts: List[torch.Tensor]) -> Tuple[torch.Tensor, List[int]]:
    """The matrices stacked along their rows, each starting at a multiple of COLUMN_ALIGN (rows of zeros between), and
    where each starts: the columns of the packed product's result."""
    cols, rows, at = [], [], 0
    for p in parts:
        cols.append(at)
        rows.append(p)
        pad = -p.shape[0] % COLUMN_ALIGN
        if pad:
            rows.append(torch.zeros((pad, p.shape[1]), dtype=p.dtype, device=p.device))
        at += p.shape[0] + pad
    return torch.cat(rows, dim=0).contiguous(), cols


class ProjectedMixer(Mixer):
    """A mixer whose projections are one packed product of its input rows with a float32 result (what follows, norms, gates,
    a recurrence, is computed in 32-bit from unrounded projections) and whose result is one product of the rows its core
    writes.  A subclass packs its projections in `bind` through `take` and implements `mix`, which reads columns `col` .. of
    the projection and writes `out_dim` columns from `act_col` on of the activation rows, times `scale`.  So two such mixers
    can share both products (`SideBySide`).  `tag` is the tag of the state it keeps."""
    replayable = True
    tag = ""

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.hidden = int(spec["hidden_size"])
        self.in_weight: Optional[torch.Tensor] = None
        self.out_weight: Optional[torch.Tensor] = None
        self.inp: Optional[Linear] = None
        self.out: Optional[Linear] = None

    @property
    def out_dim(self) -> int:
        raise NotImplementedError

    def take(self, projections: List[torch.Tensor], out_weight: torch.Tensor) -> List[int]:
        self.in_weight, cols = pack_rows(projections)
        self.out_weight = out_weight
        return cols

    def release_weights(self) -> Tuple[torch.Tensor, torch.Tensor]:
        """The packed projection and the output matrix, handed over to a part that packs them further."""
        w = (self.in_weight, self.out_weight)
        self.in_weight = self.out_weight = None
        return w

    def weight_bytes(self) -> int:
        return (self.inp.weight_bytes() + self.out.weight_bytes()) if self.inp is not None else 0

    def mix(self, ctx, entry: int, proj: torch.Tensor, col: int, act: torch.Tensor, act_col: int, scale: float, n_rows: int) -> None:
        raise NotImplementedError

    def forward(self, ctx, entry, x, n_rows, cache_entry=None, write_cache=True):
        if cache_entry is not None or not write_cache:
            raise ValueError("this mixer keeps a cache or state of its own; it cannot read another entry's")
        if self.inp is None:
            self.inp, self.out = (Linear(w) for w in self.release_weights())
        return project_mix_project(ctx, self.env.dtype, x, n_rows, self.inp, self.out, self.hidden,
                                   lambda proj, act: self.mix(ctx, entry, proj, 0, act, 0, 1.0, n_rows))


def project_mix_project(ctx, dtype, x, n_rows, inp: Linear, out: Linear, hidden: int, core) -> torch.Tensor:
    ws, rows = ctx.ws, ctx.ws.max_rows
    proj = ws.buffer("mix.proj", (rows, inp.out_features), torch.float32)
    act = ws.buffer("mix.act", (rows, out.in_features), dtype)
    delta = ws.buffer("delta", (rows, hidden), dtype)
    inp(x, proj, n_rows)
    core(proj, act)
    out(act, delta, n_rows)
    return delta


class SideBySide(Mixer):
    """left_scale * left(x) + right_scale * right(x): two projected mixers over the same rows.  One product makes both mixers'
    projections, each core writes its results, times its scale, into its columns of one activation row, and one product
    with both output matrices side by side projects and sums them (in the product's float32 accumulators).
    Parameters: hidden_size, left, right (PartSpecs of projected mixers), left_scale, right_scale."""
    replayable = True
    SIDES = ("left", "right")

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.hidden = int(spec["hidden_size"])
        self.scales = [float(spec[s + "_scale"]) for s in self.SIDES]
        self.sides: List[ProjectedMixer] = []
        for s in self.SIDES:
            side = self._class(spec[s])(spec[s], env)
            side.tag = s
            self.sides.append(side)
        self.inp = self.out = None
        self.cols: List[int] = []
        self.act_cols: List[int] = []

    @staticmethod
    def _class(spec: PartSpec):
        cls = MIXERS.get(spec.kind)
        if not issubclass(cls, ProjectedMixer):
            raise ConfigError(f"a mixer of kind {spec.kind!r} cannot run beside another one")
        return cls

    @classmethod
    def cache_needs(cls, spec: PartSpec) -> List[CacheNeed]:
        return [replace(n, tag=s) if n.kind == "state" else n for s in cls.SIDES for n in cls._class(spec[s]).cache_needs(spec[s])]

    @staticmethod
    def tensor_needs(spec: PartSpec) -> List[TensorNeed]:
        return [n for s in SideBySide.SIDES for n in SideBySide._class(spec[s]).tensor_needs(spec[s])]

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        ins, outs = [], []
        for side in self.sides:
            side.bind(tensors)
            w_in, w_out = side.release_weights()
            ins.append(w_in)
            outs.append(w_out)
        packed, self.cols = pack_rows(ins)
        self.inp, self.out = Linear(packed), Linear(torch.cat(outs, dim=1).contiguous())
        self.act_cols = [0, self.sides[0].out_dim]

    def weight_bytes(self) -> int:
        return self.inp.weight_bytes() + self.out.weight_bytes()

    def forward(self, ctx, entry, x, n_rows, cache_entry=None, write_cache=True):
        if cache_entry is not None or not write_cache:
            raise ValueError("mixers side by side keep caches and states of their own; they cannot read another entry's")

        def core(proj, act):
            for side, col, act_col, scale in zip(self.sides, self.cols, self.act_cols, self.scales):
                side.mix(ctx, entry, proj, col, act, act_col, scale, n_rows)

        return project_mix_project(ctx, self.env.dtype, x, n_rows, self.inp, self.out, self.hidden, core)


MIXERS.register("side_by_side", SideBySide)
