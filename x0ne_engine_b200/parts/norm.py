"""Norms with the residual add fused in front of them."""
from __future__ import annotations

from typing import List, Mapping

import torch

from ..config.spec import PartSpec
from ..csrc import ops
from ..weights.loader import TensorNeed
from .base import NORMS, Norm


class PostNormed:
    """A sublayer's result that is still to be normed by `norm` (an RMSNorm of its own) before it joins the
    residual: what a layer with norms after its sublayers hands to the next add.  The norm that takes it
    norms the delta in float32, adds it, and norms the sum, in one launch.  `bias` (float32, or None) is still to be
    added to the delta before its norm."""
    __slots__ = ("delta", "norm", "bias")

    def __init__(self, delta: torch.Tensor, norm: "RMSNorm", bias=None):
        self.delta = delta
        self.norm = norm
        self.bias = bias


def scaled_weight(spec: PartSpec, tensors: Mapping[str, torch.Tensor], weight: torch.Tensor) -> torch.Tensor:
    """A norm's weight times the layer scale its result is multiplied by (`names.scale`), if it has one."""
    scale = spec["names"].get("scale")
    return weight if scale is None else (weight * tensors[scale]).contiguous()


def scale_needs(spec: PartSpec) -> List[TensorNeed]:
    scale = spec["names"].get("scale")
    return [] if scale is None else [TensorNeed(scale, (int(spec["size"]),), role="vector", init="norm")]


class RMSNorm(Norm):
    """out = r * rsqrt(mean(r^2) + eps) * w with r = resid + delta, in float32; eps inside the
    root, the weight multiplies directly (x0ne-core/kernels/cuda/rmsnorm.cu:11-20).
    With `groups` > 1 the row is that many equal consecutive parts and each is divided by its own root mean square;
    the weight still has one value per value of the row.  With `one_plus` the stored weight is centred on zero: the factor is
    1 + w.  With `names.scale` the result is multiplied by a second vector (a layer scale).
    Parameters: size, eps, groups (default 1), one_plus (default False), names.{weight, scale}."""
    replayable = True
    centred = False

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.size = int(spec["size"])
        self.eps = float(spec["eps"])
        self.groups = int(spec.get("groups") or 1)
        if self.groups < 1 or self.size % self.groups:
            raise ValueError(f"a norm over {self.size} values cannot have {self.groups} equal groups")
        self.one_plus = bool(spec.get("one_plus"))
        self.weight = None

    @staticmethod
    def tensor_needs(spec: PartSpec) -> List[TensorNeed]:
        return [TensorNeed(spec["names"]["weight"], (int(spec["size"]),), role="vector", init="linear" if spec.get("one_plus") else "norm")] + scale_needs(spec)

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        w = tensors[self.spec["names"]["weight"]]
        self.weight = scaled_weight(self.spec, tensors, (w + 1.0).contiguous() if self.one_plus else w)

    def add_norm(self, ctx, resid, delta, out, n_rows, rows=None):
        if isinstance(delta, PostNormed):
            if self.groups != 1 or delta.norm.groups != 1:
                raise ValueError("a norm in groups does not take a result that is still to be normed")
            if delta.norm.centred:
                add_any_norm(self, resid, delta, out, n_rows, rows)
                return
            ops.add_normed_rmsnorm(resid, delta.delta, delta.norm.weight, delta.norm.eps, self.weight, out, n_rows, self.eps, rows,
                                   delta_bias=delta.bias)
        else:
            ops.add_rmsnorm(resid, delta, self.weight, out, n_rows, self.eps, rows, groups=self.groups)


class LayerNorm(Norm):
    """out = (r - mean(r)) / sqrt(mean((r - mean(r))^2) + eps) * w with r = resid + delta, in float32: a weight, no bias.  With
    `names.scale` the result is multiplied by a second vector (a layer scale).
    Parameters: size, eps, names.{weight, scale}."""
    replayable = True
    centred = True
    groups = 1

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.size = int(spec["size"])
        self.eps = float(spec["eps"])
        self.weight = None

    @staticmethod
    def tensor_needs(spec: PartSpec) -> List[TensorNeed]:
        return [TensorNeed(spec["names"]["weight"], (int(spec["size"]),), role="vector", init="norm")] + scale_needs(spec)

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        self.weight = scaled_weight(self.spec, tensors, tensors[self.spec["names"]["weight"]])

    def add_norm(self, ctx, resid, delta, out, n_rows, rows=None):
        if isinstance(delta, PostNormed) and delta.norm.groups != 1:
            raise ValueError("a result that is still to be normed in groups is not taken by this norm")
        add_any_norm(self, resid, delta, out, n_rows, rows)


def add_any_norm(norm, resid, delta, out, n_rows, rows) -> None:
    """The add and the norm where one of the two norms involved subtracts the mean."""
    if isinstance(delta, PostNormed):
        ops.add_norm(resid, delta.delta, norm.weight, out, n_rows, norm.eps, norm.centred, rows, delta_weight=delta.norm.weight,
                     delta_eps=delta.norm.eps, delta_centred=delta.norm.centred, delta_bias=delta.bias)
    elif delta is None or isinstance(delta, torch.Tensor):
        ops.add_norm(resid, delta, norm.weight, out, n_rows, norm.eps, norm.centred, rows)
    else:
        raise ValueError("a norm that subtracts the mean takes the pending result of a layer as one tensor")


NORMS.register("rmsnorm", RMSNorm)
NORMS.register("layernorm", LayerNorm)
