"""Norms of the residual stream: RMS norm with a weight offset, layer norm, Dynamic Tanh, and the RMS norm in groups.

y = x / sqrt(mean(x^2) + eps) * (offset + w).  Gemma2 stores w and uses 1 + w
(`gemma/gemma.go:22-28`); offset 0 is the usual RMS norm (`qwen/norm.go:10-27`).
eps lies inside the root, added to the mean (`cpu/cpu_ops.go:145-162`).  The
sum of squares, the root and offset + w are float32 whatever the model's dtype.

`LayerNorm` takes the mean off first and has a weight and no bias: y = (x - mean) / sqrt(mean((x - mean)^2) + eps) * w.

`DynamicTanh` takes no statistics of the row: y = tanh(alpha x) * w + b with a stored scalar alpha and vectors w
and b, element by element, in float32.

`GroupRMSNorm` cuts the row into `groups` equal runs and divides each by its own sqrt(mean(run^2) + eps) before the
whole is multiplied by w.  It can norm the stream itself after a scaled residual sum (`scaled_add`: h <- N(a h + r)),
which is what a block that norms after the sum needs.

`plain_residual_add` is the residual sum of blocks without a norm after the sublayer; it also takes a factor per feature
on the sublayer's result (`FeatureScale`), a result that is still two branches to be normed and averaged
(`NormedBranches`), and rows that join the sum (`StreamPlus`, a norm over the stream plus those rows): all of it and
the norm behind it are one pass over the stream.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from ..weights.loader import TensorSpec
from .base import Norm, Part, Runtime, StepContext


class RMSNorm(Norm):
    def __init__(self, width: int, eps: float, weight_name: str, offset: float = 0.0, init_std: float = 0.1,
                 init_mean: float = 0.0):
        self.width = width
        self.eps = float(eps)
        self.offset = float(offset)
        self.weight_name = weight_name
        self.init_std, self.init_mean = init_std, init_mean      # how random weights are drawn
        self.weight = None          # float32: offset + w

    def tensor_specs(self):
        return {self.weight_name: TensorSpec((self.width,), init_std=self.init_std, init_mean=self.init_mean)}

    def load(self, store, rt: Runtime):
        self.weight = (store.get(self.weight_name).to(torch.float32) + self.offset).contiguous()

    def forward(self, x, ctx: StepContext, out, rows=None):
        return ctx.rt.ops.rmsnorm(x, self.weight, self.eps, out, rows)

    def residual_add(self, h, r, ctx: StepContext, next_norm: Norm | None = None, out=None):
        """h += self(r); out = next_norm(h) when a next norm is given."""
        if next_norm is None:
            ctx.rt.ops.add_rmsnorm(h, r, self.weight, self.eps)
            return None
        if isinstance(next_norm, RMSNorm):
            return ctx.rt.ops.add_rmsnorm(h, r, self.weight, self.eps, next_norm.weight, next_norm.eps, out)
        ctx.rt.ops.add_rmsnorm(h, r, self.weight, self.eps)
        return next_norm.forward(h, ctx, out)


class LayerNorm(Norm):
    """(x - mean) / sqrt(mean((x - mean)^2) + eps) * w, without a bias; x is the float32 stream."""

    def __init__(self, width: int, eps: float, weight_name: str, init_std: float = 0.1, init_mean: float = 1.0):
        self.width, self.eps, self.weight_name = width, float(eps), weight_name
        self.init_std, self.init_mean = init_std, init_mean
        self.weight = None          # float32

    def tensor_specs(self):
        return {self.weight_name: TensorSpec((self.width,), init_std=self.init_std, init_mean=self.init_mean)}

    def load(self, store, rt: Runtime):
        self.weight = store.get(self.weight_name).to(torch.float32).contiguous()

    def forward(self, x, ctx: StepContext, out, rows=None):
        return ctx.rt.ops.stream_norm(x, w_next=self.weight, eps_next=self.eps, centred=True, out=out, rows=rows)

    def residual_add(self, h, r, ctx: StepContext, next_norm: Norm | None = None, out=None):
        raise NotImplementedError("a layer norm stands before a sublayer, not after one")


class DynamicTanh(Norm):
    """y = tanh(alpha x) * w + b.  Tensors: `weight_name` [width], `<weight_name>.b` [width], `<weight_name>.alpha` []
    (other names through `bias_name` and `alpha_name`)."""

    def __init__(self, width: int, weight_name: str, bias_name: str | None = None, alpha_name: str | None = None,
                 init_std: float = 0.1, init_mean: float = 1.0, init_alpha: float = 0.5):
        self.width = width
        self.weight_name = weight_name
        self.bias_name = bias_name or weight_name + ".b"
        self.alpha_name = alpha_name or weight_name + ".alpha"
        self.init_std, self.init_mean, self.init_alpha = init_std, init_mean, init_alpha
        self.weight = self.bias = None      # float32
        self.alpha = 0.0

    def tensor_specs(self):
        return {self.weight_name: TensorSpec((self.width,), init_std=self.init_std, init_mean=self.init_mean),
                self.bias_name: TensorSpec((self.width,), init_std=self.init_std),
                self.alpha_name: TensorSpec((), init_std=0.1 * self.init_alpha, init_mean=self.init_alpha)}

    def load(self, store, rt: Runtime):
        self.weight = store.get(self.weight_name).to(torch.float32).contiguous()
        self.bias = store.get(self.bias_name).to(torch.float32).contiguous()
        self.alpha = float(store.get(self.alpha_name).to(torch.float32).reshape(()).item())

    def forward(self, x, ctx: StepContext, out, rows=None):
        return ctx.rt.ops.dyt_norm(x, None, self.alpha, self.weight, self.bias, out, rows)

    def after_add(self, h, r, ctx: StepContext, out):
        """h += r and out = self(h) in one pass over the stream."""
        return ctx.rt.ops.dyt_norm(h, r, self.alpha, self.weight, self.bias, out)

    def residual_add(self, h, r, ctx: StepContext, next_norm: Norm | None = None, out=None):
        raise NotImplementedError("Dynamic Tanh stands before a sublayer, not after one")


class GroupRMSNorm(Norm):
    def __init__(self, width: int, eps: float, groups: int, weight_name: str, init_std: float = 0.1, init_mean: float = 1.0):
        if groups < 1 or width % groups:
            raise ValueError(f"{groups} groups do not divide a width of {width}")
        self.width, self.eps, self.groups = width, float(eps), int(groups)
        self.weight_name = weight_name
        self.init_std, self.init_mean = init_std, init_mean
        self.weight = None          # float32

    def tensor_specs(self):
        return {self.weight_name: TensorSpec((self.width,), init_std=self.init_std, init_mean=self.init_mean)}

    def load(self, store, rt: Runtime):
        self.weight = store.get(self.weight_name).to(torch.float32).contiguous()

    def forward(self, x, ctx: StepContext, out, rows=None):
        return ctx.rt.ops.group_norm(x, None, 1.0, self.weight, self.eps, self.groups, out, rows)

    def scaled_add(self, h, r, alpha: float, ctx: StepContext, out=None):
        """h <- self(alpha h + r) on the float32 stream in place; out (when given) = the new h in the activation type."""
        return ctx.rt.ops.group_norm(h, r, alpha, self.weight, self.eps, self.groups, out)

    def residual_add(self, h, r, ctx: StepContext, next_norm: Norm | None = None, out=None):
        raise NotImplementedError("the norm in groups norms the stream itself (scaled_add), not a sublayer's output")


class FeatureScale(Part):
    """A stored factor per feature on a sublayer's result."""

    def __init__(self, width: int, weight_name: str, init_std: float = 0.1, init_mean: float = 1.0):
        self.width, self.weight_name = width, weight_name
        self.init_std, self.init_mean = init_std, init_mean
        self.weight = None          # float32

    def tensor_specs(self):
        return {self.weight_name: TensorSpec((self.width,), init_std=self.init_std, init_mean=self.init_mean)}

    def load(self, store, rt: Runtime):
        self.weight = store.get(self.weight_name).to(torch.float32).contiguous()


@dataclass
class NormedBranches:
    """A sublayer's result as its branches: share * sum_i r_i / sqrt(mean(r_i^2) + eps) * weight_i."""
    parts: list
    weights: list
    eps: float
    share: float


class StreamPlus(Norm):
    """A norm over the stream plus rows that join it for good: h += rows, then the norm."""

    def __init__(self, norm: Norm, plus):
        self.norm, self.plus = norm, plus

    def forward(self, x, ctx: StepContext, out, rows=None):
        if rows is not None:
            raise NotImplementedError("rows that join the stream join all of it")
        ctx.rt.ops.stream_norm(x, self.plus)
        return self.norm.forward(x, ctx, out)


def plain_residual_add(h, r, ctx: StepContext, next_norm: Norm | None = None, out=None, scale: FeatureScale | None = None):
    """h += scale * r for blocks without a norm after the sublayer; out = next_norm(h) when given."""
    branches = r if isinstance(r, NormedBranches) else None
    if branches is not None or scale is not None or isinstance(next_norm, (LayerNorm, StreamPlus)):
        more = None
        if isinstance(next_norm, StreamPlus):
            more, next_norm = next_norm.plus, next_norm.norm
        kw = {} if branches is None else {"branch_weights": branches.weights, "eps": branches.eps, "share": branches.share}
        fused = isinstance(next_norm, (LayerNorm, RMSNorm))
        if fused:
            kw.update(w_next=next_norm.weight, eps_next=next_norm.eps, centred=isinstance(next_norm, LayerNorm), out=out)
        ctx.rt.ops.stream_norm(h, r if branches is None else branches.parts, scale=scale.weight if scale is not None else None,
                               more=more, **kw)
        return out if fused else (next_norm.forward(h, ctx, out) if next_norm is not None else None)
    if isinstance(next_norm, RMSNorm):
        return ctx.rt.ops.add_rmsnorm(h, r, None, 0.0, next_norm.weight, next_norm.eps, out)
    if hasattr(next_norm, "after_add"):
        return next_norm.after_add(h, r, ctx, out)
    ctx.rt.ops.add_rmsnorm(h, r, None, 0.0)
    return next_norm.forward(h, ctx, out) if next_norm is not None else None
