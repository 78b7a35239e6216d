"""Normalisation parts."""
from __future__ import annotations

import torch

from .. import kernels
from ..weights.spec import VECTOR, TensorSpec
from .base import Norm
from .linear import LazyNorm


class LayerNorm(Norm):
    """Affine LayerNorm over the last axis, biased variance, statistics in 32-bit
    (src/models/gpt2/model.rs:143-148, 235-239 of the reference)."""

    def __init__(self, width: int, eps: float, bias: bool = True):
        self.width, self.eps, self.has_bias = width, float(eps), bias

    def specs(self):
        specs = {"weight": TensorSpec((self.width,), VECTOR, ("ones",))}
        if self.has_bias:
            specs["bias"] = TensorSpec((self.width,), VECTOR, ("zeros",))
        return specs

    fusable = True      # linear kernels know how to apply this norm to their rows on the way in
    fused_kind = "layernorm"

    def forward(self, ctx, x32, out_dtype, rows=None, n_rows=None, lazy=False):
        """Normalised rows; with `lazy` (and bfloat16 output, few rows) a handle that the next matrix product
        resolves, normalising inside its own kernel."""
        n = n_rows if n_rows is not None else ctx.n_tokens
        if lazy and out_dtype == torch.bfloat16 and n <= 16:
            return LazyNorm(self, x32, rows, n)
        return self.apply(ctx, x32, out_dtype, rows, n)

    def apply(self, ctx, x32, out_dtype, rows, n):
        out = ctx.ws.take((n, self.width), out_dtype)
        kernels.layernorm(x32, self.t_weight, self.t_bias if self.has_bias else None, out, self.eps, rows=rows, n_rows=n)
        return out


class RmsNorm(Norm):
    """x / sqrt(mean(x^2) + eps) * (offset + weight) over the last axis, in 32-bit, eps inside the root; no shift.
    `offset` 1: the file keeps the gain minus one; the sum is formed once, in 32-bit, when the weights are bound.
    `one_gain`: the file keeps a single number (a tensor of no axes) that scales all channels; it is spread over the
    channels when the weights are bound, so that every kernel that takes a norm's weight takes this one."""

    has_bias = False

    def __init__(self, width: int, eps: float, offset: float = 0.0, one_gain: bool = False):
        self.width, self.eps, self.offset, self.one_gain = width, float(eps), float(offset), one_gain

    def specs(self):
        shape = () if self.one_gain else (self.width,)
        return {"weight": TensorSpec(shape, VECTOR, ("ones",) if self.offset == 0.0 else ("normal", 0.1))}

    def bind(self, tensors):
        if self.offset != 0.0:
            tensors = {name: t.to(torch.float32) + self.offset for name, t in tensors.items()}
        if self.one_gain:
            tensors = {name: t.to(torch.float32).reshape(1).expand(self.width).contiguous() for name, t in tensors.items()}
        super().bind(tensors)

    fusable = True      # (as LayerNorm: the products for few rows norm on the way in)
    fused_kind = "rmsnorm"

    def forward(self, ctx, x32, out_dtype, rows=None, n_rows=None, lazy=False):
        n = n_rows if n_rows is not None else ctx.n_tokens
        if lazy and out_dtype == torch.bfloat16 and n <= 16:
            return LazyNorm(self, x32, rows, n)
        return self.apply(ctx, x32, out_dtype, rows, n)

    def apply(self, ctx, x32, out_dtype, rows, n):
        if rows is not None:
            x32 = x32.index_select(0, rows[:n].long())
        out = ctx.ws.take((n, self.width), out_dtype)
        kernels.rmsnorm(x32, self.t_weight, out, self.eps, n_rows=n)
        return out
