"""A minimal gated recurrence: one gate that reads the current token only, a state of one number a channel."""
from __future__ import annotations

import torch

from .. import kernels
from ..cache.spec import CacheNeed, StateSpec
from ..errors import ShapeError
from ..weights.spec import MATRIX, VECTOR, TensorSpec
from .base import Mixer
from .linear import linear


class MinGru(Mixer):
    """Per channel of `inner` a 32-bit state S (zero for a new sequence) that every token moves towards a value of its own:

        z = sigmoid(W_z h + b_z)                        how far
        u = W_x h + b_x,  v = u + 1/2 if u >= 0 else sigmoid(u)      towards what
        S <- (1 - z) S + z v
        y = S * g sigmoid(g),  g = W_g h,  then W_o

    The three projections are one product; from the biases on everything is 32-bit (csrc/min_gru.cu), long runs of new
    tokens are scanned in parallel.  The state is the layer's only cache: `StateSpec("s", (inner,))`, one row per live
    sequence.

    Tensors (stored [out, in]): `in.weight` = rows of W_z, W_x, W_g; `bias` [2 * inner] = b_z, b_x; `out.weight`
    [width, inner].
    """

    accepts_lazy_norm = True
    # `forward(..., store=True)` writes the result into `residual` instead of adding it (rows that hold nothing yet)
    can_store = True

    def __init__(self, width: int, inner: int, *, init_std: float = 0.02, out_init_std: float | None = None):
        if min(width, inner) <= 0:
            raise ShapeError("minimal GRU: sizes must be positive")
        self.width, self.inner, self.in_width = width, inner, 3 * inner
        self.init_std = init_std
        self.out_init_std = init_std if out_init_std is None else out_init_std

    def specs(self):
        return {"in.weight": TensorSpec((self.in_width, self.width), MATRIX, ("normal", self.init_std)),
                "bias": TensorSpec((2 * self.inner,), VECTOR, ("normal", 0.5)),
                "out.weight": TensorSpec((self.width, self.inner), MATRIX, ("normal", self.out_init_std))}

    def bind(self, tensors):
        super().bind(tensors)
        self.z_bias, self.x_bias = self.t_bias[:self.inner].contiguous(), self.t_bias[self.inner:].contiguous()

    def cache_need(self):
        return CacheNeed(states=(StateSpec("s", (self.inner,), torch.float32),))

    def forward(self, ctx, x, residual, entry, owns_cache=True, store=False):
        if getattr(ctx, "program", None) is not None:
            from ..engine.program import ProgramUnsupported
            raise ProgramUnsupported("a minimal GRU has no phase in the fused step")
        if not owns_cache:
            raise ShapeError("minimal GRU: a recurrent state cannot be another layer's")
        mark = ctx.ws.mark()      # (this layer's scratch is handed out again to the next one)
        n, inner = ctx.n_tokens, self.inner
        proj = ctx.ws.take((n, self.in_width), ctx.dtype)
        linear(ctx, x, self.t_in_weight, None, proj, m=n, w_is_nk=True)
        read = ctx.ws.take((n, inner), ctx.dtype)
        kernels.min_gru(proj, 0, inner, 2 * inner, self.z_bias, self.x_bias, ctx.cache.state(entry, "s"), ctx.slots,
                        ctx.seq_start, read, n_seqs=ctx.n_seqs, max_new=ctx.max_new)
        linear(ctx, read, self.t_out_weight, None, residual, m=n, residual=None if store else residual, w_is_nk=True)
        ctx.ws.release(mark)
