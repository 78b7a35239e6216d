"""Gated linear attention: a recurrent state that forgets by a number per key channel and token."""
from __future__ import annotations

import torch

from .. import kernels
from ..cache.spec import CacheNeed, StateSpec
from ..errors import ShapeError
from ..weights.spec import MATRIX, VECTOR, TensorSpec
from .base import Mixer
from .linear import linear


class GatedLinearAttention(Mixer):
    """Per head a state S (dim x vdim, 32-bit, zero for a new sequence):

        q = W_q h * dim^-1/2,  k = W_k h,  v = W_v h
        z = W_a2 (W_a1 h) + b                          W_a1 of `rank` rows; z: heads * dim numbers
        a = sigmoid(z)^(1 / tau)                       the decay of every key channel
        S_t = diag(a_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t

    Each head's o_t is RMS-normed (one weight of vdim numbers for all heads, eps inside the root); the heads side by side
    are multiplied by g * sigmoid(g), g = W_g h, and projected by W_o into the residual stream.

    The logarithm of a decay is -softplus(-z) / tau: csrc/selective_scan.cu forms the softplus in 32-bit from the low-rank
    rows (with W_a2 and b negated when the weights are bound), csrc/gla.cu the rest.  The state is the layer's only cache:
    `StateSpec("s", (heads, dim, vdim))`, one row per live sequence.

    Tensors (stored [out, in]): `in.weight` = rows of W_q, W_k, W_v, W_g, W_a1 and zero rows up to `in_width`, a multiple of
    8; `decay.weight` [heads * dim, rank], `decay.bias` [heads * dim]; `norm.weight` [vdim]; `out.weight`
    [width, heads * vdim].
    """

    accepts_lazy_norm = True
    MAX_RANK = 160

    def __init__(self, width: int, n_heads: int, dim: int, vdim: int, rank: int, tau: float, eps: float, *,
                 init_std: float = 0.02, out_init_std: float | None = None):
        if min(width, n_heads, dim, vdim, rank) <= 0 or tau <= 0:
            raise ShapeError("gated linear attention: sizes must be positive")
        if dim > 256 or rank > self.MAX_RANK:
            raise ShapeError(f"gated linear attention: {dim} key channels a head (at most 256) and a decay rank of {rank} (at "
                             f"most {self.MAX_RANK}) are what its kernels take")
        self.width, self.n_heads, self.dim, self.vdim, self.rank, self.tau = width, n_heads, dim, vdim, rank, float(tau)
        self.eps = float(eps)
        self.qk_width, self.v_width = n_heads * dim, n_heads * vdim
        self.g_off = 2 * self.qk_width + self.v_width
        self.low_off = self.g_off + self.v_width
        self.low_rows = -(-(self.low_off + rank) // 8) * 8 - self.low_off       # W_a1's rows and the zero rows behind them
        self.in_width = self.low_off + self.low_rows
        self.init_std = init_std
        self.out_init_std = init_std if out_init_std is None else out_init_std

    def specs(self):
        return {"in.weight": TensorSpec((self.in_width, self.width), MATRIX, ("normal", self.init_std)),
                "decay.weight": TensorSpec((self.qk_width, self.rank), VECTOR, ("normal", self.rank ** -0.5)),
                "decay.bias": TensorSpec((self.qk_width,), VECTOR, ("normal", 1.0)),
                "norm.weight": TensorSpec((self.vdim,), VECTOR, ("ones",)),
                "out.weight": TensorSpec((self.width, self.v_width), MATRIX, ("normal", self.out_init_std))}

    def bind(self, tensors):
        super().bind(tensors)
        self.minus_decay = (-self.t_decay_weight).contiguous()
        self.minus_bias = (-self.t_decay_bias).contiguous()
        self.head_weights = self.t_norm_weight.repeat(self.n_heads).contiguous()

    def cache_need(self):
        return CacheNeed(states=(StateSpec("s", (self.n_heads, self.dim, self.vdim), torch.float32),))

    # `forward(..., store=True)` writes the result into `residual` instead of adding it (rows that hold nothing yet)
    can_store = True

    def forward(self, ctx, x, residual, entry, owns_cache=True, store=False):
        if getattr(ctx, "program", None) is not None:
            from ..engine.program import ProgramUnsupported
            raise ProgramUnsupported("gated linear attention has no phase in the fused step")
        if not owns_cache:
            raise ShapeError("gated linear attention: a recurrent state cannot be another layer's")
        mark = ctx.ws.mark()
        n, heads, dim, vdim = ctx.n_tokens, self.n_heads, self.dim, self.vdim
        proj = ctx.ws.take((n, self.in_width), ctx.dtype)
        linear(ctx, x, self.t_in_weight, None, proj, m=n, w_is_nk=True)
        dt = ctx.ws.take((n, self.qk_width), torch.float32)
        kernels.selective_scan_dt(proj[:, self.low_off:self.low_off + self.rank], self.minus_decay, self.minus_bias, dt,
                                  n_tokens=n)
        read = ctx.ws.take((n, self.v_width), torch.float32)
        mixed = ctx.ws.take((n, self.v_width), ctx.dtype)
        scratch = None
        if ctx.max_new > kernels.GLA_CHUNK:
            scratch = ctx.ws.take((kernels.gla_chunked_scratch_floats(n, ctx.n_seqs, ctx.max_new, heads, dim, vdim),),
                                  torch.float32)
        done = kernels.gla_scan(proj, 0, self.qk_width, 2 * self.qk_width, dim ** -0.5, dt, -1.0 / self.tau,
                                ctx.cache.state(entry, "s"), ctx.slots, ctx.seq_start, read, n_seqs=ctx.n_seqs, n_heads=heads,
                                dim=dim, vdim=vdim, max_new=ctx.max_new, scratch=scratch,
                                norm=(self.t_norm_weight, self.eps, self.g_off, mixed))
        if not done:
            kernels.rmsnorm(read, self.head_weights, mixed, self.eps, n_rows=n, gate=proj[:, self.g_off:self.low_off],
                            groups=heads, gate_rule="swish")
        linear(ctx, mixed, self.t_out_weight, None, residual, m=n, residual=None if store else residual, w_is_nk=True)
        ctx.ws.release(mark)
