"""Differential attention: every head is the difference of two softmax attentions over the same values."""
from __future__ import annotations

import torch

from .. import kernels
from ..cache.spec import PAGE_SIZE, CacheNeed, KvSpec, StateSpec
from ..errors import ShapeError
from ..weights.spec import MATRIX, VECTOR, TensorSpec
from .attention import _sm_count
from .base import Mixer
from .linear import linear


class DifferentialAttention(Mixer):
    """Causal attention with grouped key heads, two maps a head, behind a short convolution.

    With h the mixer's input, per position:

        u = W_in h + b_in                              rows [q | k | v]: 2 heads dim, 2 kv_heads dim, kv_heads vdim, each
                                                       head's two maps side by side
        c_t = sum_j conv[:, j] u_(t - taps + 1 + j)    per channel, causal, zeros before the sequence's start
        q, k <- per head and map x / rms(x) * weight ([dim], one for queries, one for keys), then turned by the position
        a_m[i, h] = sum_(j <= i) softmax_j(q_m[i, h] . k_m[j, g] * scale) v[j, g]       m = 1, 2; g = h // (heads / kv_heads)
        o = a_1 - share * a_2,  share = exp(lq1 . lk1) - exp(lq2 . lk2) + offset        one number for the layer
        y = W_out (o / rms(o) * (1 - offset))          rms over a head's vdim channels, no weight

    The convolution, norms, rotation, scores, softmax and everything up to the rounding of y's operand are 32-bit
    (csrc/differential_attention.cu).  The cache: one row [key 1 | key 2 | value] per position and key head
    (`KvSpec(kv_heads, 2 dim + vdim, has_values=False)`) and the last taps - 1 projected rows of every sequence as the state
    "qkv_taps".

    Tensors: `in.weight` [q + k + v rows, width], `in.bias`; `conv.weight` [q + k + v rows, taps]; `q_norm.weight`,
    `k_norm.weight` [dim]; `lq1`, `lk1`, `lq2`, `lk2` [dim]; `out.weight` [width, heads * vdim].  `taps` 1 is a product with
    one number a channel.
    """

    accepts_lazy_norm = True
    MAX_TAPS = 16
    # Steps whose longest run of new tokens is at least this take the tcgen05 kernel in bfloat16 where it takes the head sizes
    # (csrc/attention_prefill_tcgen05.cu: up to 128 key and 128 value channels, multiples of 8).
    prompt_from = 32

    def __init__(self, width: int, n_heads: int, n_kv_heads: int, dim: int, vdim: int, taps: int, scale: float, offset: float,
                 eps: float, positions, *, init_std: float = 0.02, out_init_std: float | None = None):
        if min(width, n_heads, n_kv_heads, dim, vdim) <= 0 or n_heads % n_kv_heads:
            raise ShapeError(f"differential attention: {n_heads} query heads cannot share {n_kv_heads} key heads")
        if max(dim, vdim) > 256:
            raise ShapeError(f"differential attention: heads of {dim} and {vdim} channels exceed the 256 its kernels take")
        if not 1 <= taps <= self.MAX_TAPS:
            raise ShapeError(f"short convolution: {taps} taps are outside 1..{self.MAX_TAPS}")
        if positions is None or not positions.rotates or positions.dims > dim:
            raise ShapeError("differential attention: needs a rotating position encoding over at most dim channels")
        self.width, self.n_heads, self.n_kv_heads, self.dim, self.vdim, self.taps = width, n_heads, n_kv_heads, dim, vdim, taps
        self.scale, self.offset, self.eps, self.positions = float(scale), float(offset), float(eps), positions
        self.q_width, self.k_width, self.v_width = 2 * n_heads * dim, 2 * n_kv_heads * dim, n_kv_heads * vdim
        self.proj_width = self.q_width + self.k_width + self.v_width
        self.init_std = init_std
        self.out_init_std = init_std if out_init_std is None else out_init_std

    def specs(self):
        specs = {"in.weight": TensorSpec((self.proj_width, self.width), MATRIX, ("normal", self.init_std)),
                 "in.bias": TensorSpec((self.proj_width,), VECTOR, ("normal", 0.1)),
                 "conv.weight": TensorSpec((self.proj_width, self.taps), VECTOR, ("normal", self.taps ** -0.5)),
                 "q_norm.weight": TensorSpec((self.dim,), VECTOR, ("ones",)),
                 "k_norm.weight": TensorSpec((self.dim,), VECTOR, ("ones",)),
                 "out.weight": TensorSpec((self.width, self.n_heads * self.vdim), MATRIX, ("normal", self.out_init_std))}
        for name in ("lq1", "lk1", "lq2", "lk2"):
            specs[name] = TensorSpec((self.dim,), VECTOR, ("normal", 0.1))
        return specs

    def bind(self, tensors):
        super().bind(tensors)
        self.conv_taps = self.t_conv_weight.t().contiguous()           # [taps, channels]: a tap's channels side by side
        wide = [t.to(torch.float64) for t in (self.t_lq1, self.t_lk1, self.t_lq2, self.t_lk2)]
        share = torch.exp((wide[0] * wide[1]).sum()) - torch.exp((wide[2] * wide[3]).sum()) + self.offset
        self.share = share.to(torch.float32).reshape(1).contiguous()
        self.positions.inv_freq(self.t_in_weight.device)
        # (a convolution of one tap keeps nothing: an empty state of the right shape)
        self.no_state = torch.empty((1, 0, self.proj_width), dtype=torch.float32, device=self.t_in_weight.device)

    def cache_need(self):
        states = (StateSpec("qkv_taps", (self.taps - 1, self.proj_width), torch.float32),) if self.taps > 1 else ()
        return CacheNeed(kv=KvSpec(self.n_kv_heads, 2 * self.dim + self.vdim, None, has_values=False), states=states)

    def _splits(self, ctx, n: int) -> int:
        """Blocks a token's keys are shared among: enough to fill the GPU about twice, none with fewer than 128 keys."""
        units = max(1, n * self.n_kv_heads * -(-(self.n_heads // self.n_kv_heads) // 4))
        by_fill = -(-2 * _sm_count(ctx.ws.device) // units)
        return int(max(1, min(by_fill, -(-ctx.ctx_bound // 128), kernels.MAX_SPLITS)))

    # `forward(..., store=True)` writes the result into `residual` instead of adding it (rows that hold nothing yet)
    can_store = True

    def forward(self, ctx, x, residual, entry, owns_cache=True, store=False):
        if getattr(ctx, "program", None) is not None:
            from ..engine.program import ProgramUnsupported
            raise ProgramUnsupported("differential attention has no phase in the fused step")
        if not owns_cache:
            raise ShapeError("differential attention: a layer files its own keys and values")
        mark = ctx.ws.mark()
        n, dtype, heads, groups, dim, vdim = ctx.n_tokens, ctx.dtype, self.n_heads, self.n_kv_heads, self.dim, self.vdim
        proj = ctx.ws.take((n, self.proj_width), dtype)
        linear(ctx, x, self.t_in_weight, self.t_in_bias, proj, m=n, w_is_nk=True)
        k_pool, _, group, g = ctx.cache.layer_pools(entry)
        row = 2 * dim + vdim
        if group.spec.head_dim != row or group.spec.n_kv_heads != groups or group.is_ring:
            raise ShapeError("differential attention: the cache entry does not hold this layer's rows")
        pool = k_pool.view(-1, groups, PAGE_SIZE, row)
        table = ctx.tables[g]
        tensor_cores = (dtype == torch.bfloat16 and not ctx.is_decode and ctx.max_new >= self.prompt_from
                        and kernels.two_map_attention_tcgen05_supports(dim, vdim))
        pad = dim if not tensor_cores else (64 if dim <= 64 else 128)
        q = ctx.ws.take((n, 2 * heads * pad), dtype)
        state = ctx.cache.state(entry, "qkv_taps") if self.taps > 1 else self.no_state
        kernels.differential_prep(proj, self.conv_taps, state, ctx.slots, ctx.seq_start, ctx.token_seq, ctx.positions,
                                  self.t_q_norm_weight, self.t_k_norm_weight, self.eps, self.positions.inv_freq(proj.device),
                                  self.positions.dims, self.positions.size, table, group.table_len, pool, q, n_tokens=n,
                                  n_seqs=ctx.n_seqs, max_new=ctx.max_new, n_heads=heads, n_kv_heads=groups, dim=dim, vdim=vdim)
        splits = 1 if tensor_cores else self._splits(ctx, n)
        parts = ctx.ws.take((kernels.two_map_attention_floats(n, heads, vdim, splits),), torch.float32)
        sizes = dict(n_tokens=n, n_heads=heads, n_kv_heads=groups, dim=dim, vdim=vdim, scale=self.scale)
        if tensor_cores:
            kernels.two_map_attention_tcgen05(q, pool, table, group.table_len, ctx.seq_start, ctx.past_len, parts,
                                              n_seqs=ctx.n_seqs, max_new=ctx.max_new, **sizes)
        else:
            kernels.two_map_attention(q, pool, table, group.table_len, ctx.token_seq, ctx.positions, parts, n_splits=splits,
                                      **sizes)
        mixed = ctx.ws.take((n, heads * vdim), dtype)
        kernels.differential_combine(parts, self.share, 1.0 - self.offset, self.eps, mixed, n_tokens=n, n_heads=heads,
                                     vdim=vdim, n_splits=splits)
        linear(ctx, mixed, self.t_out_weight, None, residual, m=n, residual=None if store else residual, w_is_nk=True)
        ctx.ws.release(mark)
