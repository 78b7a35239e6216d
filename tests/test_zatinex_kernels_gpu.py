"""The kernels Zatinex brought, each alone against the plain implementation's function for the same mechanism (float64), at
sizes the models of the other tests do not have: the recurrence with a decay per key channel token by token and by chunks,
the convolution with norm, rotation and filing, two maps over one value head in both forms, their join, RMS norms alone and
inside products, and output gates of one number a head in every kernel that takes a gate."""
import math

import numpy as np
import pytest
import torch

import plain_zatinex as plain
from burn_transformers_b200 import kernels
from burn_transformers_b200.parts import InterleavedRotary

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [(torch.float32, 2e-5), (torch.bfloat16, 2e-2)]
PAGE = 64


def dev(a, dtype=torch.float32):
    return torch.tensor(np.asarray(a), dtype=torch.float64).to(dtype).to(DEV)


def ints(a):
    return torch.tensor(np.asarray(a), dtype=torch.int32, device=DEV)


def host(t):
    return t.detach().double().cpu()


def rel(got, want):
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    return float(np.abs(got - want).max() / max(1e-30, np.abs(want).max()))


def starts(news):
    return ints(np.concatenate([[0], np.cumsum(news)]))


# ---- the recurrence ------------------------------------------------------------------------------------------------------

def recurrence(proj, dt, tau, heads, dim, vdim, states, q_scale):
    """Every head of one sequence through the plain recurrence: (outputs [tokens, heads, vdim], states)."""
    p, n = host(proj), proj.shape[0]
    alpha = torch.exp(-host(dt).view(n, heads, dim) / tau)
    q, k = (p[:, o:o + heads * dim].reshape(n, heads, dim) for o in (0, heads * dim))
    v = p[:, 2 * heads * dim:2 * heads * dim + heads * vdim].reshape(n, heads, vdim)
    out, last = torch.zeros(n, heads, vdim, dtype=torch.float64), states.clone()
    for h in range(heads):
        out[:, h], last[h] = plain.gated_recurrence(q[:, h] * q_scale, k[:, h], v[:, h], alpha[:, h], states[h])
    return out, last


@pytest.mark.parametrize("dtype, tol", DTYPES)
@pytest.mark.parametrize("heads, dim, vdim, tau", [(3, 16, 24, 16.0), (2, 5, 7, 1.0), (1, 64, 64, 16.0), (2, 72, 130, 4.0),
                                                   (1, 200, 40, 8.0), (1, 33, 96, 2.0)])
def test_recurrence_of_unequal_runs_with_a_state_carried_over(dtype, tol, heads, dim, vdim, tau):
    """Single tokens, short runs, runs on both sides of a group (4) and a chunk (64); slots that no sequence names keep
    their state; rows behind the step's stay as they are; with and without the norm and gate inside."""
    rng = np.random.default_rng(dim)
    state = dev(rng.standard_normal((9, heads, dim, vdim)))
    weight = dev(1.0 + 0.3 * rng.standard_normal(vdim))
    width = 2 * heads * dim + 2 * heads * vdim
    g_off = 2 * heads * dim + heads * vdim
    for news, slots in (([1], [4]), ([1, 1, 1], [3, 0, 6]), ([2, 16, 1, 9], [5, 2, 0, 3]), ([64, 3], [1, 7]),
                        ([65, 1, 66, 5], [2, 6, 5, 8]), ([131, 67, 64, 200], [0, 1, 2, 6])):
        n = sum(news)
        proj = dev(rng.standard_normal((n, width)), dtype)
        dt = dev(np.abs(rng.standard_normal((n, heads * dim))) * 2.0)
        before = host(state).clone()
        out = torch.full((n + 1, heads * vdim), 9.0, device=DEV)
        mixed = torch.full((n + 1, heads * vdim), 9.0, dtype=dtype, device=DEV)
        scratch = None
        if max(news) > kernels.GLA_CHUNK:
            scratch = torch.empty(kernels.gla_chunked_scratch_floats(n, len(news), max(news), heads, dim, vdim), device=DEV)
        done = kernels.gla_scan(proj, 0, heads * dim, 2 * heads * dim, 0.3, dt, -1.0 / tau, state, ints(slots), starts(news),
                                out[:n], n_seqs=len(news), n_heads=heads, dim=dim, vdim=vdim, max_new=max(news), scratch=scratch,
                                norm=(weight, 1e-5, g_off, mixed[:n]))
        assert done == (scratch is None and kernels.gla_scan_fuses(dim, vdim))
        assert bool((out[n:] == 9.0).all()) and bool((mixed[n:] == 9.0).all())
        at = 0
        for s, count in zip(slots, news):
            want, last = recurrence(proj[at:at + count], dt[at:at + count], tau, heads, dim, vdim, before[s], 0.3)
            if done:
                gate = plain.swish(host(proj)[at:at + count, g_off:]).reshape(want.shape)
                assert rel(host(mixed[at:at + count]).view(want.shape), plain.rms_norm(want, host(weight), 1e-5) * gate) < tol, (news, s)
            else:
                assert rel(host(out[at:at + count]).view(want.shape), want) < 3e-5, (news, s)
            assert rel(host(state[s]), last) < 3e-5, (news, s)
            at += count
        idle = [i for i in range(9) if i not in slots]
        assert torch.equal(host(state[idle]), before[idle])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_recurrence_with_decays_that_vanish_and_that_last(dtype):
    """Channels that forget everything at every token (their decays over a chunk are far below the smallest number), at some
    tokens only, slowly, and never, side by side: nothing overflows, nothing is lost, by chunks and token by token."""
    rng = np.random.default_rng(3)
    heads, dim, vdim, n = 2, 40, 24, 333
    proj = dev(rng.standard_normal((n, 2 * heads * dim + 2 * heads * vdim)), dtype)
    rates = np.zeros((n, heads, dim))
    rates[:, :, :10] = 400.0
    rates[:, :, 10:20] = np.where(rng.random((n, heads, 10)) < 0.02, 90.0, 0.01)
    rates[:, :, 20:30] = 1e-4
    dt = dev(rates.reshape(n, heads * dim))
    start = rng.standard_normal((heads, dim, vdim)) * 3.0
    want, last = recurrence(proj, dt, 1.0, heads, dim, vdim, torch.tensor(start), dim ** -0.5)
    assert float(last[:, 30:].abs().mean()) > 5.0 and bool(torch.isfinite(want).all())
    results = []
    for size in (n, 64, 65, 2, 1):
        state, out = dev(start[None]), torch.zeros((n, heads * vdim), device=DEV)
        for lo in range(0, n, size):
            m = min(size, n - lo)
            scratch = torch.empty(kernels.gla_chunked_scratch_floats(m, 1, m, heads, dim, vdim), device=DEV) if m > 64 else None
            kernels.gla_scan(proj[lo:lo + m], 0, heads * dim, 2 * heads * dim, dim ** -0.5, dt[lo:lo + m], -1.0, state, ints([0]),
                             ints([0, m]), out[lo:lo + m], n_seqs=1, n_heads=heads, dim=dim, vdim=vdim, max_new=m, scratch=scratch)
        assert rel(host(out).view(want.shape), want) < 3e-5 and rel(host(state)[0], last) < 3e-5, size
        results.append(host(out))
    assert all(rel(r, results[0]) < 2e-5 for r in results)


@pytest.mark.parametrize("dtype, tol", DTYPES)
def test_logarithms_of_decays(dtype, tol):
    """-softplus(-z) from low-rank rows with the weights negated is the logarithm of sigmoid(z), also far out."""
    rng = np.random.default_rng(2)
    n, channels, rank = 37, 90, 5
    low, w, b = dev(rng.standard_normal((n, rank + 3)), dtype), dev(rng.standard_normal((channels, rank)) * 6.0), dev(rng.standard_normal(channels))
    b[0], b[1] = 120.0, -120.0
    dt = torch.zeros((n, channels), device=DEV)
    kernels.selective_scan_dt(low[:, 2:2 + rank], -w, -b, dt, n_tokens=n)
    z = host(low)[:, 2:2 + rank] @ host(w).T + host(b)
    want = -torch.nn.functional.logsigmoid(z)
    assert float(((host(dt) - want).abs() / (1e-6 + want.abs())).max()) < 1e-4 or rel(host(dt), want) < 1e-6
    assert float(host(dt).min()) >= 0.0


# ---- convolution, norm, rotation, filing -----------------------------------------------------------------------------------

class Tables:
    """Scattered pages for sequences of the given lengths."""

    def __init__(self, lens, kv_heads, row, dtype, seed=7):
        self.width = -(-max(lens) // PAGE)
        self.order = np.random.default_rng(seed).permutation(len(lens) * self.width).reshape(len(lens), self.width)
        self.pages = ints(self.order)
        self.pool = torch.zeros((len(lens) * self.width, kv_heads, PAGE, row), dtype=dtype, device=DEV)

    def rows(self, s, length):
        """[length, kv_heads, row] of sequence s, float64 on the host."""
        pool = host(self.pool)
        return torch.stack([pool[self.order[s, j // PAGE], :, j % PAGE] for j in range(length)])


@pytest.mark.parametrize("dtype, tol", DTYPES)
@pytest.mark.parametrize("heads, groups, dim, vdim, taps, rot, scaling, normed, pad", [
    (4, 2, 16, 24, 4, 8, None, True, 16), (3, 3, 9, 7, 6, 4, None, True, 12), (6, 1, 64, 128, 3, 64, (8.0, 100.0, 16.0, 0.5), True, 64),
    (2, 2, 72, 40, 2, 72, None, True, 128), (5, 5, 6, 3, 1, 0, None, True, 6), (2, 1, 200, 250, 4, 130, None, False, 200)])
def test_convolution_norm_rotation_and_filing(dtype, tol, heads, groups, dim, vdim, taps, rot, scaling, normed, pad):
    """Three steps on the same slots (a prompt, portions shorter than the taps' reach, single tokens) against whole sequences
    through the plain functions; the state afterwards is the last projected rows; other slots are untouched."""
    rng = np.random.default_rng(dim)
    q_w, k_w = 2 * heads * dim, 2 * groups * dim
    channels = q_w + k_w + groups * vdim
    positions = InterleavedRotary(rot, 50.0, yarn=scaling)
    conv = rng.standard_normal((channels, taps))
    gains = [1.0 + 0.4 * rng.standard_normal(dim) for _ in range(2)]
    lens, slots = [75, 9, 30], [4, 0, 2]
    whole = [dev(rng.standard_normal((n, channels)), dtype) for n in lens]
    t = Tables(lens, groups, 2 * dim + vdim, dtype)
    state = torch.zeros((6, max(1, taps - 1), channels), device=DEV)
    state[5] = 3.0
    got_q = [[] for _ in lens]
    done = [0, 0, 0]
    for news in ([70, 3, 1], [2, 1, 26], [1, 1, 1], [1, 2, 1], [1, 2, 1]):
        n = sum(news)
        proj = torch.cat([w[d:d + c] for w, d, c in zip(whole, done, news)]).contiguous()
        q_out = torch.full((n + 1, 2 * heads * pad), 9.0, dtype=dtype, device=DEV)
        token_seq = ints(np.repeat(range(3), news))
        place = ints(np.concatenate([np.arange(d, d + c) for d, c in zip(done, news)]))
        kernels.differential_prep(proj, dev(np.ascontiguousarray(conv.T)), state if taps > 1 else state[:, :0], ints(slots), starts(news), token_seq, place,
                                  dev(gains[0]) if normed else None, dev(gains[1]) if normed else None, 1e-4,
                                  positions.inv_freq(DEV), rot, positions.size, t.pages, t.width, t.pool, q_out[:n], n_tokens=n,
                                  n_seqs=3, max_new=max(news), n_heads=heads, n_kv_heads=groups, dim=dim, vdim=vdim)
        assert bool((q_out[n] == 9.0).all())
        at = 0
        for s, c in enumerate(news):
            got_q[s].append(host(q_out[at:at + c]).view(c, 2 * heads, pad))
            at += c
            done[s] += c
    rot_cfg = {"dims": rot, "base": 50.0}
    if scaling:
        rot_cfg["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    for s, n in enumerate(done):
        assert n == lens[s]
        u = plain.short_convolution(host(whole[s]), torch.tensor(conv))
        q, k, v = u[:, :q_w].reshape(n, 2 * heads, dim), u[:, q_w:q_w + k_w].reshape(n, 2 * groups, dim), u[:, q_w + k_w:]
        if normed:
            q, k = (plain.rms_norm(x, torch.tensor(g), 1e-4) for x, g in zip((q, k), gains))
        q, k = (plain.rotate_neighbours(x, torch.arange(n), rot_cfg) for x in (q, k))
        got = torch.cat(got_q[s])
        assert rel(got[..., :dim], q) < tol and not bool(got[..., dim:].any())
        rows = t.rows(s, n)
        assert rel(rows[..., :2 * dim].reshape(n, 2 * groups, dim), k) < tol
        assert rel(rows[..., 2 * dim:].reshape(n, -1), v) < tol
        if taps > 1:
            assert torch.equal(host(state[slots[s]]), host(whole[s])[n - taps + 1:])
    assert bool((state[5] == 3.0).all()) and not bool(state[1].any())


# ---- two maps ----------------------------------------------------------------------------------------------------------------

def two_maps(q, rows, past, scale, dim, heads):
    """[new tokens, 2 heads, vdim] of one sequence: q [new, 2 heads, dim], rows [length, groups, 2 dim + vdim]."""
    n, groups = q.shape[0], rows.shape[1]
    seen = torch.ones(rows.shape[0], rows.shape[0]).tril().bool()[past:past + n]
    out = []
    for i in range(2 * heads):
        g, m = (i // 2) // (heads // groups), i % 2
        scores = q[:, i] @ rows[:, g, m * dim:(m + 1) * dim].T * scale
        out.append(torch.softmax(scores.masked_fill(~seen, float("-inf")), -1) @ rows[:, g, 2 * dim:])
    return torch.stack(out, 1)


CASES = [([0], [200]), ([0, 0, 0], [130, 33, 257]), ([64, 63, 300, 0], [1, 1, 1, 1]), ([100, 7, 64], [70, 40, 128]),
         ([31, 127], [2, 130])]


@pytest.mark.parametrize("impl", ["float32", "bfloat16", "tcgen05"])
@pytest.mark.parametrize("heads, groups, dim, vdim", [(4, 2, 16, 24), (3, 3, 64, 64), (6, 1, 64, 128), (5, 1, 9, 7), (2, 2, 72, 40),
                                                      (4, 1, 128, 128), (8, 2, 8, 8), (1, 1, 136, 200), (2, 1, 120, 72)])
def test_two_maps_over_scattered_pages(impl, heads, groups, dim, vdim):
    """Prompts, portions that continue, single tokens; keys at every page's and tile's border that stand out in one map
    only; rows of pages past a sequence's end hold large numbers that must not count; one split and several."""
    dtype = torch.float32 if impl == "float32" else torch.bfloat16
    tol = 2e-5 if impl == "float32" else 2e-2
    if impl == "tcgen05":
        assert kernels.two_map_attention_tcgen05_supports(dim, vdim) == (dim % 8 == 0 and vdim % 8 == 0 and max(dim, vdim) <= 128)
        if not kernels.two_map_attention_tcgen05_supports(dim, vdim):
            return
    pad = dim if impl != "tcgen05" else 64 if dim <= 64 else 128
    rng = np.random.default_rng(dim + heads)
    scale = 1.5 / math.sqrt(dim)
    for pasts, news in CASES:
        lens = [p + n for p, n in zip(pasts, news)]
        t = Tables(lens, groups, 2 * dim + vdim, dtype)
        t.pool.fill_(50.0)
        stored = []
        for s, length in enumerate(lens):
            rows = rng.standard_normal((length, groups, 2 * dim + vdim))
            for j in (0, 63, 64, 127, 128, length - 1):
                if j < length:
                    rows[j, :, (j % 2) * dim:(j % 2 + 1) * dim] *= 3.0
            rows = dev(rows, dtype)
            stored.append(host(rows))
            for j in range(length):
                t.pool[int(t.order[s, j // PAGE]), :, j % PAGE] = rows[j]
        n = sum(news)
        q = torch.zeros((n, 2 * heads, pad), dtype=dtype, device=DEV)
        q[..., :dim] = dev(rng.standard_normal((n, 2 * heads, dim)), dtype)
        q = q.view(n, -1)
        token_seq = ints(np.repeat(range(len(news)), news))
        place = ints(np.concatenate([np.arange(p, p + c) for p, c in zip(pasts, news)]))
        for splits in (1, 2, 7) if impl != "tcgen05" else (1,):
            out = torch.full((kernels.two_map_attention_floats(n, heads, vdim, splits) + 4,), 9.0, device=DEV)
            sizes = dict(n_tokens=n, n_heads=heads, n_kv_heads=groups, dim=dim, vdim=vdim, scale=scale)
            if impl == "tcgen05":
                kernels.two_map_attention_tcgen05(q, t.pool, t.pages, t.width, starts(news), ints(pasts), out, n_seqs=len(news),
                                                  max_new=max(news), **sizes)
                kernels.check_status(torch.device(DEV))
            else:
                kernels.two_map_attention(q, t.pool, t.pages, t.width, token_seq, place, out, n_splits=splits, **sizes)
            assert bool((out[-4:] == 9.0).all())
            parts = host(out[:-4])
            if splits > 1:
                parts = parts.view(n, 2 * heads, splits, vdim + 2)
                share = torch.exp(parts[..., vdim] - parts[..., vdim].max(-1, keepdim=True).values)
                got = (parts[..., :vdim] * share[..., None]).sum(2) / (parts[..., vdim + 1] * share).sum(2)[..., None]
            else:
                got = parts.view(n, 2 * heads, vdim)
            at = 0
            for s, c in enumerate(news):
                want = two_maps(host(q[at:at + c]).view(c, 2 * heads, pad)[..., :dim], stored[s], pasts[s], scale, dim, heads)
                assert np.abs(np.asarray(got[at:at + c] - want)).max() < tol * max(0.3, float(want.abs().max())), (pasts, news, splits, s)
                at += c


@pytest.mark.parametrize("dtype, tol", [(torch.float32, 1e-5), (torch.bfloat16, 6e-3)])
@pytest.mark.parametrize("heads, vdim, splits", [(3, 24, 1), (5, 7, 1), (1, 128, 3), (4, 200, 64), (2, 64, 33), (6, 100, 2)])
def test_maps_joined_subtracted_and_normed(dtype, tol, heads, vdim, splits):
    rng = np.random.default_rng(vdim)
    n, gain, eps = 13, 0.35, 1e-3
    share = dev([0.8])
    results = rng.standard_normal((n, 2 * heads, splits, vdim))
    tops, sums = 5.0 * rng.standard_normal((n, 2 * heads, splits)), 0.5 + rng.random((n, 2 * heads, splits))
    if splits > 1:
        tops[:, :, -1], sums[:, :, -1], results[:, :, -1] = -np.inf, 0.0, 0.0        # (a split that holds no key)
        parts = dev(np.concatenate([results, tops[..., None], sums[..., None]], -1))
        weight = np.exp(tops - tops.max(-1, keepdims=True))
        merged = (results * weight[..., None]).sum(2) / (sums * weight).sum(2)[..., None]
    else:
        parts, merged = dev(results), results[:, :, 0]
    a = torch.tensor(merged).view(n, heads, 2, vdim)
    want = plain.combine_maps(a[:, :, 0], a[:, :, 1], 0.8, 1.0 - gain, eps)
    out = torch.full((n + 1, heads * vdim), 9.0, dtype=dtype, device=DEV)
    kernels.differential_combine(parts.contiguous().view(-1), share, gain, eps, out, n_tokens=n, n_heads=heads, vdim=vdim, n_splits=splits)
    assert rel(host(out[:n]).view(want.shape), want) < tol and bool((out[n] == 9.0).all())


# ---- norms -------------------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("x_type, out_type", [(torch.float32, torch.bfloat16), (torch.bfloat16, torch.bfloat16),
                                              (torch.float32, torch.float32)])
@pytest.mark.parametrize("width, groups", [(24, 1), (64, 5), (7, 3), (128, 2), (320, 1), (384, 3), (768, 1), (770, 1), (1000, 1),
                                           (1024, 1), (1300, 1)])
def test_norm_alone_and_with_a_gate(x_type, out_type, width, groups):
    rng = np.random.default_rng(width)
    n, full = 11, width * groups
    x = dev(rng.standard_normal((n + 1, full + 8)), x_type)[:, 4:4 + full]
    weight, gate = dev(rng.standard_normal(full)), dev(rng.standard_normal((n, full)), out_type)
    for rule in (None, "sigmoid", "swish"):
        out = torch.full((n + 1, full), 9.0, dtype=out_type, device=DEV)
        kernels.rmsnorm(x, weight, out, 1e-2, n_rows=n, groups=groups, **({} if rule is None else {"gate": gate, "gate_rule": rule}))
        want = plain.rms_divide(host(x[:n]).reshape(n, groups, width), 1e-2).reshape(n, full) * host(weight)
        if rule is not None:
            want = want * (plain.sigmoid if rule == "sigmoid" else plain.swish)(host(gate))
        assert rel(host(out[:n]), want) < (1e-5 if out_type == torch.float32 else 1e-2) and bool((out[n] == 9.0).all())


@pytest.mark.parametrize("rows", [1, 3, 8, 9, 16])
@pytest.mark.parametrize("n, k", [(96, 64), (264, 768), (8200, 256)])
def test_norm_inside_a_product(rows, n, k):
    """Rows with a mean far from zero (a norm that took it off would show), picked by an index."""
    rng = np.random.default_rng(rows + k)
    x, gain = dev(rng.standard_normal((20, k)) + 2.0), dev(1.0 + 0.3 * rng.standard_normal(k))
    w, index = dev(rng.standard_normal((n, k)) * k ** -0.5, torch.bfloat16), ints(rng.permutation(20)[:rows])
    want = plain.rms_norm(host(x)[index.cpu().long()], host(gain), 1e-3) @ host(w).T
    norm = (x, gain, None, 1e-3, index)
    out = torch.full((rows + 1, n), 9.0, device=DEV)
    assert kernels.linear_skinny_supports(rows, n, k, True, True)
    kernels.linear_skinny(None, w, None, out, m=rows, w_is_nk=True, norm=norm, rms=True)
    assert rel(host(out[:rows]), want) < 1e-2 and bool((out[rows] == 9.0).all())
    if kernels.linear_stream_supports(rows, n, k, True):
        out.fill_(9.0)
        kernels.linear_stream(None, w, None, out, m=rows, norm=norm, rms=True)
        assert rel(host(out[:rows]), want) < 1e-2 and bool((out[rows] == 9.0).all())
    else:
        assert n < 8192


# ---- gates of one number a head --------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype, tol", DTYPES)
@pytest.mark.parametrize("heads, k, n", [(3, 48, 24), (6, 40, 128), (5, 9, 7), (1, 64, 8)])
def test_products_per_head_with_one_gate_a_head(dtype, tol, heads, k, n):
    rng = np.random.default_rng(k)
    tokens = 70
    a, w = dev(rng.standard_normal((tokens, heads, k)), dtype), dev(rng.standard_normal((heads, k, n)) * k ** -0.5, dtype)
    rows = dev(rng.standard_normal((tokens, heads + 5)) * 2.0, dtype)
    gate = rows[:, 3:3 + heads].unsqueeze(2).expand(tokens, heads, n)
    want = torch.einsum("thk,hkn->thn", host(a), host(w)) * plain.sigmoid(host(rows)[:, 3:3 + heads, None])
    for tensor_cores in (True, False):
        out = torch.zeros((tokens, heads, n), dtype=dtype, device=DEV)
        kernels.head_linear(a, w, out, n_tokens=tokens, gate=gate, tensor_cores=tensor_cores)
        assert rel(host(out), want) < tol
    mixed = torch.zeros((tokens, heads * n), dtype=dtype, device=DEV)
    kernels.latent_decode_finish(w, mixed, n_tokens=tokens, n_splits=1, mixed_latent=a.view(tokens, heads * k), gate=rows[:, 3:3 + heads])
    assert rel(host(mixed).view(tokens, heads, n), want) < tol


@pytest.mark.parametrize("impl", ["mma", "tcgen05"])
@pytest.mark.parametrize("heads, dq, dv", [(3, 40, 24), (2, 96, 64), (5, 72, 56), (4, 128, 128)])
def test_prompt_attention_with_one_gate_a_head(impl, heads, dq, dv):
    rng = np.random.default_rng(dq)
    news = [200, 1, 70]
    n = sum(news)
    q = dev(rng.standard_normal((n, heads, dq)), torch.bfloat16)
    k, v = (dev(rng.standard_normal((heads, n, d)), torch.bfloat16).transpose(0, 1) for d in (dq, dv))
    rows = dev(rng.standard_normal((n, heads + 3)) * 2.0, torch.bfloat16)
    gate = rows[:, 1:1 + heads].unsqueeze(2).expand(n, heads, dv)
    out = torch.full((n + 1, heads, dv), 9.0, dtype=torch.bfloat16, device=DEV)
    assert kernels.sink_attention_supports(q, k, v, gate, out[:n]) and kernels.sink_attention_tcgen05_supports(q, k, v, gate, out[:n])
    scale = 1.0 / math.sqrt(dq)
    kernels.sink_attention(q, k, v, out[:n], starts(news), n_seqs=3, max_new=200, scale=scale, gate=gate, past_len=ints([0, 0, 0]), impl=impl)
    kernels.check_status(torch.device(DEV))
    assert bool((out[n] == 9.0).all())
    at = 0
    for c in news:
        for h in range(heads):
            want = plain.causal_softmax(host(q[at:at + c, h]) @ host(k[at:at + c, h]).T * scale) @ host(v[at:at + c, h])
            want = want * plain.sigmoid(host(rows)[at:at + c, 1 + h:2 + h])
            assert np.abs(np.asarray(host(out[at:at + c, h]) - want)).max() < 2e-2 * max(0.3, float(want.abs().max()))
        at += c
