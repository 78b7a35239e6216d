"""The kernels Visadra brought, each alone against the plain implementation's function for the same mechanism (float64), at
sizes the models of the other tests do not have: the gated average token by token and scanned by clusters of blocks with
runs on both sides of every length a warp, a block and a cluster hold, the router whose weights are a softmax over the
chosen, the x sigmoid(x) rule of a gated feed-forward, and attention with a sink and no gate in every form."""
import math

import numpy as np
import pytest
import torch

import plain_visadra as plain
from burn_transformers_b200 import kernels
from burn_transformers_b200.parts import RmsNorm

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


def average_case(rng, width, news, dtype, shift=0.0):
    """Projections [g | a | x] of a step, biases, and what the plain functions make of them."""
    n = sum(news)
    proj = dev(rng.standard_normal((n, 3 * width)) * 2.0, dtype)
    zb, xb = dev(rng.standard_normal(width) + shift), dev(rng.standard_normal(width))
    p = host(proj)
    z = plain.sigmoid(p[:, width:2 * width] + host(zb))
    values = plain.candidate(p[:, 2 * width:] + host(xb))
    return proj, zb, xb, z, values, plain.swish(p[:, :width])


@pytest.mark.parametrize("dtype, tol", DTYPES)
@pytest.mark.parametrize("width", [1, 7, 64, 70, 130, 1104])
def test_gated_average_of_unequal_runs_with_a_state_carried_over(dtype, tol, width):
    """Several steps on the same slots: single tokens, short runs, runs at and beside what a warp (8 tokens), a block
    (64) and a cluster (up to 512) hold, and some that go round the cluster's loop; slots that no sequence names
    keep their state, rows behind the step's stay as they are."""
    rng = np.random.default_rng(width)
    state = dev(rng.standard_normal((9, width)))
    for news, slots in (([1], [4]), ([1, 1, 1, 1, 1], [3, 0, 6, 1, 8]), ([2, 16, 1, 9], [5, 2, 0, 3]), ([17, 1, 8, 128], [1, 7, 4, 0]),
                        ([129, 63, 3], [2, 6, 5]), ([65, 64, 24], [6, 5, 7]), ([513, 1, 512, 1025], [0, 1, 2, 6]), ([130, 2300], [8, 3])):
        proj, zb, xb, z, values, gate = average_case(rng, width, news, dtype)
        before = host(state).clone()
        n = sum(news)
        out = torch.full((n + 1, width), 9.0, dtype=dtype, device=DEV)
        kernels.min_gru(proj, width, 2 * width, 0, zb, xb, state, ints(slots), ints(np.concatenate([[0], np.cumsum(news)])), out[:n],
                        n_seqs=len(news), max_new=max(news))
        assert bool((out[n:] == 9.0).all())
        at = 0
        for s, count in zip(slots, news):
            states, last = plain.gated_average(z[at:at + count], values[at:at + count], before[s])
            assert rel(host(out[at:at + count]), states * gate[at:at + count]) < tol, (news, s)
            assert rel(host(state[s]), last) < 2e-5, (news, s)
            at += count
        idle = [i for i in range(9) if i not in slots]
        assert torch.equal(host(state[idle]), before[idle])


@pytest.mark.parametrize("count", [40, 1500])
def test_gated_average_keeps_a_state_for_long_and_drops_it_at_once(count):
    """Gates near zero: the state a run starts from is still there at its end, after every composition of maps.  Gates
    that saturate either way give exactly what was there or exactly the value."""
    rng = np.random.default_rng(3)
    width = 66
    proj = np.zeros((count, 3 * width))
    proj[:, width:2 * width] = -9.0 + 0.5 * rng.standard_normal((count, width))
    proj[:, :width] = 3.0
    proj[:, 2 * width:] = rng.standard_normal((count, width))
    proj[:, width] = -200.0                      # channel 0 never moves, channel 1 takes every value whole
    proj[:, width + 1] = 200.0
    zero = dev(np.zeros(width))
    state = dev(100.0 + rng.standard_normal((1, width)))
    before = host(state)[0]
    p = dev(proj)
    out = torch.zeros((count, width), device=DEV)
    kernels.min_gru(p, width, 2 * width, 0, zero, zero, state, ints([0]), ints([0, count]), out, n_seqs=1, max_new=count)
    z, values = plain.sigmoid(host(p)[:, width:2 * width]), plain.candidate(host(p)[:, 2 * width:])
    states, last = plain.gated_average(z, values, before)
    assert float(last[2:].min()) > 60.0
    assert rel(host(state)[0], last) < 2e-5 and rel(host(out), states * plain.swish(host(p)[:, :width])) < 2e-5
    assert float(host(state)[0, 0]) == float(before[0])
    assert abs(float(host(state)[0, 1]) - float(values[-1, 1])) < 1e-6


def test_gated_average_does_not_depend_on_how_a_run_is_cut():
    rng = np.random.default_rng(5)
    width, n = 90, 700
    proj, zb, xb, _, _, _ = average_case(rng, width, [n], torch.float32)
    whole = torch.zeros((n, width), device=DEV)
    kept = dev(np.zeros((1, width)))
    kernels.min_gru(proj, width, 2 * width, 0, zb, xb, kept, ints([0]), ints([0, n]), whole, n_seqs=1, max_new=n)
    for size in (1, 2, 15, 64, 333):
        state = dev(np.zeros((1, width)))
        out = torch.zeros((n, width), device=DEV)
        for lo in range(0, n, size):
            m = min(size, n - lo)
            kernels.min_gru(proj[lo:lo + m], width, 2 * width, 0, zb, xb, state, ints([0]), ints([0, m]), out[lo:lo + m], n_seqs=1,
                            max_new=m)
        assert rel(host(out), host(whole)) < 1e-6 and rel(host(state), host(kept)) < 1e-6


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts, top, width", [(6, 2, 50), (1, 1, 64), (7, 7, 72), (40, 6, 128), (33, 32, 96), (5, 1, 33)])
def test_router_with_a_softmax_over_the_chosen(dtype, experts, top, width):
    rng = np.random.default_rng(experts * 10 + top)
    tokens = 77
    x, router = dev(rng.standard_normal((tokens, width)), dtype), dev(rng.standard_normal((experts, width)) * 0.3, dtype)
    bias = dev(rng.standard_normal(experts) * 2.0)
    ids = torch.full((tokens + 1, top), -1, dtype=torch.int32, device=DEV)
    weights = torch.full((tokens + 1, top), 9.0, device=DEV)
    kernels.moe_route(x, router, ids, weights, n_tokens=tokens, top=top, rule="softmax_of_chosen", logit_bias=bias)
    assert bool((ids[tokens] == -1).all()) and bool((weights[tokens] == 9.0).all())
    numbers = host(x) @ host(router).T + host(bias)
    ranked = numbers.sort(-1, descending=True).values
    gap = (ranked[:, :-1] - ranked[:, 1:])[:, :top].min(-1).values if experts > 1 else torch.ones(tokens)
    sure = gap > 1e-4                 # (a choice between two nearly equal numbers proves nothing)
    assert int(sure.sum()) > 0.8 * tokens
    for t in torch.nonzero(sure).flatten().tolist():
        best = numbers[t].topk(top)
        assert ids[t].tolist() == best.indices.tolist()
        np.testing.assert_allclose(host(weights[t]), torch.softmax(best.values, 0), rtol=1e-4, atol=1e-6)
    np.testing.assert_allclose(host(weights[:tokens]).sum(-1), 1.0, rtol=1e-5)


@pytest.mark.parametrize("dtype, tol", DTYPES)
@pytest.mark.parametrize("tokens, width, inner, experts, top", [(150, 64, 48, 6, 2), (9, 40, 24, 12, 4), (70, 72, 20, 3, 3)])
def test_gated_experts_with_the_plain_pair_rule(dtype, tol, tokens, width, inner, experts, top):
    """Route, sort, both products and the weighted sum against the plain implementation; and the rule alone."""
    rng = np.random.default_rng(tokens)
    x = dev(rng.standard_normal((tokens, width)), dtype)
    router, bias = dev(rng.standard_normal((experts, width)) * 0.5, dtype), dev(rng.standard_normal(experts))
    w_in = dev(rng.standard_normal((experts, 2 * inner, width)) * width ** -0.5, dtype)
    w_out = dev(rng.standard_normal((experts, width, inner)) * inner ** -0.5, dtype)
    ids, weights = torch.zeros((tokens, top), dtype=torch.int32, device=DEV), torch.zeros((tokens, top), device=DEV)
    kernels.moe_route(x, router, ids, weights, n_tokens=tokens, top=top, rule="softmax_of_chosen", logit_bias=bias)
    pairs = tokens * top
    offsets, tile_first = (torch.zeros(experts + 1, dtype=torch.int32, device=DEV) for _ in range(2))
    order, place = (torch.zeros(pairs, dtype=torch.int32, device=DEV) for _ in range(2))
    kernels.moe_sort(ids, offsets, tile_first, order, place, pairs=pairs, n_experts=experts)
    hidden = torch.zeros((pairs, inner), dtype=dtype, device=DEV)
    kernels.moe_expert(True, x, w_in, hidden, offsets, tile_first, order, None, pairs=pairs, top=top, activation="swish")
    part = torch.zeros((pairs, width), device=DEV)
    kernels.moe_expert(False, hidden, w_out, part, offsets, tile_first, order, weights, pairs=pairs, top=top)
    out = torch.zeros((tokens, width), device=DEV)
    kernels.moe_combine(part, place, out, n_tokens=tokens, top=top)
    w = {"router": host(router), "router.b": host(bias)}
    for e in range(experts):
        w.update({f"e{e}.gate": host(w_in[e, :inner]), f"e{e}.up": host(w_in[e, inner:]), f"e{e}.down": host(w_out[e])})
    want = plain.routed_experts(host(x), w, {"router": {"experts": experts, "top": top}})
    numbers = host(x) @ host(router).T + host(bias)
    ranked = numbers.sort(-1, descending=True).values
    sure = (ranked[:, top - 1] - ranked[:, top]) > 1e-4 if top < experts else torch.ones(tokens, dtype=torch.bool)
    assert int(sure.sum()) > 0.8 * tokens
    assert rel(host(out)[sure], want[sure]) < tol
    for width_of in (24, 20):
        both = dev(rng.standard_normal((7, 2 * width_of)) * 2.5, dtype)
        got = torch.zeros((7, width_of), dtype=dtype, device=DEV)
        kernels.gated_activation(both, got, n_rows=7, activation="swish")
        assert rel(host(got), plain.swish(host(both)[:, :width_of]) * host(both)[:, width_of:]) < tol


def test_one_number_scales_all_channels():
    norm = RmsNorm(70, 1e-3, one_gain=True)
    norm.bind({"weight": torch.tensor(-1.7, device=DEV)})
    rng = np.random.default_rng(1)
    x, stream = dev(rng.standard_normal((5, 70)) * 0.05), dev(rng.standard_normal((5, 70)))
    want = host(stream) + plain.norm_one_gain(host(x), torch.tensor(-1.7, dtype=torch.float64), 1e-3)
    kernels.rmsnorm_add(x, norm.t_weight, stream, norm.eps, n_rows=5)
    assert rel(host(stream), want) < 1e-5


def latent_rows(rng, lens, rank, rot, pages, n_pages, dtype):
    pool = torch.zeros((n_pages, PAGE, rank + rot), dtype=dtype, device=DEV)
    stored = []
    for s, length in enumerate(lens):
        rows = dev(rng.standard_normal((length, rank + rot)), dtype)
        stored.append(host(rows))
        for j in range(length):
            pool[int(pages[s, j // PAGE]), j % PAGE] = rows[j]
    return pool, stored


@pytest.mark.parametrize("dtype, tol", DTYPES)
@pytest.mark.parametrize("tensor_cores", [False, True])
@pytest.mark.parametrize("heads, rank, rot, splits", [(3, 48, 8, 1), (6, 160, 16, 3), (2, 40, 0, 2), (5, 512, 16, 4), (1, 20, 6, 1)])
def test_latent_attention_with_a_sink(dtype, tol, tensor_cores, heads, rank, rot, splits):
    """Portions that continue a sequence and single tokens over scattered pages; sinks that take nearly everything and
    sinks that take nothing; the sink counts once however many runs the keys are cut into."""
    rng = np.random.default_rng(rank)
    dk = rank + rot
    scale = 2.0 / math.sqrt(dk)
    sink = dev(np.linspace(-6.0, 7.0, heads) if heads > 1 else [1.5])
    for pasts, news in (([0, 0], [150, 2]), ([64, 63, 300, 0], [1, 1, 1, 1]), ([100, 7], [70, 40])):
        lens = [p + n for p, n in zip(pasts, news)]
        width = -(-max(lens) // PAGE)
        order = np.random.default_rng(7).permutation(len(news) * width).reshape(len(news), width)
        pages, n_pages = ints(order), len(news) * width
        pool, stored = latent_rows(rng, lens, rank, rot, pages, n_pages, dtype)
        n = sum(news)
        q = dev(rng.standard_normal((n, heads * dk)), dtype)
        out = torch.full((n + 1, heads * rank), 9.0, dtype=dtype, device=DEV)
        scratch = None
        if splits > 1:
            scratch = torch.zeros(kernels.latent_attention_scratch_floats(n, heads, rank, splits), device=DEV)
        kernels.latent_attention(q, out, pool, pages, width, ints(np.concatenate([[0], np.cumsum(news)])), ints(pasts), n_tokens=n,
                                 n_seqs=len(news), max_new=max(news), n_heads=heads, rank=rank, rot=rot, scale=scale, sink=sink,
                                 n_splits=splits, scratch=scratch, tensor_cores=tensor_cores)
        assert bool((out[n:] == 9.0).all())
        at = 0
        for s, count in enumerate(news):
            rows = stored[s]
            seen = torch.ones(lens[s], lens[s]).tril().bool()[pasts[s]:]
            got = host(out[at:at + count]).view(count, heads, rank)
            for h in range(heads):
                scores = host(q[at:at + count]).view(count, heads, dk)[:, h] @ rows.T * scale
                want = plain.softmax_beside_a_sink(scores, seen, host(sink)[h]) @ rows[:, :rank]
                assert np.abs(np.asarray(got[:, h] - want)).max() < tol * max(0.2, float(want.abs().max())), (pasts, news, s, h)
            at += count


@pytest.mark.parametrize("impl", ["mma", "tcgen05"])
@pytest.mark.parametrize("window, gated", [(0, False), (0, True), (70, False)])
@pytest.mark.parametrize("heads, dq, dv", [(3, 40, 24), (2, 96, 64), (4, 128, 128), (5, 72, 56), (1, 264, 16), (2, 64, 104),
                                           (7, 8, 8), (3, 120, 72)])
def test_attention_of_fresh_prompts_with_a_sink(impl, window, gated, heads, dq, dv):
    """Both kernels for prompts that start a sequence, keys and values head by head in memory: head sizes that fill the
    tcgen05 kernel's boxes of 64 channels and that do not (what lies beyond a head must not count), several tiles of 128
    keys, sinks that take nearly everything and nothing, a gate and a window or none."""
    rng = np.random.default_rng(dq)
    news = [200, 1, 70, 129, 300]
    n = sum(news)
    # (queries inside longer rows, as a projection leaves them; a large number right behind the last head's channels)
    rows = dev(rng.standard_normal((n, heads * dq + heads * dv + 8)), torch.bfloat16)
    rows[:, heads * (dq + dv):] = 1e4
    q = rows[:, :heads * dq].view(n, heads, dq) if heads * dq else None
    gate = rows[:, heads * dq:heads * (dq + dv)].view(n, heads, dv) if gated else None
    k, v = (dev(rng.standard_normal((heads, n, d)), torch.bfloat16).transpose(0, 1) for d in (dq, dv))
    out = torch.full((n + 1, heads, dv), 9.0, dtype=torch.bfloat16, device=DEV)
    takes = kernels.sink_attention_tcgen05_supports(q, k, v, gate, out[:n])
    assert takes == (dq <= 128) and kernels.sink_attention_supports(q, k, v, gate, out[:n])
    if impl == "tcgen05" and not takes:
        return
    sink = dev(np.linspace(-5.0, 6.0, heads) if heads > 1 else [0.7])
    scale = 1.5 / math.sqrt(dq)
    kernels.sink_attention(q, k, v, out[:n], ints(np.concatenate([[0], np.cumsum(news)])), n_seqs=len(news), max_new=max(news),
                           scale=scale, sink=sink, gate=gate, window=window, past_len=ints([0] * len(news)), impl=impl)
    kernels.check_status(torch.device(DEV))
    assert bool((out[n] == 9.0).all())
    at = 0
    for count in news:
        seen = torch.ones(count, count).tril().bool()
        if window:
            seen &= ~torch.ones(count, count).tril(-window).bool()
        for h in range(heads):
            scores = host(q[at:at + count, h]) @ host(k[at:at + count, h]).T * scale
            want = plain.softmax_beside_a_sink(scores, seen, host(sink)[h]) @ host(v[at:at + count, h])
            if gated:
                want = want * plain.sigmoid(host(gate[at:at + count, h]))
            assert np.abs(np.asarray(host(out[at:at + count, h]) - want)).max() < 2e-2 * max(0.3, float(want.abs().max())), (count, h)
        at += count


@pytest.mark.parametrize("width", [70, 64, 516, 1000, 2000, 3000, 4096, 4100, 5000])
@pytest.mark.parametrize("top, extra", [(0, False), (0, True), (3, False), (1, True), (6, True)])
def test_norm_added_over_gathered_rows(width, top, extra):
    """A token's rows gathered by place and summed with the shared expert's, normed, added to the stream, and handed on
    as they are, normed, or not at all; rows behind the last stay as they are."""
    rng = np.random.default_rng(width + top)
    n, eps = 9, 1e-3
    rows = n * max(1, top)
    x, stream = dev(rng.standard_normal((rows, width))), dev(rng.standard_normal((n + 1, width)))
    weight, after = dev(rng.standard_normal(width)), dev(rng.standard_normal(width))
    more = dev(rng.standard_normal((n, width))) if extra else None
    order = rng.permutation(rows)
    before = host(stream).clone()
    value = host(x)[torch.tensor(order)].view(n, -1, width).sum(1) if top else host(x)
    if extra:
        value = value + host(more)
    want = before[:n] + 0.7 * plain.rms_divide(value, eps) * host(weight)
    gathered = dict(place=ints(order), top=top) if top else {}
    for next_weight, next_dtype in ((None, None), (None, torch.bfloat16), (after, torch.float32), (after, torch.bfloat16)):
        stream.copy_(before)
        out = None if next_dtype is None else torch.full((n + 1, width), 9.0, dtype=next_dtype, device=DEV)
        kernels.rmsnorm_add(x, weight, stream, eps, n_rows=n, factor=0.7, extra=more, next_weight=next_weight, next_out=out,
                            **gathered)
        assert rel(host(stream[:n]), want) < 1e-5 and torch.equal(host(stream[n]), before[n])
        if out is None:
            continue
        handed = want if next_weight is None else plain.rms_divide(want, eps) * host(after)
        assert rel(host(out[:n]), handed) < (1e-5 if next_dtype == torch.float32 else 1e-2)
        assert bool((out[n] == 9.0).all())
