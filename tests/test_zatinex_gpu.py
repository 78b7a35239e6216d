"""Zatinex through the engine against the plain implementation: every mechanism alone and together, whole prompts,
decoding token by token, prompts in portions down to two tokens, batches of unequal requests with slots and pages used
again, long decoding, sharp scores, one loud key far back and at page borders, gates of one number a head, states that must
last, and greedy generation through the library's entry points and programs."""
import json
import os
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

import engine_replay as replay
import plain_zatinex as plain
import zatinex_configs as zc
from burn_transformers_b200 import (AutoCausalLm, AutoLoadOptions, CausalGenerationRequest, Engine, GenerationConfig,
                                    StepEntry, generate_causal)

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
# 32-bit: every position.  16-bit: these models are a few dozen channels wide, so one rounding moves a logit by about a
# hundredth of the largest (the norm over a difference of two maps enlarges it where the maps nearly agree): the bound holds
# for all but a few positions in a hundred, the typical one stays far below
TOL = {"float32": 1e-4, "bfloat16": 1e-1}
TYPICAL_16 = 2.5e-2
# lengths around the borders of a page (64), of the kernels' tiles (32, 128), of the recurrence's chunks (64) and groups (4),
# and around the lengths from which prompts take their tensor-core forms (32, 48)
LENGTHS = {"mixed": [1, 2, 7, 17, 47, 64, 65, 129, 260], "odd": [1, 9, 33, 64, 130], "large": [1, 31, 48, 200],
           "only_attention": [1, 2, 31, 32, 64, 65, 128, 129, 300], "only_gla": [1, 2, 16, 17, 64, 65, 67, 128, 131, 700],
           "only_latent": [1, 5, 47, 48, 64, 140], "shared_latent": [1, 5, 47, 48, 66, 140], "only_dense": [1, 5, 70]}


def assert_close(got, ref, dtype, tol=None, note=""):
    tol = TOL[dtype] if tol is None else tol
    each = [float(np.abs(row - ref[r][p]).max() / np.abs(ref[r]).max()) for (r, p), row in got.items()]
    if dtype == "float32":
        err, where = replay.worst_error(got, ref)
        assert err < tol, f"{note}{err:.3e} at {where}"
    else:
        assert np.quantile(each, 0.95) < tol, f"{note}95th percentile {np.quantile(each, 0.95):.3e}"
        assert np.median(each) < TYPICAL_16, f"{note}median {np.median(each):.3e}"


@pytest.fixture(scope="module", params=list(zc.CONFIGS))
def case(request, tmp_path_factory):
    name = request.param
    config = zc.CONFIGS[name]
    folder = zc.make_folder(tmp_path_factory.mktemp(name), config, seed=21)
    pcfg, pw = zc.load_plain(folder)
    seqs = zc.prompts(config, LENGTHS[name], seed=2)
    return name, folder, seqs, [plain.forward(pcfg, pw, s) for s in seqs]


def engine_for(folder, dtype, max_tokens=64 * 16, **kw):
    return Engine.from_folder(folder, dtype, max_tokens=max_tokens, **kw)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_each_request_whole(case, dtype):
    _, folder, seqs, ref = case
    got = replay.whole(engine_for(folder, dtype), seqs)
    assert len(got) == sum(len(s) for s in seqs)
    assert_close(got, ref, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_last_tokens_one_by_one(case, dtype):
    _, folder, seqs, ref = case
    got = replay.tail_one_by_one(engine_for(folder, dtype), seqs, tail=45)
    assert_close(got, ref, dtype)


def in_portions(engine, seqs, size):
    """Each request alone, `size` tokens a step."""
    got = {}
    for r, seq in enumerate(seqs):
        slot = engine.new_sequence()
        for lo in range(0, len(seq), size):
            piece = seq[lo:lo + size]
            logits = engine.step([StepEntry(slot, piece, list(range(len(piece))))]).detach().cpu().double().numpy()
            for i, row in enumerate(logits):
                got[(r, lo + i)] = row
        engine.release(slot)
    return got


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size", [2, 3, 17, 64, 70])
def test_prompts_in_portions(case, dtype, size):
    """The pages, the convolution's inputs and the recurrent states carry a sequence from one portion to the next (a
    portion of two tokens is shorter than a convolution's reach)."""
    name, folder, seqs, ref = case
    if name not in ("mixed", "odd", "only_attention", "only_gla") and size in (3, 17, 70):
        pytest.skip("the full set of portion sizes runs on four configurations")
    got = in_portions(engine_for(folder, dtype), seqs, size)
    assert_close(got, ref, dtype, note=f"portions of {size}: ")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batches_of_unequal_requests_use_slots_and_pages_again(case, dtype):
    _, folder, seqs, ref = case
    n = len(seqs)
    groups = [list(range(0, n, 2)), list(range(1, n, 2)), list(range(n))[:3], list(range(n))[::-1][:3]]
    cut = [max(1, len(s) // 3) for s in seqs]
    cut[0] = 1
    need = max(sum(-(-len(seqs[r]) // 64) * 64 for r in g) for g in groups)
    engine = engine_for(folder, dtype, max_tokens=need, max_slots=max(len(g) for g in groups))
    got = replay.batches(engine, seqs, groups, cut)
    assert_close(got, ref, dtype)
    assert engine.cache.slots.held == 0 and all(g.pool.held == 0 for g in engine.cache.groups)
    if dtype == "float32":
        # a request's logits do not depend on what else is in the batch
        alone = replay.whole(engine, seqs)
        drift = max(float(np.abs(alone[k] - got[k]).max() / np.abs(ref[k[0]]).max()) for k in got)
        assert drift < TOL[dtype]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_from_the_first_token(case, dtype):
    """Every token decoded alone, from the zero state and an empty cache."""
    _, folder, seqs, ref = case
    long = max(range(len(seqs)), key=lambda r: len(seqs[r]))
    got = replay.tail_one_by_one(engine_for(folder, dtype), [seqs[long]], tail=10 ** 6)
    assert len(got) == len(seqs[long])
    assert_close({(long, p): row for (_, p), row in got.items()}, ref, dtype)


def test_a_released_slot_starts_from_an_empty_state(case):
    """A sequence that takes over a slot finds neither the old state, the old convolution inputs nor the old keys."""
    _, folder, seqs, ref = case
    engine = engine_for(folder, "float32", max_tokens=64 * 11, max_slots=1)
    for r in (len(seqs) - 1, 1, len(seqs) - 2, 0):
        slot = engine.new_sequence()
        assert slot == 0
        got = engine.step([StepEntry(slot, seqs[r], [len(seqs[r]) - 1])]).cpu().double().numpy()[0]
        engine.release(slot)
        assert np.abs(got - ref[r][-1]).max() / np.abs(ref[r]).max() < TOL["float32"], r


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_many_requests_at_once(dtype, tmp_path):
    """70 requests decode together (the fused steps' bound of 64 tokens is passed, and that of 16 rows for norms inside
    products), then fewer as they end; then portions of a few sequences and single tokens of others in one step."""
    folder = zc.make_folder(tmp_path, zc.MIXED, seed=6)
    pcfg, pw = zc.load_plain(folder)
    rng = np.random.default_rng(8)
    seqs = zc.prompts(zc.MIXED, rng.integers(4, 96, 70).tolist(), seed=4)
    ref = [plain.forward(pcfg, pw, s) for s in seqs]
    engine = engine_for(folder, dtype, max_tokens=64 * 140, max_slots=70, max_context=128)
    got = replay.batches(engine, seqs, [list(range(70))], [max(1, len(s) - 6) for s in seqs])
    assert_close(got, ref, dtype)
    slots = [engine.new_sequence() for _ in range(4)]
    cuts = [(0, 3), (0, 1), (0, 2), (0, 4)]
    got = {}
    while any(lo < len(seqs[r]) for r, (lo, _) in enumerate(cuts)):
        live = [r for r in range(4) if cuts[r][0] < len(seqs[r])]
        entries = [StepEntry(slots[r], seqs[r][cuts[r][0]:cuts[r][0] + cuts[r][1]],
                             list(range(len(seqs[r][cuts[r][0]:cuts[r][0] + cuts[r][1]])))) for r in live]
        rows = iter(engine.step(entries).cpu().double().numpy())
        for r, e in zip(live, entries):
            for i in range(len(e.tokens)):
                got[(r, cuts[r][0] + i)] = next(rows)
            cuts[r] = (cuts[r][0] + len(e.tokens), 1 if cuts[r][1] > 3 else cuts[r][1] + 1)
    assert_close(got, ref, dtype)


@pytest.mark.parametrize("name", ["mixed", "only_attention", "shared_latent", "odd"])
def test_sharp_scores(name, tmp_path):
    """Scores scaled up eightfold: a softmax row's weight sits on one or two keys, so a key lost at a page's border or filed
    in the wrong place moves the logits visibly; in prompts, in decoding, and in a batch."""
    config = zc.sharp(zc.CONFIGS[name])
    folder = zc.make_folder(tmp_path, config, seed=8)
    pcfg, pw = zc.load_plain(folder)
    seqs = zc.prompts(config, [290, 131], seed=6)
    ref = [plain.forward(pcfg, pw, s) for s in seqs]
    engine = engine_for(folder, "float32")
    for got in (replay.whole(engine, seqs), replay.tail_one_by_one(engine, seqs, tail=120),
                replay.batches(engine, seqs, [[0, 1]], [150, 3]), in_portions(engine, seqs, 37)):
        err, where = replay.worst_error(got, ref)
        assert err < 5e-4, f"{err:.3e} at {where}"


def _loud_attention(which):
    """Token 7's key in map `which` (0 or 1) stands out for every query: channel 1 of the stream is the same large number for
    every token and all queries of that map read it into the unrotated last channel; channel 0, zero for every token but
    token 7, makes the same channel of its key; no position turns it, the convolution passes the newest input on.  Value
    rows read channel 0 too, so what is found shows."""
    def edit(tensors):
        tensors["embed"][:, 1] = 5.0
        tensors["embed"][:, 0] = 0.0
        tensors["embed"][7] = 0.0
        tensors["embed"][7, 0], tensors["embed"][7, 1] = 30.0, 5.0
        dim = 16
        for name in "qkv":
            tensors[f"l0.mix.{name}.conv"][:, :-1] *= 0.05
            tensors[f"l0.mix.{name}.conv"][:, -1] = 1.0
            tensors[f"l0.mix.{name}.b"] *= 0.1
        for name in "qk":
            tensors[f"l0.mix.{name}.norm"] = np.ones(dim)
            tensors[f"l0.mix.{name}"] *= 0.3
        rows = tensors["l0.mix.q"].reshape(4, 2, dim, -1)
        rows[:, which, dim - 1, 1] = 3.0
        rows = tensors["l0.mix.k"].reshape(2, 2, dim, -1)
        rows[:, which, dim - 1, 0] = 6.0
        tensors["l0.mix.v"][:, 0] = np.linspace(-1.0, 1.0, tensors["l0.mix.v"].shape[0])
        return tensors
    return edit


@pytest.mark.parametrize("which", [0, 1])
def test_a_key_far_back_among_hundreds_in_either_map(which, tmp_path):
    """The loud key at position 5 still carries its map 600 tokens later, across ten pages; one at each side of a page's
    and a tile's border does so for itself; the plain implementation says by how much."""
    config = zc.sharp(zc.ONLY_ATTENTION, 3.0)
    folder = zc.make_folder(tmp_path, config, seed=5, edit=_loud_attention(which))
    pcfg, pw = zc.load_plain(folder)
    rng = np.random.default_rng(4)
    base = rng.integers(8, config["vocab"], 640).tolist()
    plain_base = plain.forward(pcfg, pw, base)
    engine, bf16 = engine_for(folder, "float32"), engine_for(folder, "bfloat16")
    for at in (0, 5, 63, 64, 127, 128, 638):
        seq = list(base)
        seq[at] = 7
        ref = plain.forward(pcfg, pw, seq)
        assert np.abs(plain_base[-1] - ref[-1]).max() > 100 * TOL["float32"] * np.abs(ref).max()
        for got in (replay.whole(engine, [seq]), replay.tail_one_by_one(engine, [seq], tail=40)):
            err, where = replay.worst_error(got, [ref])
            assert err < TOL["float32"], f"{err:.3e} at {where} with the key at {at}"
        for got in (replay.whole(bf16, [seq]), replay.tail_one_by_one(bf16, [seq], tail=40)):
            assert_close(got, [ref], "bfloat16", note=f"the key at {at}: ")


def _loud_latent(tensors):
    """Token 7's key stands out for every query of both layers: channel 1 of the stream is the same large number for every
    token and the queries' latent reads it; channel 0, which is zero for every token but token 7, makes the keys' latent;
    up-projections of one sign carry both into heads that agree.  The rotated part stays quiet."""
    tensors["embed"][:, 1] = 5.0
    tensors["embed"][:, 0] = 0.0
    tensors["embed"][7] = 0.0
    tensors["embed"][7, 0], tensors["embed"][7, 1] = 30.0, 5.0
    rank = 32
    tensors["l0.mix.dkv"] *= 0.02
    tensors["l0.mix.dkv"][:rank, 0] = 3.0
    tensors["l0.mix.dkv"][rank:, 0] = 0.0
    tensors["l0.mix.dkv.norm"] = np.abs(tensors["l0.mix.dkv.norm"]) + 0.5
    for i in (0, 1):
        tensors[f"l{i}.mix.dq"] *= 0.02
        tensors[f"l{i}.mix.dq"][:, 1] = 1.0
        tensors[f"l{i}.mix.dq.norm"] = np.abs(tensors[f"l{i}.mix.dq.norm"]) + 0.5
        tensors[f"l{i}.mix.uq"] = np.abs(tensors[f"l{i}.mix.uq"])
        tensors[f"l{i}.mix.uk"][:] = 0.1
        tensors[f"l{i}.norm1"] = np.ones(64)
    return tensors


def test_a_latent_far_back_read_by_its_own_layer_and_a_later_one(tmp_path):
    config = zc.sharp(zc.SHARED_LATENT, 4.0)
    folder = zc.make_folder(tmp_path, config, seed=5, edit=_loud_latent)
    pcfg, pw = zc.load_plain(folder)
    base = np.random.default_rng(4).integers(8, config["vocab"], 640).tolist()
    plain_base = plain.forward(pcfg, pw, base)
    engine = engine_for(folder, "float32")
    for at in (0, 5, 63, 64, 638):
        seq = list(base)
        seq[at] = 7
        ref = plain.forward(pcfg, pw, seq)
        assert np.abs(plain_base[-1] - ref[-1]).max() > 100 * TOL["float32"] * np.abs(ref).max()
        for got in (replay.whole(engine, [seq]), replay.tail_one_by_one(engine, [seq], tail=40)):
            err, where = replay.worst_error(got, [ref])
            assert err < TOL["float32"], f"{err:.3e} at {where} with the key at {at}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_gate_is_one_number_a_head(dtype, tmp_path):
    """Gates biased apart through a stream channel that is the same for every token: the first head shut, the last open."""
    def edit(tensors):
        tensors["embed"][:, 1] = 4.0
        tensors["l0.norm1"] = np.ones(64)
        tensors["l0.mix.g"][:, 1] = np.array([-4.0, -0.5, 0.5, 4.0])
        return tensors
    folder = zc.make_folder(tmp_path, zc.ONLY_LATENT, seed=5, edit=edit)
    seqs = zc.prompts(zc.ONLY_LATENT, [1, 90, 3], seed=5)
    ref = [plain.forward(*zc.load_plain(folder), s) for s in seqs]
    engine = engine_for(folder, dtype)
    for got in (replay.whole(engine, seqs), replay.tail_one_by_one(engine, seqs, tail=30), in_portions(engine, seqs, 7)):
        assert_close(got, ref, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_state_that_must_last(dtype, tmp_path):
    """Decays biased towards one: what one early token left in the state still decides the logits 700 tokens later, whole,
    in portions and token by token."""
    def slow(tensors):
        tensors["l0.mix.a2.b"][:] = 9.0
        tensors["embed"][:, 0] = 0.0
        tensors["embed"][:, 1] = 4.0
        tensors["embed"][7, 0] = 30.0
        for name in "qk":
            tensors[f"l0.mix.{name}"] *= 0.1
        tensors["l0.mix.q"][:, 1] = 0.3            # (every query finds what token 7 alone has written)
        tensors["l0.mix.k"][:, 0] = 2.0
        return tensors
    folder = zc.make_folder(tmp_path, zc.ONLY_GLA, seed=9, edit=slow)
    pcfg, pw = zc.load_plain(folder)
    seq = np.random.default_rng(1).integers(8, 120, 720).tolist()
    other = list(seq)
    seq[1] = 7
    ref = plain.forward(pcfg, pw, seq)
    assert np.abs(plain.forward(pcfg, pw, other)[-1] - ref[-1]).max() > 0.05 * np.abs(ref).max()
    engine = engine_for(folder, dtype)
    for got in (replay.whole(engine, [seq]), replay.tail_one_by_one(engine, [seq], tail=300), in_portions(engine, [seq], 50)):
        assert_close(got, [ref], dtype)


def plain_greedy(pcfg, pw, prompt, n):
    seq = list(prompt)
    margins = []
    for _ in range(n):
        row = plain.forward(pcfg, pw, seq)[-1]
        order = np.argsort(row)
        margins.append(float(row[order[-1]] - row[order[-2]]))
        seq.append(int(order[-1]))
    return seq[len(prompt):], margins


def test_greedy_generation_through_the_entry_point(tmp_path):
    """Three unequal prompts as one batch through load_local and generate_causal (the scheduler, the recorded decode
    steps, the device sampler), with and without prompts fed in portions: the plain implementation's tokens."""
    folder = zc.make_folder(tmp_path, zc.MIXED, seed=13)
    pcfg, pw = zc.load_plain(folder)
    prompts = zc.prompts(zc.MIXED, [3, 70, 18], seed=9)
    want = [plain_greedy(pcfg, pw, p, 12) for p in prompts]
    loaded = AutoCausalLm.load_local(folder, AutoLoadOptions(dtype="float32", max_tokens=64 * 4))
    for portion in (None, 16):
        out = generate_causal(loaded.model, CausalGenerationRequest(prompts, GenerationConfig(max_new_tokens=12),
                                                                    prefill_chunk_size=portion))
        for sequence, (tokens, margins) in zip(out.sequences, want):
            # (compared up to the first step the plain implementation itself decides by less than rounding can move)
            sure = next((i for i, m in enumerate(margins) if m < 1e-3), len(tokens))
            assert sequence.token_ids[:sure] == tokens[:sure] and sure >= 4
    bf16 = AutoCausalLm.load_local(folder, AutoLoadOptions(dtype="bfloat16", max_tokens=64 * 4))
    out16 = generate_causal(bf16.model, CausalGenerationRequest(prompts, GenerationConfig(max_new_tokens=12)))
    assert all(len(s.token_ids) == 12 for s in out16.sequences)
    assert sum(a == b for s, (t, _) in zip(out16.sequences, want) for a, b in zip(s.token_ids, t)) >= 12


def test_the_programs_serve_the_model(tmp_path):
    """bin/random_model writes a folder from a configuration file, bin/generate decodes from it, bin/trace_run replays a
    batch of two unequal requests on it."""
    cfg_file = tmp_path / "cfg.json"
    cfg_file.write_text(json.dumps(zc.ODD))
    folder = tmp_path / "model"
    made = subprocess.run([sys.executable, str(ROOT / "bin" / "random_model"), str(cfg_file), str(folder), "--seed", "4"],
                          capture_output=True, text=True, timeout=600)
    assert made.returncode == 0, made.stderr
    pcfg, pw = zc.load_plain(folder)
    done = subprocess.run([str(ROOT / "bin" / "generate"), str(folder), "5,6,7,8", "6", "--dtype", "float32"],
                          capture_output=True, text=True, timeout=900)
    assert done.returncode == 0, done.stderr
    ids = [int(x) for x in done.stdout.split()]
    tokens, margins = plain_greedy(pcfg, pw, [5, 6, 7, 8], 6)
    sure = next((i for i, m in enumerate(margins) if m < 1e-3), 6)
    assert ids[:4] == [5, 6, 7, 8] and ids[4:4 + sure] == tokens[:sure]
    a, b = zc.prompts(zc.ODD, [70, 9], seed=1)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [0, 65]}, {"id": "b", "tokens": b[:2], "want": []}],
              "end": []}]
    for i in range(7):
        live = [("a", a, 66 + i)] * (66 + i < len(a)) + [("b", b, 2 + i)]
        steps.append({"step": i + 1, "entries": [{"id": r, "tokens": [s[p]], "want": [0]} for r, s, p in live],
                      "end": [r for r, s, p in live if p + 1 == len(s)]})
    out = tmp_path / "out"
    run = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(out),
                          "--max-tokens", "79"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                         capture_output=True, text=True, timeout=900, env=dict(os.environ))
    assert run.returncode == 0, run.stderr
    assert run.stdout.split() == [w for s in steps for w in ("done", str(s["step"]))]
    ref = {"a": plain.forward(pcfg, pw, a), "b": plain.forward(pcfg, pw, b)}
    first = np.frombuffer((out / "0.f32").read_bytes(), dtype="<f4").reshape(2, -1)
    assert np.abs(first[1] - ref["a"][65]).max() / np.abs(ref["a"]).max() < 1e-4
    last = np.frombuffer((out / "7.f32").read_bytes(), dtype="<f4").reshape(1, -1)
    assert np.abs(last[0] - ref["b"][8]).max() / np.abs(ref["b"]).max() < 1e-4
