"""Zatinex's configuration, plan and weights on the CPU: the registry finds the design by its `architecture` key, every
broken field is named, the plan asks a checkpoint for exactly the stored tensors and lays projections of one input end
to end, the decays' rank comes from the checkpoint, the layers' cache needs follow the configuration, and the plain
implementation's functions agree with closed forms."""
import copy
import json
import math

import numpy as np
import pytest
import torch

import plain_zatinex as plain
import zatinex_configs as zc
from burn_transformers_b200 import models  # noqa: F401
from burn_transformers_b200.cache import CacheBank, CacheConfig
from burn_transformers_b200.config.registry import architecture_for, config_from_folder
from burn_transformers_b200.config.zatinex import ZatinexConfig
from burn_transformers_b200.errors import CheckpointError, ConfigError
from burn_transformers_b200.parts import (DifferentialAttention, GatedFeedForward, GatedLinearAttention, InterleavedRotary,
                                          LatentAttention)
from burn_transformers_b200.weights.loader import load_weights

F64 = torch.float64


def build(config):
    return architecture_for("Zatinex").build(ZatinexConfig.from_dict(config))


def test_the_registry_knows_the_design(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(zc.MIXED))
    arch, config = config_from_folder(tmp_path)
    assert arch.name == "zatinex" and isinstance(config, ZatinexConfig) and config.eps == 1e-5
    assert architecture_for("zatinex") is arch
    assert config.to_dict()["layers"] == zc.MIXED["layers"]


def test_the_layers_and_their_cache_needs_follow_the_configuration():
    plan = build(zc.MIXED)
    D, G, L = DifferentialAttention, GatedLinearAttention, LatentAttention
    assert [type(b.mixer) for b in plan.blocks] == [G, L, D, L, L, D, G, L, L]
    none, ff = type(None), GatedFeedForward
    assert [type(b.feed_forward) for b in plan.blocks] == [ff, none, ff, ff, ff, none, none, none, ff]
    assert [call.cache for call in plan.schedule] == [None, None, None, None, 1, None, None, 1, 3]
    needs = plan.cache_needs()
    # a state per head, or rows [key 1 | key 2 | value] with the convolution's inputs, or rows [latent | rotated key part]
    assert needs[0].kv is None and [(s.name, s.shape, s.dtype) for s in needs[0].states] == [("s", (3, 24, 40), torch.float32)]
    assert (needs[2].kv.n_kv_heads, needs[2].kv.head_dim, needs[2].kv.window, needs[2].kv.has_values) == (2, 56, None, False)
    assert [(s.name, s.shape) for s in needs[2].states] == [("qkv_taps", (3, 2 * 6 * 16 + 2 * 2 * 16 + 2 * 24))]
    assert (needs[1].kv.n_kv_heads, needs[1].kv.head_dim) == (1, 56) and not needs[1].states
    assert needs[4].kv is None and not needs[4].states and needs[7].kv is None
    m = plan.blocks[4].mixer
    assert (m.owns_latent, m.has_sink, m.gate_per_head, m.gate_width, m.q_rank) == (False, False, True, 8, 24)
    a = plan.blocks[2].mixer
    assert (a.taps, a.offset, a.positions.dims, a.positions.yarn) == (4, 0.45, 12, (6.0, 200.0, 20.0, 0.5))
    # what is not mentioned does not exist
    assert plan.blocks[5].mixer.positions.yarn is None and plan.blocks[5].mixer.positions.size == 1.0
    assert plan.blocks[1].norm2 is None and plan.blocks[6].mixer.rank == 24
    odd = build(zc.ODD)
    assert odd.cache_needs()[3].states == () and odd.blocks[3].mixer.positions.dims == 0      # (one tap keeps nothing)
    layer = copy.deepcopy(zc.ODD["layers"][5])
    del layer["mixer"]["rot"]
    assert build(dict(zc.ODD, layers=[layer])).blocks[0].mixer.positions.dims == 0


def test_a_model_of_recurrent_layers_only_needs_no_pages():
    bank = CacheBank(build(zc.ONLY_GLA).cache_needs(), CacheConfig(max_tokens=256, max_slots=3, max_context=256), torch.float32,
                     "cpu")
    assert bank.groups == [] and bank.state(0, "s").shape == (3, 3, 32, 24)
    slot = bank.acquire()
    bank.reserve([(slot, 100)])
    bank.commit(slot, 100)
    bank.state(0, "s")[slot] = 5.0
    bank.release(slot)
    assert float(bank.state(0, "s").abs().sum()) == 0.0


@pytest.mark.parametrize("path, value, named", [
    (("width",), 0, "width"),
    (("vocab",), -1, "vocab"),
    (("norm",), {}, "norm.eps"),
    (("norm", "eps"), 0.0, "norm.eps"),
    (("layers",), [], "layers"),
    (("layers", 0, "type"), "linear", "layers[0].type"),
    (("layers", 0, "mixer"), None, "layers[0].mixer"),
    (("layers", 0, "mixer", "tau"), 0, "layers[0].mixer.tau"),
    (("layers", 0, "mixer", "dim"), 0, "layers[0].mixer.dim"),
    (("layers", 0, "mixer", "decay_rank"), 0.5, "layers[0].mixer.decay_rank"),
    (("layers", 0, "mlp", "kind"), "sparse", "layers[0].mlp.kind"),
    (("layers", 0, "mlp", "ff"), 1.5, "layers[0].mlp.ff"),
    (("layers", 1, "mixer", "kv_rank"), 0, "layers[1].mixer.kv_rank"),
    (("layers", 1, "mixer", "q_rank"), None, "layers[1].mixer.q_rank"),
    (("layers", 1, "mixer", "scale"), "a", "layers[1].mixer.scale"),
    (("layers", 1, "mixer", "rot", "dims"), 7, "layers[1].mixer.rot.dims"),
    (("layers", 1, "mixer", "rot", "dims"), 10, "layers[1].mixer.rot.dims"),
    (("layers", 1, "mixer", "rot", "scaling"), {"factor": 2.0}, "layers[1].mixer.rot.scaling"),
    (("layers", 2, "mixer", "kv_heads"), 4, "layers[2].mixer.kv_heads"),
    (("layers", 2, "mixer", "conv"), 0, "layers[2].mixer.conv"),
    (("layers", 2, "mixer", "diff"), None, "layers[2].mixer.diff"),
    (("layers", 2, "mixer", "rot", "dims"), 18, "layers[2].mixer.rot.dims"),
    (("layers", 2, "mixer", "rot", "scaling", "factor"), -1.0, "layers[2].mixer.rot.scaling.factor"),
    (("layers", 2, "mixer", "rot", "scaling"), {"factor": 2.0}, "layers[2].mixer.rot.scaling.original"),
    (("layers", 4, "mixer", "kv_from"), 4, "layers[4].mixer.kv_from"),
    (("layers", 4, "mixer", "kv_from"), 2, "layers[4].mixer.kv_from"),
    (("layers", 7, "mixer", "kv_from"), 4, "layers[7].mixer.kv_from"),
    (("layers", 7, "mixer", "kv_rank"), 40, "layers[7].mixer.kv_rank"),
    (("layers", 7, "mixer", "rot_dim"), 16, "layers[7].mixer.rot_dim"),
])
def test_a_broken_field_is_named(path, value, named):
    data = copy.deepcopy(zc.MIXED)
    at = data
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError) as error:
        ZatinexConfig.from_dict(data)
    assert named in str(error.value)


def test_the_rank_of_the_decays_comes_from_the_checkpoint(tmp_path):
    folder = zc.make_folder(tmp_path / "model", zc.MIXED, seed=2)
    assert "decay_rank" not in (folder / "config.json").read_text()
    arch, config = config_from_folder(folder)
    plan = arch.build(config)
    assert (plan.blocks[0].mixer.rank, plan.blocks[6].mixer.rank) == (8, 24)
    # without a checkpoint, and without the key, the builder says what it lacks
    bare = copy.deepcopy(zc.ONLY_GLA)
    del bare["layers"][0]["mixer"]["decay_rank"]
    with pytest.raises(ConfigError) as error:
        build(bare)
    assert "layers[0].mixer.decay_rank" in str(error.value)


def test_the_plan_reads_exactly_the_stored_tensors(tmp_path):
    folder = zc.make_folder(tmp_path, zc.MIXED, seed=5)
    _, weights = zc.load_plain(folder)
    arch, config = config_from_folder(folder)
    plan = arch.build(config)
    assert set(plan.weights.stored()) == set(weights)
    assert "l1.norm2" not in weights and "l4.mix.dkv" not in weights and weights["l4.mix.g"].shape == (4, 96)
    assert weights["l2.mix.v.conv"].shape == (48, 4) and weights["l0.mix.a2"].shape == (72, 8)
    tensors, _ = load_weights(folder, plan.weights, "float32", torch.device("cpu"))
    f32 = lambda name: weights[name].astype(np.float32)
    # queries, keys and values as one product, their biases and taps likewise
    rows = tensors["l2.mix.in"].numpy()
    assert rows.shape == (192 + 64 + 48, 96)
    np.testing.assert_array_equal(rows[192:256], f32("l2.mix.k"))
    np.testing.assert_array_equal(tensors["l2.mix.in.b"].numpy()[256:], f32("l2.mix.v.b"))
    np.testing.assert_array_equal(tensors["l2.mix.conv"].numpy()[:192], f32("l2.mix.q.conv"))
    # the gates' rows padded by zeros to whole 16-byte pieces, between the queries' latent and the keys'
    rows = tensors["l3.mix.in"].numpy()
    assert rows.shape == (56 + 8 + 48, 96)
    np.testing.assert_array_equal(rows[56:61], f32("l3.mix.g"))
    assert not rows[61:64].any()
    np.testing.assert_array_equal(rows[64:], f32("l3.mix.dkv"))
    # a gated linear attention's five matrices as one
    rows = tensors["l6.mix.in"].numpy()
    assert rows.shape == (112 + 112 + 32 + 32 + 24, 96)
    np.testing.assert_array_equal(rows[288:], f32("l6.mix.a1"))
    np.testing.assert_array_equal(rows[256:288], f32("l6.mix.g"))
    plan.bind(tensors)
    share = plan.blocks[2].mixer.share
    w = plain.layer_tensors(weights, 2, "mix")
    np.testing.assert_allclose(share.numpy(), float(plain.two_map_share(w, 0.45)), rtol=1e-6)
    # a second norm of a layer without a feed-forward is let pass; a missing tensor is named
    from burn_transformers_b200.weights.safetensors_io import write_file

    def rewrite():
        (folder / "model.safetensors").unlink()
        write_file(folder / "model.safetensors", {k: torch.tensor(np.asarray(v)).to(torch.float32) for k, v in weights.items()})
    weights["l1.norm2"] = np.ones(96)
    rewrite()
    load_weights(folder, plan.weights, "float32", torch.device("cpu"))
    del weights["l2.mix.lk2"]
    rewrite()
    with pytest.raises(CheckpointError) as error:
        load_weights(folder, plan.weights, "float32", torch.device("cpu"))
    assert "l2.mix.lk2" in str(error.value)


@pytest.mark.parametrize("dims, base, scaling", [(16, 1e4, (5.0, 1024.0, 24.0, 1.0)), (64, 5e5, (4.0, 4096.0, 40.0, 0.5)),
                                                 (2, 100.0, (3.0, 10.0, 4.0, 1.0)), (8, 50.0, (2.0, 30.0, 900.0, 600.0)),
                                                 (32, 1e6, (1.0, 512.0, 16.0, 2.0)), (12, 20.0, (5.0, 9e9, 2.0, 1.0))])
def test_the_scaled_frequencies_of_the_rotation(dims, base, scaling):
    part = InterleavedRotary(dims, base, yarn=scaling)
    rates, size = plain.turn_rates(dims, base, dict(zip(("factor", "original", "fast", "slow"), scaling)))
    np.testing.assert_allclose(part.frequencies(), rates, rtol=1e-13)
    assert abs(part.size - size) < 1e-15
    # the fastest pair is never faster than unscaled, the slowest never slower than divided by the factor
    free = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    assert all(f / scaling[0] * (1 - 1e-12) <= r <= f * (1 + 1e-12) for r, f in zip(rates, free))
    with pytest.raises(NotImplementedError):
        InterleavedRotary(4, 10.0, yarn=(2.0, 64.0, 8.0, 1.0)).rotate_vectors(None, None, None)


def test_the_plain_rotation_turns_neighbours_and_scales_them():
    rng = np.random.default_rng(2)
    x = torch.from_numpy(rng.standard_normal((5, 2, 10)))
    turned = plain.rotate_neighbours(x, torch.arange(5), {"dims": 6, "base": 100.0})
    assert torch.equal(turned[..., 6:], x[..., 6:]) and torch.equal(turned[0], x[0])
    np.testing.assert_allclose((turned ** 2).sum(-1), (x ** 2).sum(-1), rtol=1e-12)
    np.testing.assert_allclose(turned[1, 0, 0], x[1, 0, 0] * math.cos(1.0) - x[1, 0, 1] * math.sin(1.0), rtol=1e-12)
    scaled = plain.rotate_neighbours(x, torch.arange(5), {"dims": 6, "base": 100.0, "scaling": {
        "factor": math.e, "original": 1e12, "fast": 2.0, "slow": 1.0}})
    np.testing.assert_allclose(scaled[..., :6], 1.1 * turned[..., :6], rtol=1e-12)       # (all pairs stay; size 1.1)


def test_the_plain_convolution_reads_the_newest_input_with_the_last_tap():
    u = torch.arange(1.0, 6.0, dtype=F64)[:, None].repeat(1, 2)
    taps = torch.tensor([[100.0, 10.0, 1.0], [0.0, 0.0, 1.0]], dtype=F64)
    out = plain.short_convolution(u, taps)
    np.testing.assert_array_equal(out[:, 0], [1.0, 12.0, 123.0, 234.0, 345.0])
    np.testing.assert_array_equal(out[:, 1], u[:, 1])


def test_the_plain_recurrence_forgets_per_key_channel_and_goes_on_from_its_state():
    rng = np.random.default_rng(1)
    q, k = (torch.from_numpy(rng.standard_normal((30, 4))) for _ in range(2))
    v, a = torch.from_numpy(rng.standard_normal((30, 3))), torch.from_numpy(rng.random((30, 4)))
    zero = torch.zeros(4, 3, dtype=F64)
    whole, last = plain.gated_recurrence(q, k, v, a, zero)
    first, kept = plain.gated_recurrence(q[:13], k[:13], v[:13], a[:13], zero)
    second, end = plain.gated_recurrence(q[13:], k[13:], v[13:], a[13:], kept)
    np.testing.assert_allclose(torch.cat([first, second]), whole, rtol=1e-12)
    assert torch.equal(end, last)
    # unrolled: token s reaches token t by the product of the decays in between, channel by channel
    t = 17
    want = sum((q[t] * k[s] * torch.prod(a[s + 1:t + 1], 0)).sum() * v[s] for s in range(t + 1))
    np.testing.assert_allclose(whole[t], want, rtol=1e-10)


def test_the_plain_maps_are_subtracted_and_normed():
    w = {n: torch.tensor(v, dtype=F64) for n, v in (("lq1", [1.0, 0.0]), ("lk1", [0.5, 9.0]), ("lq2", [0.0, 2.0]), ("lk2", [7.0, 0.1]))}
    share = plain.two_map_share(w, 0.25)
    np.testing.assert_allclose(share, math.exp(0.5) - math.exp(0.2) + 0.25, rtol=1e-12)
    a, b = torch.tensor([[3.0, 1.0]], dtype=F64), torch.tensor([[1.0, 1.0]], dtype=F64)
    out = plain.combine_maps(a, b, torch.tensor(1.0, dtype=F64), 0.25, 0.0)
    np.testing.assert_allclose(out, [[math.sqrt(2.0) * 0.75, 0.0]], rtol=1e-12)
