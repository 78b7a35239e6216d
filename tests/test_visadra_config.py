"""Visadra's configuration, plan and weights on the CPU: the registry finds the design by its `architecture` key, every
broken field is named, the plan asks a checkpoint for exactly the stored tensors and lays projections of one input end
to end, the layers' cache needs follow the configuration, and the plain implementation's functions agree with closed
forms."""
import copy
import json
import math

import numpy as np
import pytest
import torch

import plain_visadra as plain
import visadra_configs as vc
from burn_transformers_b200 import models  # noqa: F401
from burn_transformers_b200.cache import CacheBank, CacheConfig
from burn_transformers_b200.config.registry import architecture_for, config_from_folder
from burn_transformers_b200.config.visadra import VisadraConfig
from burn_transformers_b200.errors import CheckpointError, ConfigError
from burn_transformers_b200.parts import GatedFeedForward, LatentAttention, MinGru, RoutedFeedForward
from burn_transformers_b200.weights.loader import load_weights


def build(config):
    return architecture_for("Visadra").build(VisadraConfig.from_dict(config))


def test_the_registry_knows_the_design(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(vc.MIXED))
    arch, config = config_from_folder(tmp_path)
    assert arch.name == "visadra" and isinstance(config, VisadraConfig)
    assert architecture_for("visadra") is arch
    assert config.to_dict()["layers"] == vc.MIXED["layers"]
    assert (config.eps, config.embedding_scale, config.logit_scale) == (1e-5, 3.0, 0.7)


def test_the_layers_and_their_cache_needs_follow_the_configuration():
    plan = build(vc.MIXED)
    kinds = [type(b.mixer) for b in plan.blocks]
    assert kinds == [MinGru, LatentAttention, MinGru, LatentAttention, MinGru, LatentAttention, MinGru]
    assert [type(b.feed_forward) for b in plan.blocks] == [GatedFeedForward, RoutedFeedForward, RoutedFeedForward,
                                                           GatedFeedForward, type(None), type(None), RoutedFeedForward]
    needs = plan.cache_needs()
    # a state of one number a channel, or one row [latent | rotated key part] a position
    assert [(s.name, s.shape, s.dtype) for s in needs[0].states] == [("s", (136,), torch.float32)] and needs[0].kv is None
    assert needs[2].states[0].shape == (64,) and needs[4].states[0].shape == (200,)
    assert (needs[1].kv.n_kv_heads, needs[1].kv.head_dim, needs[1].kv.window, needs[1].kv.has_values) == (1, 56, None, False)
    assert not needs[1].states
    # what is not mentioned does not exist
    assert plan.blocks[6].feed_forward.shared is None and plan.blocks[1].feed_forward.shared.inner == 72
    assert plan.blocks[5].norm2 is None
    ff = plan.blocks[2].feed_forward
    assert (ff.n_experts, ff.top, ff.inner, ff.router, ff.gated, ff.has_logit_bias, ff.activation) == (
        5, 3, 56, "softmax_of_chosen", True, True, "swish")
    m = plan.blocks[3].mixer
    assert (m.has_sink, m.has_gate, m.window, m.q_rank, m.positions.dims, m.positions.base) == (True, False, None, None, 16, 20000.0)
    bare = {k: v for k, v in vc.MIXED.items() if k not in ("logit_scale", "embedding")}
    config = VisadraConfig.from_dict(bare)
    assert config.embedding_scale == 1.0 and config.logit_scale == 1.0
    # a latent layer without rotated channels needs no rotation
    plain_layer = copy.deepcopy(vc.ODD["layers"][4])
    del plain_layer["mixer"]["rot"]
    assert build(dict(vc.ODD, layers=[plain_layer])).blocks[0].mixer.positions.dims == 0


def test_a_model_of_recurrent_layers_only_needs_no_pages():
    bank = CacheBank(build(vc.ONLY_GRU).cache_needs(), CacheConfig(max_tokens=256, max_slots=3, max_context=256), torch.float32,
                     "cpu")
    assert bank.groups == [] and bank.state(0, "s").shape == (3, 72)
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
    (("embedding", "scale"), "x", "embedding.scale"),
    (("logit_scale",), None, "logit_scale"),
    (("layers",), [], "layers"),
    (("layers", 0, "type"), "gru", "layers[0].type"),
    (("layers", 0, "mixer"), None, "layers[0].mixer"),
    (("layers", 0, "mixer", "width"), 0, "layers[0].mixer.width"),
    (("layers", 2, "mixer"), {}, "layers[2].mixer.width"),
    (("layers", 0, "mlp", "kind"), "sparse", "layers[0].mlp.kind"),
    (("layers", 0, "mlp", "ff"), 1.5, "layers[0].mlp.ff"),
    (("layers", 1, "mixer", "kv_rank"), 0, "layers[1].mixer.kv_rank"),
    (("layers", 1, "mixer", "scale"), "a", "layers[1].mixer.scale"),
    (("layers", 1, "mixer", "rot", "dims"), 7, "layers[1].mixer.rot.dims"),
    (("layers", 1, "mixer", "rot", "dims"), 10, "layers[1].mixer.rot.dims"),
    (("layers", 1, "mixer", "rot", "base"), 0, "layers[1].mixer.rot.base"),
    (("layers", 1, "mixer", "rot"), None, "layers[1].mixer.rot"),
    (("layers", 1, "mlp", "router", "top"), 7, "layers[1].mlp.router.top"),
    (("layers", 1, "mlp", "expert"), {}, "layers[1].mlp.expert.ff"),
    (("layers", 1, "mlp", "shared"), {"ff": 0}, "layers[1].mlp.shared.ff"),
])
def test_a_broken_field_is_named(path, value, named):
    data = copy.deepcopy(vc.MIXED)
    at = data
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError) as error:
        VisadraConfig.from_dict(data)
    assert named in str(error.value)


def test_the_plan_reads_exactly_the_stored_tensors(tmp_path):
    folder = vc.make_folder(tmp_path, vc.MIXED, seed=5)
    config, weights = vc.load_plain(folder)
    plan = build(config)
    assert set(plan.weights.stored()) == set(weights)
    assert weights["l0.norm1"].shape == () and weights["final.norm"].shape == () and "l5.norm2" not in weights
    assert "l6.mlp.shared.gate" not in weights and weights["l1.mlp.router.b"].shape == (6,)
    tensors, _ = load_weights(folder, plan.weights, "float32", torch.device("cpu"))
    # the gate's, the candidate's and the output gate's rows as one matrix, the two biases as one vector
    rows = tensors["l0.mix.in"].numpy()
    assert rows.shape == (3 * 136, 96)
    np.testing.assert_array_equal(rows[136:272], weights["l0.mix.x"].astype(np.float32))
    np.testing.assert_array_equal(tensors["l0.mix.b"].numpy()[136:], weights["l0.mix.x.b"].astype(np.float32))
    # queries and the latent's down-projection as one
    rows = tensors["l1.mix.in"].numpy()
    assert rows.shape == (3 * 24 + 48 + 8, 96)
    np.testing.assert_array_equal(rows[72:], weights["l1.mix.dkv"].astype(np.float32))
    # per expert the gate's rows, then up's; all experts end to end
    rows = tensors["l2.mlp.experts.gate_up"].numpy()
    assert rows.shape == (5 * 2 * 56, 96)
    np.testing.assert_array_equal(rows[2 * 112 + 56:3 * 112], weights["l2.mlp.e2.up"].astype(np.float32))
    np.testing.assert_array_equal(tensors["l2.mlp.experts.down"].numpy()[96:192], weights["l2.mlp.e1.down"].astype(np.float32))
    # one number becomes a gain for every channel when it is bound
    plan.bind(tensors)
    gain = plan.blocks[0].norm1.t_weight
    assert gain.shape == (96,) and bool((gain == float(weights["l0.norm1"])).all())
    # a second norm of a layer without a feed-forward is let pass; a missing tensor is named
    from burn_transformers_b200.weights.safetensors_io import write_file

    def rewrite():
        (folder / "model.safetensors").unlink()
        write_file(folder / "model.safetensors", {k: torch.tensor(np.asarray(v)).to(torch.float32) for k, v in weights.items()})
    weights["l5.norm2"] = np.array(0.5)
    rewrite()
    load_weights(folder, plan.weights, "float32", torch.device("cpu"))
    del weights["l3.mix.sink"]
    rewrite()
    with pytest.raises(CheckpointError) as error:
        load_weights(folder, plan.weights, "float32", torch.device("cpu"))
    assert "l3.mix.sink" in str(error.value)


def test_the_plain_average_goes_on_from_its_state_and_stays_between_its_values():
    rng = np.random.default_rng(1)
    z, v = torch.from_numpy(rng.random((40, 5))), torch.from_numpy(rng.standard_normal((40, 5)))
    whole, last = plain.gated_average(z, v, torch.zeros(5, dtype=torch.float64))
    first, kept = plain.gated_average(z[:13], v[:13], torch.zeros(5, dtype=torch.float64))
    second, end = plain.gated_average(z[13:], v[13:], kept)
    np.testing.assert_allclose(torch.cat([first, second]), whole, rtol=1e-12)
    assert torch.equal(end, last) and torch.equal(last, whole[-1])
    # S_t is a mean of zero and the values so far, each weighted by its share of what came after
    weights = torch.stack([z[s] * torch.prod(1 - z[s + 1:], 0) for s in range(40)])
    np.testing.assert_allclose((weights * v).sum(0), last, rtol=1e-9)
    np.testing.assert_allclose(plain.candidate(torch.tensor([0.0, 2.0, -1.0], dtype=torch.float64)),
                               [0.5, 2.5, 1.0 / (1.0 + math.e)], rtol=1e-12)


def test_the_plain_sink_takes_weight_and_gives_nothing():
    scores = torch.tensor([[1.0, 2.0, 300.0]], dtype=torch.float64)
    seen = torch.tensor([[True, True, False]])
    p = plain.softmax_beside_a_sink(scores, seen, torch.tensor(2.0, dtype=torch.float64))
    total = math.exp(1.0) + 2 * math.exp(2.0)
    np.testing.assert_allclose(p[0], [math.exp(1.0) / total, math.exp(2.0) / total, 0.0], rtol=1e-12)
    p = plain.softmax_beside_a_sink(scores, seen, torch.tensor(900.0, dtype=torch.float64))
    assert float(p.sum()) < 1e-300 or float(p.sum()) == 0.0


def test_the_plain_rotation_keeps_lengths_and_turns_neighbours_by_position():
    rng = np.random.default_rng(2)
    x = torch.from_numpy(rng.standard_normal((5, 2, 10)))
    turned = plain.rotate_neighbours(x, torch.arange(5), 6, 100.0)
    assert torch.equal(turned[..., 6:], x[..., 6:]) and torch.equal(turned[0], x[0])
    np.testing.assert_allclose((turned ** 2).sum(-1), (x ** 2).sum(-1), rtol=1e-12)
    np.testing.assert_allclose(turned[1, 0, 0], x[1, 0, 0] * math.cos(1.0) - x[1, 0, 1] * math.sin(1.0), rtol=1e-12)


def test_the_plain_router_weighs_by_a_softmax_over_the_chosen():
    h = torch.tensor([[1.0, 0.0]], dtype=torch.float64)
    eye = torch.eye(2, dtype=torch.float64)
    w = {"router": torch.tensor([[2.0, 0.0], [1.0, 0.0], [5.0, 0.0]], dtype=torch.float64),
         "router.b": torch.tensor([0.0, 3.0, -9.0], dtype=torch.float64)}
    for e in range(3):
        w.update({f"e{e}.gate": eye, f"e{e}.up": eye, f"e{e}.down": (e + 1.0) * eye})
    out = plain.routed_experts(h, w, {"router": {"experts": 3, "top": 2}})
    # numbers 2, 4, -4: experts 1 and 0, by e^4 and e^2
    one = plain.swish(torch.tensor(1.0, dtype=torch.float64))
    share = math.exp(4.0) / (math.exp(4.0) + math.exp(2.0))
    np.testing.assert_allclose(out[0], [one * (2.0 * share + 1.0 * (1 - share)), 0.0], rtol=1e-12)
