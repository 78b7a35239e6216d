"""Small Visadra configurations for the tests, and helpers to write model folders (with tensors edited where random
weights would hide a fault) and to read them for the plain implementation.  The configurations differ from one another
in every size, in the order and kinds of their layers, and in which sizes happen to be equal or one."""
from __future__ import annotations

import copy
import json
from pathlib import Path

import numpy as np
import torch

import burn_transformers_b200 as bt
import plain_gpt2
from burn_transformers_b200.weights.safetensors_io import write_file


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def gru(width, mlp=None, *, kind="mingru"):
    return {"type": kind, "mixer": {"width": width}, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base, mlp=None):
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
             "rot": {"dims": rot_dim, "base": base}}
    return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}


def model(vocab, width, eps, embed_scale, logit_scale, layers):
    return {"architecture": "Visadra", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"scale": embed_scale}, "logit_scale": logit_scale, "layers": layers}


# A: layers that all differ; the two names of the recurrent mixer with sizes of their own; every kind of feed-forward
# (dense, experts with and without a shared one, none) behind both kinds of mixer.
MIXED = model(310, 96, 1e-5, 3.0, 0.7, [
    gru(136, dense(160)),
    latent(3, 16, 8, 24, 48, 0.3, 5000.0, moe(6, 2, 40, shared=72)),
    gru(64, moe(5, 3, 56, shared=24), kind="mingru_2"),
    latent(6, 24, 16, 16, 32, 0.2, 20000.0, dense(88)),
    gru(200),
    latent(2, 40, 24, 32, 64, 0.15, 300.0),
    gru(96, moe(9, 4, 32), kind="mingru_2"),
])

# B: sizes that are no multiples of 8 (the kernels' element-by-element branches), an odd vocabulary, odd recurrent
# widths, a single head, one expert a token out of one, every expert chosen, no rotated channels, scales of one.
ODD = model(257, 72, 1e-6, 1.0, 1.0, [
    latent(5, 6, 2, 6, 12, 0.4, 7.0, moe(1, 1, 20, shared=12)),
    gru(51, dense(36)),
    latent(1, 10, 6, 14, 20, 0.3, 300.0, moe(3, 3, 10)),
    gru(70, moe(7, 2, 12, shared=31), kind="mingru_2"),
    latent(3, 12, 0, 10, 20, 0.3, 50.0),
])

# C: larger sizes (other branches of the kernels' size tables): a latent of 160 and one of 512 channels, heads of 72 to 200
# channels with values of 64, 128 and 130, forty experts, a recurrent width over 1,024.
LARGE = model(150, 128, 1e-5, 2.0, 0.25, [
    latent(6, 96, 32, 64, 160, 0.12, 50000.0, moe(40, 6, 24, shared=96)),
    gru(1104, dense(304)),
    latent(4, 56, 16, 128, 512, 0.12, 10000.0, dense(64)),
    latent(2, 200, 64, 130, 72, 0.07, 1e6),
])

# One mechanism at a time.
ONLY_GRU = model(120, 64, 1e-5, 2.0, 1.0, [gru(72)])
ONLY_LATENT = model(120, 64, 1e-5, 2.0, 1.0, [latent(4, 16, 8, 24, 32, 0.25, 1000.0)])
ONLY_DENSE = model(120, 64, 1e-5, 2.0, 1.5, [gru(8, dense(112))])
ONLY_EXPERTS = model(120, 64, 1e-5, 2.0, 1.5, [gru(8, moe(6, 2, 88, shared=48), kind="mingru_2")])

CONFIGS = {"mixed": MIXED, "odd": ODD, "large": LARGE, "only_gru": ONLY_GRU, "only_latent": ONLY_LATENT,
           "only_dense": ONLY_DENSE, "only_experts": ONLY_EXPERTS}


def sharp(config: dict, factor: float = 8.0) -> dict:
    """The same model with every attention score scaled up: softmaxes close to one-hot, so that a key that is lost at a
    page's border, or doubled, moves the logits by far more than rounding does."""
    out = copy.deepcopy(config)
    for entry in out["layers"]:
        if "scale" in entry["mixer"]:
            entry["mixer"]["scale"] *= factor
    return out


def make_folder(path, config: dict, *, seed=3, storage="bfloat16", edit=None) -> Path:
    """A folder with random weights.  Gains, biases and sinks are spread out further than a random model has them (one that
    is left out or read at another place would not show otherwise); `edit` then changes tensors by name."""
    folder = bt.write_random_model(path, config, seed=seed, storage=storage)
    stored = plain_gpt2.read_safetensors(folder / "model.safetensors")
    rng = np.random.default_rng(seed + 1000)
    tensors = {}
    for name, value in stored.items():
        value = np.array(value)
        if value.ndim < 2:
            value = value + rng.standard_normal(value.shape) * (1.0 if name.endswith(("sink", ".b")) else 0.2)
        tensors[name] = value
    if edit is not None:
        tensors = edit(tensors)
    as_matrix = {"bfloat16": torch.bfloat16, "float32": torch.float32}[storage]
    write_file(folder / "model.safetensors",
               {k: torch.tensor(v).to(as_matrix if v.ndim == 2 else torch.float32) for k, v in tensors.items()})
    return folder


def load_plain(folder):
    """(configuration as a dictionary, float64 weights by checkpoint name) for plain_visadra."""
    folder = Path(folder)
    return json.loads((folder / "config.json").read_text()), plain_gpt2.read_safetensors(folder / "model.safetensors")


def prompts(config: dict, lengths, seed=0):
    rng = np.random.default_rng(seed)
    return [rng.integers(0, config["vocab"], n).tolist() for n in lengths]
