"""Small Zatinex configurations for the tests, and helpers to write model folders (with tensors edited where random
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


def attention(heads, kv_heads, dim, vdim, conv, scale, diff, rot_dims, base, scaling=None, mlp=None):
    """scaling: (factor, original, fast, slow)"""
    rot = {"dims": rot_dims, "base": base}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                                                       "conv": conv, "scale": scale, "diff": diff, "rot": rot}}


def gla(heads, dim, vdim, tau, rank, mlp=None):
    return {"type": "gla", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "decay_rank": rank}}


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base, kv_from=None, mlp=None):
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
             "scale": scale, "rot": {"dims": rot_dim, "base": base}}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}


def model(vocab, width, eps, layers):
    return {"architecture": "Zatinex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# A: every mixer twice or more with sizes of its own, in another order than their names; latents read by one and by two
# later layers, one of them next to another owner; with and without a feed-forward behind each kind; a convolution of 4 and
# one of 2 taps, a scaled rotation and a plain one.
MIXED = model(310, 96, 1e-5, [
    gla(3, 24, 40, 16.0, 8, dense(160)),
    latent(3, 16, 8, 24, 48, 40, 0.3, 5000.0),
    attention(6, 2, 16, 24, 4, 0.3, 0.45, 12, 3000.0, (6.0, 200.0, 20.0, 0.5), dense(88)),
    latent(5, 24, 16, 16, 32, 56, 0.2, 20000.0, mlp=dense(72)),
    latent(4, 8, 8, 32, 48, 24, 0.25, 5000.0, kv_from=1, mlp=dense(120)),
    attention(2, 2, 40, 40, 2, 0.2, 0.8, 40, 500.0),
    gla(2, 56, 16, 4.0, 24),
    latent(2, 32, 8, 8, 48, 16, 0.2, 5000.0, kv_from=1),
    latent(3, 40, 16, 24, 32, 32, 0.15, 20000.0, kv_from=3, mlp=dense(56)),
])

# B: sizes that are no multiples of 8 or odd (the kernels' element-by-element branches), an odd vocabulary, a single head,
# a convolution of one tap and of six, no rotated channels, no share offset, a decay rank of one, tau one.
ODD = model(257, 72, 1e-6, [
    attention(5, 5, 6, 10, 6, 0.4, 0.0, 2, 7.0, mlp=dense(36)),
    latent(5, 6, 2, 6, 12, 10, 0.4, 7.0),
    gla(3, 11, 13, 1.0, 1, dense(50)),
    attention(3, 1, 9, 7, 1, 0.3, 0.3, 0, 10.0),
    latent(1, 10, 2, 14, 12, 9, 0.3, 300.0, kv_from=1, mlp=dense(20)),
    latent(3, 12, 0, 10, 20, 20, 0.3, 50.0),
])

# C: larger sizes (other branches of the kernels' size tables): latents of 160 and 512 channels, maps of 72 and 136 channels
# (beyond the tensor-core form's 128) with values of 128 and 200, groups of one and of six heads, recurrent heads of 136 x 72
# and 200 x 136 (several blocks a head).
LARGE = model(150, 128, 1e-5, [
    latent(6, 96, 32, 64, 160, 96, 0.12, 50000.0, mlp=dense(304)),
    attention(6, 1, 72, 128, 4, 0.12, 0.6, 64, 1e6, (16.0, 512.0, 32.0, 1.0)),
    gla(2, 136, 72, 16.0, 16),
    attention(4, 4, 136, 200, 3, 0.1, 0.5, 128, 1e4, mlp=dense(64)),
    gla(1, 200, 136, 8.0, 40),
    latent(4, 56, 16, 128, 512, 64, 0.12, 10000.0),
    latent(2, 200, 32, 130, 160, 72, 0.07, 50000.0, kv_from=0),
])

# One mechanism at a time.
ONLY_ATTENTION = model(120, 64, 1e-5, [attention(4, 2, 16, 32, 3, 0.25, 0.4, 8, 1000.0, (4.0, 64.0, 8.0, 0.5))])
ONLY_GLA = model(120, 64, 1e-5, [gla(3, 32, 24, 16.0, 8)])
ONLY_LATENT = model(120, 64, 1e-5, [latent(4, 16, 8, 24, 32, 40, 0.25, 1000.0)])
SHARED_LATENT = model(120, 64, 1e-5, [latent(4, 16, 8, 24, 32, 40, 0.25, 1000.0),
                                      latent(3, 24, 8, 16, 32, 24, 0.2, 1000.0, kv_from=0)])
ONLY_DENSE = model(120, 64, 1e-5, [gla(1, 8, 8, 16.0, 4, dense(112))])

CONFIGS = {"mixed": MIXED, "odd": ODD, "large": LARGE, "only_attention": ONLY_ATTENTION, "only_gla": ONLY_GLA,
           "only_latent": ONLY_LATENT, "shared_latent": SHARED_LATENT, "only_dense": ONLY_DENSE}


def sharp(config: dict, factor: float = 8.0) -> dict:
    """The same model with every attention score scaled up: softmaxes close to one-hot, so that a key that is lost at a
    page's border, or doubled, moves the logits by far more than rounding does."""
    out = copy.deepcopy(config)
    for entry in out["layers"]:
        if "scale" in entry["mixer"]:
            entry["mixer"]["scale"] *= factor
    return out


def make_folder(path, config: dict, *, seed=3, storage="bfloat16", edit=None) -> Path:
    """A folder with random weights.  Gains, biases and the maps' four vectors are spread out further than a random model
    has them (one that is left out or read at another place would not show otherwise); `edit` then changes tensors by
    name.  The written config.json does not give the decays' rank: the tensors' shapes do."""
    folder = bt.write_random_model(path, config, seed=seed, storage=storage)
    stored = plain_gpt2.read_safetensors(folder / "model.safetensors")
    rng = np.random.default_rng(seed + 1000)
    tensors = {}
    for name, value in stored.items():
        value = np.array(value)
        if value.ndim < 2:
            size = 1.0 if name.endswith(".b") else 0.3 if name.split(".")[-1] in ("lq1", "lk1", "lq2", "lk2") else 0.2
            value = value + rng.standard_normal(value.shape) * size
        tensors[name] = value
    if edit is not None:
        tensors = edit(tensors)
    as_matrix = {"bfloat16": torch.bfloat16, "float32": torch.float32}[storage]
    write_file(folder / "model.safetensors",
               {k: torch.tensor(v).to(as_matrix if v.ndim == 2 else torch.float32) for k, v in tensors.items()})
    data = json.loads((folder / "config.json").read_text())
    for layer in data["layers"]:
        layer["mixer"].pop("decay_rank", None)
    (folder / "config.json").write_text(json.dumps(data))
    return folder


def load_plain(folder):
    """(configuration as a dictionary, float64 weights by checkpoint name) for plain_zatinex."""
    folder = Path(folder)
    return json.loads((folder / "config.json").read_text()), plain_gpt2.read_safetensors(folder / "model.safetensors")


def prompts(config: dict, lengths, seed=0):
    rng = np.random.default_rng(seed)
    return [rng.integers(0, config["vocab"], n).tolist() for n in lengths]
