"""Zatinex written out plainly: one function per mechanism, float64 on the CPU, a sequence at a time, token loops where a
loop says it best.  Shares no code with the package; the tests compare the package's kernels and engine with these
functions.

A model is (config, tensors): the configuration as a dictionary and the checkpoint's tensors by name.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def sigmoid(v):
    return 1.0 / (1.0 + torch.exp(-v))


def swish(v):
    return v * sigmoid(v)


def rms_divide(x, eps):
    """x over the root of (its mean square plus eps), along the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, gain, eps):
    return rms_divide(x, eps) * gain


def turn_rates(dims, base, scaling=None):
    """(the dims / 2 frequencies, the factor on both cosine and sine).  With a scaling, frequencies whose waves turn
    more than `fast` times within `original` positions stay, those that turn less than `slow` times are divided by
    `factor`, and a straight line over the pair's index joins the two."""
    rates = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return rates, 1.0
    factor, original = scaling["factor"], scaling["original"]

    def index_of(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(scaling["fast"])), 0)
    hi = min(math.ceil(index_of(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(rates):
        slowed = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * slowed + f * (1.0 - slowed))
    return out, 0.1 * math.log(factor) + 1.0


def rotate_neighbours(x, positions, rot):
    """x [tokens, vectors, length]: channels (2i, 2i + 1) of every vector, i < dims / 2, are the plane that the token's
    position turns; the channels from dims on stay."""
    dims = rot["dims"]
    out = x.clone()
    if dims == 0:
        return out
    rates, size = turn_rates(dims, rot["base"], rot.get("scaling"))
    for i, rate in enumerate(rates):
        angle = positions.to(F64) * rate
        c, s = size * torch.cos(angle)[:, None], size * torch.sin(angle)[:, None]
        even, odd = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = even * c - odd * s
        out[..., 2 * i + 1] = odd * c + even * s
    return out


def short_convolution(u, taps):
    """u [tokens, channels] from the sequence's first token, taps [channels, T]: the newest input takes the last tap."""
    n, count = u.shape[0], taps.shape[1]
    out = torch.zeros_like(u)
    for t in range(n):
        for j in range(count):
            source = t - count + 1 + j
            if source >= 0:
                out[t] += taps[:, j] * u[source]
    return out


def causal_softmax(scores):
    n = scores.shape[-1]
    seen = torch.ones(n, n).tril().bool()
    return torch.softmax(scores.masked_fill(~seen, float("-inf")), -1)


def two_map_share(w, offset):
    """The share of the second map that is taken away from the first."""
    return torch.exp((w["lq1"] * w["lk1"]).sum()) - torch.exp((w["lq2"] * w["lk2"]).sum()) + offset


def combine_maps(first, second, share, offset, eps):
    """[..., vdim] outputs of a head's two maps."""
    return rms_divide(first - share * second, eps) * (1.0 - offset)


def differential_qkv(h, w, m, eps):
    """Queries [tokens, heads, 2, dim], keys [tokens, kv_heads, 2, dim], values [tokens, kv_heads, vdim]."""
    n = h.shape[0]
    positions = torch.arange(n)
    made = {}
    for name in "qkv":
        u = h @ w[name].T + w[name + ".b"]
        made[name] = short_convolution(u, w[name + ".conv"])
    out = []
    for name, heads in (("q", m["heads"]), ("k", m["kv_heads"])):
        x = rms_norm(made[name].reshape(n, heads * 2, m["dim"]), w[name + ".norm"], eps)
        out.append(rotate_neighbours(x, positions, m["rot"]).reshape(n, heads, 2, m["dim"]))
    return (*out, made["v"].reshape(n, m["kv_heads"], m["vdim"]))


def differential_attention(h, w, m, eps):
    """h [tokens, width] of one sequence from its first token; w: the mixer's tensors by short name."""
    n, heads = h.shape[0], m["heads"]
    q, k, v = differential_qkv(h, w, m, eps)
    share = two_map_share(w, m["diff"])
    out = torch.zeros(n, heads, m["vdim"], dtype=F64)
    for head in range(heads):
        g = head // (heads // m["kv_heads"])
        maps = [causal_softmax(q[:, head, i] @ k[:, g, i].T * m["scale"]) @ v[:, g] for i in range(2)]
        out[:, head] = combine_maps(maps[0], maps[1], share, m["diff"], eps)
    return out.reshape(n, -1) @ w["o"].T


def gated_recurrence(q, k, v, alpha, state):
    """One head, token by token: q, k, alpha [tokens, dim], v [tokens, vdim], state [dim, vdim]."""
    outs = []
    for t in range(q.shape[0]):
        state = alpha[t][:, None] * state + k[t][:, None] * v[t][None, :]
        outs.append(state.T @ q[t])
    return torch.stack(outs), state


def gated_linear_attention(h, w, m, eps, states=None):
    """Returns (the mixer's output, the heads' states after the last token)."""
    n, heads, dim, vdim = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).reshape(n, heads, dim) * dim ** -0.5
    k = (h @ w["k"].T).reshape(n, heads, dim)
    v = (h @ w["v"].T).reshape(n, heads, vdim)
    z = (h @ w["a1"].T) @ w["a2"].T + w["a2.b"]
    alpha = (sigmoid(z) ** (1.0 / m["tau"])).reshape(n, heads, dim)
    states = torch.zeros(heads, dim, vdim, dtype=F64) if states is None else states.clone()
    out = torch.zeros(n, heads, vdim, dtype=F64)
    for i in range(heads):
        out[:, i], states[i] = gated_recurrence(q[:, i], k[:, i], v[:, i], alpha[:, i], states[i])
    mixed = rms_norm(out, w["norm"], eps).reshape(n, heads * vdim) * swish(h @ w["g"].T)
    return mixed @ w["o"].T, states


def latent_rows(h, w, m, eps):
    """What a layer with a latent of its own hands to itself and to later layers: the normed latent and the turned key
    part that all heads share."""
    n, rank = h.shape[0], m["kv_rank"]
    down = h @ w["dkv"].T
    shared = rotate_neighbours(down[:, rank:].reshape(n, 1, m["rot_dim"]), torch.arange(n), m["rot"])[:, 0]
    return rms_norm(down[:, :rank], w["dkv.norm"], eps), shared


def latent_attention(h, w, m, eps, rows):
    n = h.shape[0]
    heads, dim, turned, vdim = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, shared = rows
    low = rms_norm(h @ w["dq"].T, w["dq.norm"], eps)
    q = (low @ w["uq"].T).reshape(n, heads, dim + turned)
    q_turned = rotate_neighbours(q[..., dim:], torch.arange(n), m["rot"])
    k = (c @ w["uk"].T).reshape(n, heads, dim)
    v = (c @ w["uv"].T).reshape(n, heads, vdim)
    gate = sigmoid(h @ w["g"].T)                                                # [tokens, heads]
    out = torch.zeros(n, heads, vdim, dtype=F64)
    for head in range(heads):
        scores = (q[:, head, :dim] @ k[:, head].T + q_turned[:, head] @ shared.T) * m["scale"]
        out[:, head] = causal_softmax(scores) @ v[:, head] * gate[:, head:head + 1]
    return out.reshape(n, heads * vdim) @ w["o"].T


def feed_forward(h, w):
    return (swish(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def as_f64(value):
    return value.to(F64) if isinstance(value, torch.Tensor) else torch.as_tensor(value, dtype=F64)


def layer_tensors(tensors, i, part):
    prefix = f"l{i}.{part}."
    return {k[len(prefix):]: as_f64(v) for k, v in tensors.items() if k.startswith(prefix)}


def forward(config, tensors, tokens, keep_layers=False):
    """Logits [tokens, vocab] of one sequence (and the stream after every layer)."""
    eps = config["norm"]["eps"]
    x = as_f64(tensors["embed"])[torch.tensor(tokens)]
    stream, latents = [], {}
    for i, layer in enumerate(config["layers"]):
        w, m = layer_tensors(tensors, i, "mix"), layer["mixer"]
        h = rms_norm(x, as_f64(tensors[f"l{i}.norm1"]), eps)
        if layer["type"] == "attention":
            mixed = differential_attention(h, w, m, eps)
        elif layer["type"] == "gla":
            mixed, _ = gated_linear_attention(h, w, m, eps)
        else:
            owner = m.get("kv_from")
            if owner is None:
                latents[i] = latent_rows(h, w, m, eps)
            mixed = latent_attention(h, w, m, eps, latents[i if owner is None else owner])
        x = x + mixed
        if layer.get("mlp") is not None:
            h = rms_norm(x, as_f64(tensors[f"l{i}.norm2"]), eps)
            x = x + feed_forward(h, layer_tensors(tensors, i, "mlp"))
        stream.append(x.clone())
    logits = rms_norm(x, as_f64(tensors["final.norm"]), eps) @ as_f64(tensors["head"]).T
    return (logits, torch.stack(stream)) if keep_layers else logits.numpy()
