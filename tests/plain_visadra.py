"""Visadra written out plainly: one function per mechanism, float64 on the CPU, a sequence at a time, token loops where a
loop says it best.  Shares no code with the package; the tests compare the package's kernels and engine with these
functions.

A model is (config, tensors): the configuration as a dictionary and the checkpoint's tensors by name.
"""
from __future__ import annotations

import torch

F64 = torch.float64


def sigmoid(v):
    return 1.0 / (1.0 + torch.exp(-v))


def swish(v):
    return v * sigmoid(v)


def rms_divide(x, eps):
    """x over the root of (its mean square plus eps), along the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_one_gain(x, gain, eps):
    """One number scales all coordinates."""
    return rms_divide(x, eps) * gain.reshape(())


def rotate_neighbours(x, positions, dims, base):
    """x [tokens, vectors, length]: channels (2i, 2i + 1) of every vector, i < dims / 2, are the plane that the token's
    position turns by position * base^(-2i / dims)."""
    out = x.clone()
    for i in range(dims // 2):
        angle = positions.to(F64) * base ** (-2.0 * i / dims)
        c, s = torch.cos(angle)[:, None], torch.sin(angle)[:, None]
        even, odd = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = even * c - odd * s
        out[..., 2 * i + 1] = odd * c + even * s
    return out


def softmax_beside_a_sink(scores, seen, sink):
    """Rows of weights over the seen keys; exp(sink) stands in the denominator too, without a key of its own."""
    scores = scores.masked_fill(~seen, float("-inf"))
    top = torch.clamp(scores.max(-1, keepdim=True).values, min=float(sink))
    grown = torch.exp(scores - top)
    return grown / (grown.sum(-1, keepdim=True) + torch.exp(sink - top))


def latent_attention(h, w, m, eps):
    """h [tokens, width] of one sequence from its first token; w: the mixer's tensors by short name."""
    n = h.shape[0]
    heads, dim, turned, vdim, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    positions = torch.arange(n)
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    q = (h @ w["q"].T).view(n, heads, dim + turned)
    down = h @ w["dkv"].T
    c = rms_divide(down[:, :rank], eps) * w["dkv.norm"]
    shared = rotate_neighbours(down[:, rank:].view(n, 1, turned), positions, rot["dims"], rot["base"])[:, 0]
    q_turned = rotate_neighbours(q[..., dim:], positions, rot["dims"], rot["base"])
    k = (c @ w["uk"].T).view(n, heads, dim)
    v = (c @ w["uv"].T).view(n, heads, vdim)
    seen = torch.ones(n, n).tril().bool()
    out = torch.zeros(n, heads, vdim, dtype=F64)
    for head in range(heads):
        scores = (q[:, head, :dim] @ k[:, head].T + q_turned[:, head] @ shared.T) * m["scale"]      # [query, key]
        out[:, head] = softmax_beside_a_sink(scores, seen, w["sink"][head]) @ v[:, head]
    return out.reshape(n, heads * vdim) @ w["o"].T


def candidate(u):
    """A monotone positive map: u + 1/2 from zero on, the logistic function below."""
    return torch.where(u >= 0, u + 0.5, sigmoid(u))


def gated_average(z, values, state):
    """The recurrence alone: token by token the state moves from where it is towards the token's value by the share z.
    Returns every state and the last one."""
    states = []
    for t in range(z.shape[0]):
        state = state + z[t] * (values[t] - state)
        states.append(state)
    return torch.stack(states), state


def minimal_gru(h, w, state=None):
    """Returns (the mixer's output, the state after the last token)."""
    share = sigmoid(h @ w["z"].T + w["z.b"])
    values = candidate(h @ w["x"].T + w["x.b"])
    state = torch.zeros(share.shape[1], dtype=F64) if state is None else state
    states, last = gated_average(share, values, state)
    return (states * swish(h @ w["g"].T)) @ w["o"].T, last


def pair_of_halves(h, w, prefix=""):
    return (swish(h @ w[prefix + "gate"].T) * (h @ w[prefix + "up"].T)) @ w[prefix + "down"].T


def routed_experts(h, w, mlp):
    """The experts with the largest router numbers (equal ones: the lower index); softmax among the chosen."""
    experts, top = mlp["router"]["experts"], mlp["router"]["top"]
    numbers = h @ w["router"].T + w["router.b"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen = sorted(range(experts), key=lambda e: (-float(numbers[t, e]), e))[:top]
        share = torch.softmax(numbers[t, chosen], 0)
        for weight, e in zip(share, chosen):
            out[t] += weight * pair_of_halves(h[t], w, f"e{e}.")
    if mlp.get("shared") is not None:
        out = out + pair_of_halves(h, w, "shared.")
    return out


def as_f64(value):
    return value.to(F64) if isinstance(value, torch.Tensor) else torch.as_tensor(value, dtype=F64)


def layer_tensors(tensors, i, part):
    prefix = f"l{i}.{part}."
    return {k[len(prefix):]: as_f64(v) for k, v in tensors.items() if k.startswith(prefix)}


def forward(config, tensors, tokens, keep_layers=False):
    """Logits [tokens, vocab] of one sequence (and the stream after every layer)."""
    eps = config["norm"]["eps"]
    x = as_f64(tensors["embed"])[torch.tensor(tokens)] * config["embedding"]["scale"]
    stream = []
    for i, layer in enumerate(config["layers"]):
        w = layer_tensors(tensors, i, "mix")
        if layer["type"] == "latent_attention":
            mixed = latent_attention(x, w, layer["mixer"], eps)
        else:
            mixed, _ = minimal_gru(x, w)
        x = x + norm_one_gain(mixed, as_f64(tensors[f"l{i}.norm1"]), eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            w = layer_tensors(tensors, i, "mlp")
            y = pair_of_halves(x, w) if mlp["kind"] == "dense" else routed_experts(x, w, mlp)
            x = x + norm_one_gain(y, as_f64(tensors[f"l{i}.norm2"]), eps)
        stream.append(x.clone())
    logits = norm_one_gain(x, as_f64(tensors["final.norm"]), eps) @ as_f64(tensors["head"]).T * config["logit_scale"]
    return (logits, torch.stack(stream)) if keep_layers else logits.numpy()
