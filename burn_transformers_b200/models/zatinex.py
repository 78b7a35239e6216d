"""Zatinex as a plan of parts: a token embedding; pre-norm layers (RMS norms with plain weights) whose mixer is a
differential attention (two softmax maps a head, a short convolution, normed and rotated queries and keys), a gated linear
attention (a 32-bit state whose decay is a number per key channel and token) or a latent attention whose queries come
through a latent of their own, with one output gate a head, and which may read an earlier layer's latent; a gated silu
feed-forward where a layer has one; a final norm and an untied readout.

Checkpoint names: `embed`, `l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.{q,k,v}` with `.b` and `.conv`, `l<i>.mix.{q,k}.norm`,
`l<i>.mix.{lq1,lk1,lq2,lk2,o}` (attention), `l<i>.mix.{q,k,v,g,a1,a2,a2.b,norm,o}` (gla), `l<i>.mix.{dq,dq.norm,uq,dkv,
dkv.norm,uk,uv,g,o}` (latent attention), `l<i>.mlp.{gate,up,down}`, `final.norm`, `head`; matrices are stored [out, in].
Projections that read the same input are one product here: their rows are laid end to end when the weights are loaded.
"""
from __future__ import annotations

from ..config.registry import Architecture, register_architecture
from ..config.zatinex import ZatinexConfig
from ..engine.model import UNBOUNDED_CONTEXT, LayerCall, ModelPlan
from ..parts import (DifferentialAttention, GatedFeedForward, GatedLinearAttention, InterleavedRotary, LatentAttention,
                     LinearReadout, NoPositions, PreNormBlock, RmsNorm, TokenEmbedding)
from ..weights.spec import Concat, PadBlocks, Stored


def _norm(names, name, width, eps):
    norm = RmsNorm(width, eps)
    names[name] = (norm, "weight")
    return norm


def _rotary(mixer):
    rot = mixer.get("rot") or {"dims": 0, "base": 2.0}
    scaling = rot.get("scaling")
    yarn = None if scaling is None else (scaling["factor"], scaling["original"], scaling["fast"], scaling["slow"])
    return InterleavedRotary(rot["dims"], rot["base"], yarn=yarn)


def _stack(p, pieces):
    """One matrix (or vector) out of stored ones laid end to end; pieces: (name, rows, rows with zero rows behind)."""
    parts = tuple(Stored(p + name) if rows == padded else PadBlocks(Stored(p + name), 0, rows, padded)
                  for name, rows, padded in pieces)
    return Concat(parts, 0, tuple(padded for _, _, padded in pieces))


def _differential_attention(names, sources, p, width, m, eps, std):
    mixer = DifferentialAttention(width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], m["scale"], m["diff"], eps,
                                  _rotary(m), init_std=std, out_init_std=(m["heads"] * m["vdim"]) ** -0.5)
    names.update({p + "in": (mixer, "in.weight"), p + "in.b": (mixer, "in.bias"), p + "conv": (mixer, "conv.weight"),
                  p + "q.norm": (mixer, "q_norm.weight"), p + "k.norm": (mixer, "k_norm.weight"),
                  p + "o": (mixer, "out.weight")})
    names.update({p + name: (mixer, name) for name in ("lq1", "lk1", "lq2", "lk2")})
    rows = (("q", mixer.q_width), ("k", mixer.k_width), ("v", mixer.v_width))
    for name, suffix in (("in", ""), ("in.b", ".b"), ("conv", ".conv")):
        sources[p + name] = _stack(p, [(part + suffix, n, n) for part, n in rows])
    return mixer


def _gated_linear(names, sources, p, width, m, eps, std):
    mixer = GatedLinearAttention(width, m["heads"], m["dim"], m["vdim"], m["decay_rank"], m["tau"], eps, init_std=std,
                                 out_init_std=(m["heads"] * m["vdim"]) ** -0.5)
    names.update({p + "in": (mixer, "in.weight"), p + "a2": (mixer, "decay.weight"), p + "a2.b": (mixer, "decay.bias"),
                  p + "norm": (mixer, "norm.weight"), p + "o": (mixer, "out.weight")})
    sources[p + "in"] = _stack(p, [("q", mixer.qk_width, mixer.qk_width), ("k", mixer.qk_width, mixer.qk_width),
                                   ("v", mixer.v_width, mixer.v_width), ("g", mixer.v_width, mixer.v_width),
                                   ("a1", mixer.rank, mixer.low_rows)])
    return mixer


def _latent_attention(names, sources, p, width, m, eps, std):
    owns = m.get("kv_from") is None
    mixer = LatentAttention(width, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["scale"], eps, _rotary(m),
                            owns_latent=owns, sink=False, gate="head", q_rank=m["q_rank"], init_std=std,
                            out_init_std=(m["heads"] * m["vdim"]) ** -0.5)
    names.update({p + "in": (mixer, "in.weight"), p + "dq.norm": (mixer, "q_norm.weight"), p + "uq": (mixer, "uq.weight"),
                  p + "uk": (mixer, "uk.weight"), p + "uv": (mixer, "uv.weight"), p + "o": (mixer, "out.weight")})
    pieces = [("dq", m["q_rank"], m["q_rank"]), ("g", m["heads"], mixer.gate_width)]
    if owns:
        names[p + "dkv.norm"] = (mixer, "latent_norm.weight")
        pieces.append(("dkv", mixer.latent_width, mixer.latent_width))
    sources[p + "in"] = _stack(p, pieces)
    return mixer


MIXERS = {"attention": _differential_attention, "gla": _gated_linear, "latent_attention": _latent_attention}


def build_zatinex(config: ZatinexConfig) -> ModelPlan:
    config.validate()
    for i, layer in enumerate(config.layers):
        if layer["type"] == "gla" and "decay_rank" not in layer["mixer"]:
            config._fail(f"layers[{i}].mixer.decay_rank", "is neither in the configuration nor known from a checkpoint")
    width, eps = config.width, config.eps
    std = width ** -0.5
    embedding = TokenEmbedding(config.vocab, width, 1.0)
    readout = LinearReadout(config.vocab, width, 1.0, init_std=std)
    names = {"embed": (embedding, "weight"), "head": (readout, "weight")}
    final_norm = _norm(names, "final.norm", width, eps)
    sources = {}
    blocks, schedule = [], []
    for i, layer in enumerate(config.layers):
        p, m = f"l{i}.", layer["mixer"]
        norm1 = _norm(names, p + "norm1", width, eps)
        mixer = MIXERS[layer["type"]](names, sources, p + "mix.", width, m, eps, std)
        norm2 = feed_forward = None
        if layer.get("mlp") is not None:
            inner = layer["mlp"]["ff"]
            norm2 = _norm(names, p + "norm2", width, eps)
            feed_forward = GatedFeedForward(width, inner, "swish", init_std=std, down_init_std=inner ** -0.5)
            names[p + "mlp.gate_up"] = (feed_forward, "gate_up.weight")
            names[p + "mlp.down"] = (feed_forward, "down.weight")
            sources[p + "mlp.gate_up"] = _stack(p, [("mlp.gate", inner, inner), ("mlp.up", inner, inner)])
        blocks.append(PreNormBlock(norm1, mixer, norm2, feed_forward))
        schedule.append(LayerCall(i, cache=m.get("kv_from")))
    # a layer without a feed-forward may still have its second norm stored
    ignored = frozenset(f"l{i}.norm2" for i, layer in enumerate(config.layers) if layer.get("mlp") is None)
    return ModelPlan(config=config, embedding=embedding, positions=NoPositions(), blocks=blocks, schedule=schedule,
                     final_norm=final_norm, readout=readout, names=names, vocab=config.vocab, width=width,
                     max_context=UNBOUNDED_CONTEXT, sources=sources, ignored=ignored)


ZATINEX = register_architecture(Architecture("zatinex", ZatinexConfig.MODEL_TYPES, ZatinexConfig, build_zatinex),
                                replace=True)
