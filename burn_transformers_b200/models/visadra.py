"""Visadra as a plan of parts: a scaled token embedding; layers whose norm stands on the sublayers' outputs, x +
norm(sublayer(x)), every norm an RMS norm with one number for a gain; the mixer is either a minimal GRU (a gated average
whose gate reads only the current token) or attention over a low-rank latent with a rotated shared key part and a sink
in the softmax; the feed-forward is a gated dense one or routed experts (softmax over the chosen) beside a shared one; a
final norm and a scaled, untied readout.

Checkpoint names: `embed`, `l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.{z,z.b,x,x.b,g,o}` (minimal GRU),
`l<i>.mix.{q,dkv,dkv.norm,uk,uv,sink,o}` (latent attention), `l<i>.mlp.{gate,up,down}` (dense),
`l<i>.mlp.{router,router.b,e<j>.{gate,up,down},shared.{gate,up,down}}` (experts), `final.norm`, `head`; matrices are
stored [out, in].  Projections that read the same input are one product here: their rows are laid end to end when the
weights are loaded.
"""
from __future__ import annotations

from ..config.registry import Architecture, register_architecture
from ..config.visadra import RECURRENT_TYPES, VisadraConfig
from ..engine.model import UNBOUNDED_CONTEXT, LayerCall, ModelPlan
from ..parts import (GatedFeedForward, InterleavedRotary, LatentAttention, LinearReadout, MinGru, NoPositions,
                     OutputNormBlock, RmsNorm, RoutedFeedForward, TokenEmbedding)
from ..weights.spec import Concat, Stored

ROUNDED_STREAM = "rounded_stream"      # the step tensor in which a layer hands the stream, rounded, to the next layer


def _norm(names, name, width, eps):
    norm = RmsNorm(width, eps, one_gain=True)
    names[name] = (norm, "weight")
    return norm


def _min_gru(names, sources, p, width, m, std):
    inner = m["width"]
    mixer = MinGru(width, inner, init_std=std, out_init_std=inner ** -0.5)
    names.update({p + "in": (mixer, "in.weight"), p + "b": (mixer, "bias"), p + "o": (mixer, "out.weight")})
    sources[p + "in"] = Concat((Stored(p + "z"), Stored(p + "x"), Stored(p + "g")), 0, (inner,) * 3)
    sources[p + "b"] = Concat((Stored(p + "z.b"), Stored(p + "x.b")), 0, (inner,) * 2)
    return mixer


def _latent_attention(names, sources, p, width, m, eps, std):
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    mixer = LatentAttention(width, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["scale"], eps,
                            InterleavedRotary(rot["dims"], rot["base"]), sink=True, gate=False, init_std=std,
                            out_init_std=(m["heads"] * m["vdim"]) ** -0.5)
    names.update({p + "in": (mixer, "in.weight"), p + "dkv.norm": (mixer, "latent_norm.weight"),
                  p + "uk": (mixer, "uk.weight"), p + "uv": (mixer, "uv.weight"), p + "sink": (mixer, "sink"),
                  p + "o": (mixer, "out.weight")})
    sources[p + "in"] = Concat((Stored(p + "q"), Stored(p + "dkv")), 0, (mixer.q_width, mixer.latent_width))
    return mixer


def _gated(names, sources, p, width, inner, std):
    part = GatedFeedForward(width, inner, "swish", init_std=std, down_init_std=inner ** -0.5)
    names.update({p + "gate_up": (part, "gate_up.weight"), p + "down": (part, "down.weight")})
    sources[p + "gate_up"] = Concat((Stored(p + "gate"), Stored(p + "up")), 0, (inner, inner))
    return part


def _routed(names, sources, p, width, mlp, std):
    router, inner, n = mlp["router"], mlp["expert"]["ff"], mlp["router"]["experts"]
    shared = None
    if mlp.get("shared") is not None:
        shared = _gated(names, sources, p + "shared.", width, mlp["shared"]["ff"], std)
    part = RoutedFeedForward(width, n, router["top"], inner, activation="swish", router="softmax_of_chosen",
                             logit_bias=True, shared=shared, init_std=std)
    names.update({p + "router": (part, "router.weight"), p + "router.b": (part, "router.bias"),
                  p + "experts.gate_up": (part, "in.weight"), p + "experts.down": (part, "out.weight")})
    sources[p + "experts.gate_up"] = Concat(tuple(Stored(f"{p}e{j}.{half}") for j in range(n) for half in ("gate", "up")),
                                            0, (inner,) * (2 * n))
    sources[p + "experts.down"] = Concat(tuple(Stored(f"{p}e{j}.down") for j in range(n)), 0, (width,) * n)
    return part


def build_visadra(config: VisadraConfig) -> ModelPlan:
    config.validate()
    width, eps = config.width, config.eps
    std = width ** -0.5
    embedding = TokenEmbedding(config.vocab, width, 1.0, scale=config.embedding_scale)
    readout = LinearReadout(config.vocab, width, config.logit_scale, init_std=std)
    names = {"embed": (embedding, "weight"), "head": (readout, "weight")}
    final_norm = _norm(names, "final.norm", width, eps)
    sources = {}
    blocks = []
    for i, layer in enumerate(config.layers):
        p = f"l{i}."
        if layer["type"] in RECURRENT_TYPES:
            mixer = _min_gru(names, sources, p + "mix.", width, layer["mixer"], std)
        else:
            mixer = _latent_attention(names, sources, p + "mix.", width, layer["mixer"], eps, std)
        norm1 = _norm(names, p + "norm1", width, eps)
        feed_forward = norm2 = None
        mlp = layer.get("mlp")
        if mlp is not None:
            feed_forward = (_gated(names, sources, p + "mlp.", width, mlp["ff"], std) if mlp["kind"] == "dense"
                            else _routed(names, sources, p + "mlp.", width, mlp, std))
            norm2 = _norm(names, p + "norm2", width, eps)
        blocks.append(OutputNormBlock(mixer, norm1, feed_forward, norm2, rows=ROUNDED_STREAM, first=i == 0,
                                      last=i == len(config.layers) - 1))
    # (a layer without a feed-forward has no use for a second norm; a file may hold its number all the same)
    ignored = frozenset(f"l{i}.norm2" for i, layer in enumerate(config.layers) if layer.get("mlp") is None)
    return ModelPlan(config=config, embedding=embedding, positions=NoPositions(), blocks=blocks,
                     schedule=[LayerCall(i) for i in range(len(blocks))], final_norm=final_norm, readout=readout,
                     names=names, vocab=config.vocab, width=width, max_context=UNBOUNDED_CONTEXT, sources=sources,
                     ignored=ignored, step_tensors={ROUNDED_STREAM: (width, None)})


VISADRA = register_architecture(Architecture("visadra", VisadraConfig.MODEL_TYPES, VisadraConfig, build_visadra),
                                replace=True)
