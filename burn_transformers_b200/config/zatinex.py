"""Zatinex's configuration: a list of layers, each with one of three mixers and an optional gated feed-forward.

config.json gives every size and constant but one:

    {"architecture": "Zatinex", "vocab": V, "width": D, "norm": {"eps": e},
     "layers": [{"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "conv", "scale", "diff",
                           "rot": {"dims", "base", "scaling": {"factor", "original", "fast", "slow"}}},
                 "mlp": null | {"kind": "dense", "ff": F}},
                {"type": "gla", "mixer": {"heads", "dim", "vdim", "tau"}, "mlp": ...},
                {"type": "latent_attention",
                 "mixer": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale", "rot": {"dims", "base"},
                           "kv_from": j}, "mlp": ...}]}

Sizes have no defaults: one that is missing is an error that names it.  What a configuration does not mention does not
exist: no `scaling` leaves the frequencies as they are, no `kv_from` is a layer with a latent of its own, no `mlp` a layer
without a feed-forward.  The rank of a gla layer's decays is the height of its tensor `a1`: `learn_shapes` takes it from the
checkpoint; a configuration for which there is no checkpoint yet gives it as the mixer's `decay_rank`.
"""
from __future__ import annotations

import dataclasses
from typing import ClassVar

from .base import I32_MAX, ModelConfig
from .sovozen import _is_int, _is_number

LAYER_TYPES = ("attention", "gla", "latent_attention")
FEED_FORWARD_KINDS = ("dense",)


@dataclasses.dataclass
class ZatinexConfig(ModelConfig):
    FAMILY: ClassVar[str] = "zatinex"
    MODEL_TYPES: ClassVar[tuple[str, ...]] = ("Zatinex", "zatinex")

    architecture: str = dataclasses.field(default="Zatinex", metadata={"aliases": ("model_type",)})
    vocab: int = dataclasses.field(default=0, metadata={"aliases": ()})
    width: int = dataclasses.field(default=0, metadata={"aliases": ()})
    norm: dict = dataclasses.field(default_factory=dict, metadata={"aliases": ()})
    layers: list = dataclasses.field(default_factory=list, metadata={"aliases": ()})

    @property
    def model_type(self) -> str:
        return self.MODEL_TYPES[0]

    @property
    def eps(self) -> float:
        return float(self.norm["eps"])

    def learn_shapes(self, shapes) -> None:
        for i, layer in enumerate(self.layers):
            shape = shapes.get(f"l{i}.mix.a1")
            if layer["type"] == "gla" and shape is not None and len(shape) == 2:
                self.layers[i] = dict(layer, mixer=dict(layer["mixer"], decay_rank=int(shape[0])))

    # ---- checks --------------------------------------------------------------------------------------------
    def _table(self, where: str, parent: dict, name: str) -> dict:
        value = parent.get(name) if isinstance(parent, dict) else None
        if not isinstance(value, dict):
            self._fail(f"{where}.{name}" if where else name, "is missing")
        return value

    def _ints(self, where: str, table: dict, names, *, minimum: int = 1):
        for name in names:
            if name not in table:
                self._fail(f"{where}.{name}", "is missing")
            value = table[name]
            if not _is_int(value) or value < minimum or value > I32_MAX:
                self._fail(f"{where}.{name}", f"expected an integer of at least {minimum}, found {value!r}")

    def _numbers(self, where: str, table: dict, names, *, positive: bool = False):
        for name in names:
            if name not in table:
                self._fail(f"{where}.{name}", "is missing")
            value = table[name]
            if not _is_number(value) or (positive and value <= 0):
                self._fail(f"{where}.{name}", f"expected a finite {'positive ' if positive else ''}number, found {value!r}")

    def _check_rotation(self, where: str, mixer: dict, most: int, scaling_allowed: bool) -> None:
        if mixer.get("rot") is None:
            return
        rot = self._table(where, mixer, "rot")
        self._ints(f"{where}.rot", rot, ("dims",), minimum=0)
        self._numbers(f"{where}.rot", rot, ("base",), positive=True)
        if rot["dims"] % 2 or rot["dims"] > most:
            self._fail(f"{where}.rot.dims", f"expected an even number of at most {most} channels, found {rot['dims']}")
        if rot.get("scaling") is not None:
            if not scaling_allowed:
                self._fail(f"{where}.rot.scaling", "this mixer's frequencies are not scaled")
            self._numbers(f"{where}.rot.scaling", self._table(f"{where}.rot", rot, "scaling"),
                          ("factor", "original", "fast", "slow"), positive=True)
            if rot["base"] <= 1:
                self._fail(f"{where}.rot.base", "must exceed one where the frequencies are scaled")

    def _check_attention(self, where: str, mixer: dict) -> None:
        self._ints(where, mixer, ("heads", "kv_heads", "dim", "vdim", "conv"))
        self._numbers(where, mixer, ("scale", "diff"))
        if mixer["heads"] % mixer["kv_heads"]:
            self._fail(f"{where}.kv_heads", f"{mixer['heads']} query heads cannot share {mixer['kv_heads']} key heads")
        self._check_rotation(where, mixer, mixer["dim"], True)

    def _check_gla(self, where: str, mixer: dict) -> None:
        self._ints(where, mixer, ("heads", "dim", "vdim"))
        self._numbers(where, mixer, ("tau",), positive=True)
        if "decay_rank" in mixer:
            self._ints(where, mixer, ("decay_rank",))

    def _check_latent(self, index: int, where: str, mixer: dict) -> None:
        self._ints(where, mixer, ("heads", "dim", "vdim", "kv_rank", "q_rank"))
        self._ints(where, mixer, ("rot_dim",), minimum=0)
        self._numbers(where, mixer, ("scale",))
        self._check_rotation(where, mixer, mixer["rot_dim"], False)
        owner = mixer.get("kv_from")
        if owner is None:
            return
        if not _is_int(owner) or not 0 <= owner < index:
            self._fail(f"{where}.kv_from", f"expected the index of an earlier layer, found {owner!r}")
        other = self.layers[owner]
        if other["type"] != "latent_attention" or other["mixer"].get("kv_from") is not None:
            self._fail(f"{where}.kv_from", f"layer {owner} has no latent of its own")
        for name in ("kv_rank", "rot_dim"):
            if other["mixer"][name] != mixer[name]:
                self._fail(f"{where}.{name}", f"{mixer[name]} differs from layer {owner}'s {other['mixer'][name]}")

    def validate(self) -> None:
        self._check_model_type(self.architecture)
        self._check_extents(("vocab", "width"))
        if not isinstance(self.norm, dict):
            self._fail("norm", "must be an object")
        self._numbers("norm", self.norm, ("eps",), positive=True)
        if not isinstance(self.layers, list) or not self.layers:
            self._fail("layers", "must be a list with at least one layer")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            if not isinstance(layer, dict) or layer.get("type") not in LAYER_TYPES:
                self._fail(f"{where}.type", f"expected one of {list(LAYER_TYPES)}, found "
                                            f"{layer.get('type') if isinstance(layer, dict) else layer!r}")
            mixer = self._table(where, layer, "mixer")
            if layer["type"] == "attention":
                self._check_attention(f"{where}.mixer", mixer)
            elif layer["type"] == "gla":
                self._check_gla(f"{where}.mixer", mixer)
            else:
                self._check_latent(i, f"{where}.mixer", mixer)
            mlp = layer.get("mlp")
            if mlp is not None:
                if not isinstance(mlp, dict) or mlp.get("kind") not in FEED_FORWARD_KINDS:
                    self._fail(f"{where}.mlp.kind", f"expected one of {list(FEED_FORWARD_KINDS)}")
                self._ints(f"{where}.mlp", mlp, ("ff",))
