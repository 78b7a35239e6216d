"""Visadra's configuration: a list of layers, each with a recurrent or a latent-attention mixer and an optional
feed-forward, dense or of routed experts.

config.json gives every size and constant:

    {"architecture": "Visadra", "vocab": V, "width": D, "norm": {"eps": e}, "embedding": {"scale": s}, "logit_scale": l,
     "layers": [{"type": "mingru" | "mingru_2", "mixer": {"width": W},
                 "mlp": null | {"kind": "dense", "ff": F}
                             | {"kind": "moe", "expert": {"ff": F}, "router": {"experts", "top"}, "shared": {"ff": S}}},
                {"type": "latent_attention",
                 "mixer": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "rot": {"dims", "base"}},
                 "mlp": ...}]}

`mingru` and `mingru_2` are one mixer under two names (a model may give each a size of its own).  Sizes have no defaults:
one that is missing is an error that names it.  What a configuration does not mention does not exist: no `mlp` is a
layer without a feed-forward, no `shared` a layer without an expert that every token uses, no `rot` with a `rot_dim` of 0
no rotated channels, no `embedding` or `logit_scale` no scale.
"""
from __future__ import annotations

import dataclasses
from typing import ClassVar

from .base import I32_MAX, ModelConfig
from .sovozen import _is_int, _is_number

RECURRENT_TYPES = ("mingru", "mingru_2")
LAYER_TYPES = RECURRENT_TYPES + ("latent_attention",)
FEED_FORWARD_KINDS = ("dense", "moe")


@dataclasses.dataclass
class VisadraConfig(ModelConfig):
    FAMILY: ClassVar[str] = "visadra"
    MODEL_TYPES: ClassVar[tuple[str, ...]] = ("Visadra", "visadra")

    architecture: str = dataclasses.field(default="Visadra", metadata={"aliases": ("model_type",)})
    vocab: int = dataclasses.field(default=0, metadata={"aliases": ()})
    width: int = dataclasses.field(default=0, metadata={"aliases": ()})
    logit_scale: float = dataclasses.field(default=1.0, metadata={"aliases": ()})
    norm: dict = dataclasses.field(default_factory=dict, metadata={"aliases": ()})
    embedding: dict = dataclasses.field(default_factory=dict, metadata={"aliases": ()})
    layers: list = dataclasses.field(default_factory=list, metadata={"aliases": ()})

    @property
    def model_type(self) -> str:
        return self.MODEL_TYPES[0]

    @property
    def eps(self) -> float:
        return float(self.norm["eps"])

    @property
    def embedding_scale(self) -> float:
        return float(self.embedding.get("scale", 1.0))

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

    def _number(self, where: str, table: dict, name: str, *, positive: bool = False):
        if name not in table:
            self._fail(f"{where}.{name}", "is missing")
        value = table[name]
        if not _is_number(value) or (positive and value <= 0):
            self._fail(f"{where}.{name}", f"expected a finite {'positive ' if positive else ''}number, found {value!r}")

    def _check_latent(self, where: str, mixer: dict) -> None:
        self._ints(where, mixer, ("heads", "dim", "vdim", "kv_rank"))
        self._ints(where, mixer, ("rot_dim",), minimum=0)
        self._number(where, mixer, "scale")
        if mixer.get("rot") is None and mixer["rot_dim"] == 0:
            return
        rot = self._table(where, mixer, "rot")
        self._ints(f"{where}.rot", rot, ("dims",), minimum=0)
        self._number(f"{where}.rot", rot, "base", positive=True)
        if rot["dims"] % 2 or rot["dims"] > mixer["rot_dim"]:
            self._fail(f"{where}.rot.dims", f"expected an even number of at most {mixer['rot_dim']} channels, found "
                                            f"{rot['dims']}")

    def _check_mlp(self, where: str, mlp: dict) -> None:
        if not isinstance(mlp, dict) or mlp.get("kind") not in FEED_FORWARD_KINDS:
            self._fail(f"{where}.kind", f"expected one of {list(FEED_FORWARD_KINDS)}")
        if mlp["kind"] == "dense":
            self._ints(where, mlp, ("ff",))
            return
        self._ints(f"{where}.expert", self._table(where, mlp, "expert"), ("ff",))
        router = self._table(where, mlp, "router")
        self._ints(f"{where}.router", router, ("experts", "top"))
        if router["top"] > router["experts"]:
            self._fail(f"{where}.router.top", f"{router['top']} choices among {router['experts']} experts")
        if mlp.get("shared") is not None:
            self._ints(f"{where}.shared", self._table(where, mlp, "shared"), ("ff",))

    def validate(self) -> None:
        self._check_model_type(self.architecture)
        self._check_extents(("vocab", "width"))
        for name, table in (("norm", self.norm), ("embedding", self.embedding)):
            if not isinstance(table, dict):
                self._fail(name, "must be an object")
        self._number("norm", self.norm, "eps", positive=True)
        if "scale" in self.embedding:
            self._number("embedding", self.embedding, "scale")
        if not _is_number(self.logit_scale):
            self._fail("logit_scale", f"expected a finite number, found {self.logit_scale!r}")
        if not isinstance(self.layers, list) or not self.layers:
            self._fail("layers", "must be a list with at least one layer")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            if not isinstance(layer, dict) or layer.get("type") not in LAYER_TYPES:
                self._fail(f"{where}.type", f"expected one of {list(LAYER_TYPES)}, found "
                                            f"{layer.get('type') if isinstance(layer, dict) else layer!r}")
            mixer = self._table(where, layer, "mixer")
            if layer["type"] in RECURRENT_TYPES:
                self._ints(f"{where}.mixer", mixer, ("width",))
            else:
                self._check_latent(f"{where}.mixer", mixer)
            if layer.get("mlp") is not None:
                self._check_mlp(f"{where}.mlp", layer["mlp"])
