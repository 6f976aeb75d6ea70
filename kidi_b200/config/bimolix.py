"""Typed configuration of Bimolix, read from the model's own config.json keys.

    architecture: "Bimolix"        vocab, width, norm: {eps}
    layers: [{type: "retention" | "attention", mixer: {...}, mlp: null | {...}, weights_of: index (optional)}, ...]

A retention mixer has heads, dim, vdim, decay (one number per head) and rot: {base, dims}; an attention mixer heads,
kv_heads, dim, vdim (equal to dim: a value is its key before the norm), scale, bias_max and, optional, mask: {size} (runs
of positions that see each other; absent: every earlier token). `mlp` is {kind: "dense", ff} or {kind: "moe", expert: {ff,
limit}, router: {experts, top, groups: {count, keep}, scale}, shared: {ff, limit}} with `groups`, `scale` (1) and `shared`
optional. A layer with `weights_of` runs with the tensors of the layer it names and is otherwise described as that layer
is. `max_positions` is optional (the longest sequence that is served; default 65,536). A missing or ill-typed key is
INVALID_MANIFEST naming the key.
"""
from __future__ import annotations

import dataclasses
import math
from typing import Any, Mapping, Optional, Tuple, Union

from ..errors import invalid_manifest, unsupported
from .reader import ConfigReader

RETENTION, ATTENTION = "retention", "attention"
DEFAULT_MAX_POSITIONS = 65536


@dataclasses.dataclass(frozen=True)
class Retention:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot_dims: int
    rot_base: float

    kind = RETENTION

    @classmethod
    def read(cls, mixer: ConfigReader, where: str) -> "Retention":
        decay = mixer.raw("decay")
        if not isinstance(decay, (list, tuple)) or any(isinstance(value, bool) or not isinstance(value, (int, float))
                                                       for value in decay):
            raise invalid_manifest(f"{where}: 'decay' must be a list of numbers")
        rot = mixer.child("rot")
        if rot is None:
            raise invalid_manifest(f"{where}: 'rot' must be an object")
        return cls(heads=mixer.integer("heads"), dim=mixer.integer("dim"), vdim=mixer.integer("vdim"),
                   decay=tuple(float(value) for value in decay), rot_dims=rot.integer("dims"), rot_base=rot.number("base"))

    def to_dict(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay),
                "rot": {"base": self.rot_base, "dims": self.rot_dims}}

    def validate(self, where: str) -> None:
        if min(self.heads, self.dim, self.vdim) <= 0:
            raise invalid_manifest(f"{where}: every size must be positive")
        if len(self.decay) != self.heads or not all(math.isfinite(value) and 0.0 <= value <= 1.0 for value in self.decay):
            raise invalid_manifest(f"{where}: decay must hold a number between 0 and 1 for every head")
        if self.rot_dims < 0 or self.rot_dims % 2 or self.rot_dims > self.dim or not self.rot_base > 0:
            raise invalid_manifest(f"{where}: rot.dims must be even and at most dim, rot.base positive")


@dataclasses.dataclass(frozen=True)
class Attention:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    bias_max: int
    chunk: Optional[int] = None           # None: every earlier token is seen

    kind = ATTENTION

    @classmethod
    def read(cls, mixer: ConfigReader, where: str) -> "Attention":
        mask = mixer.child("mask")
        dim = mixer.integer("dim")
        if mixer.integer("vdim") != dim:
            raise invalid_manifest(f"{where}: a value is its key before the norm, so 'vdim' equals 'dim'")
        return cls(heads=mixer.integer("heads"), kv_heads=mixer.integer("kv_heads"), dim=dim, scale=mixer.number("scale"),
                   bias_max=mixer.integer("bias_max"),
                   chunk=mask.integer("size") if mask is not None and mask.has("size") else None)

    def to_dict(self) -> dict:
        values: dict = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.dim,
                        "scale": self.scale, "bias_max": self.bias_max}
        if self.chunk is not None:
            values["mask"] = {"size": self.chunk}
        return values

    def validate(self, where: str) -> None:
        if min(self.heads, self.kv_heads, self.dim) <= 0 or self.heads % self.kv_heads:
            raise invalid_manifest(f"{where}: sizes must be positive and heads a multiple of kv_heads")
        if self.bias_max <= 0:
            raise invalid_manifest(f"{where}: bias_max must be positive")
        if self.chunk is not None and self.chunk <= 0:
            raise invalid_manifest(f"{where}: mask.size must be positive")


@dataclasses.dataclass(frozen=True)
class BimolixFeedForward:
    ff: int                               # of the dense layer, or of an expert
    experts: Optional[int] = None         # None: a dense layer
    top: int = 0
    limit: float = 0.0
    groups: int = 1
    keep_groups: int = 1
    router_scale: float = 1.0
    shared_ff: Optional[int] = None
    shared_limit: float = 0.0

    @classmethod
    def read(cls, mlp: ConfigReader, where: str) -> "BimolixFeedForward":
        kind = mlp.string("kind")
        if kind == "dense":
            return cls(ff=mlp.integer("ff"))
        if kind != "moe":
            raise unsupported(f"{where}: feed-forward kind '{kind}' is not supported")
        expert, router, shared = mlp.child("expert"), mlp.child("router"), mlp.child("shared")
        if expert is None or router is None:
            raise invalid_manifest(f"{where}:mlp: 'expert' and 'router' must be objects")
        groups = router.child("groups")
        return cls(ff=expert.integer("ff"), limit=expert.number("limit"), experts=router.integer("experts"),
                   top=router.integer("top"), groups=groups.integer("count") if groups is not None else 1,
                   keep_groups=groups.integer("keep") if groups is not None else 1,
                   router_scale=router.number("scale", 1.0),
                   shared_ff=shared.integer("ff") if shared is not None else None,
                   shared_limit=shared.number("limit") if shared is not None else 0.0)

    def to_dict(self) -> dict:
        if self.experts is None:
            return {"kind": "dense", "ff": self.ff}
        router: dict = {"experts": self.experts, "top": self.top, "scale": self.router_scale}
        if (self.groups, self.keep_groups) != (1, 1):
            router["groups"] = {"count": self.groups, "keep": self.keep_groups}
        values: dict = {"kind": "moe", "expert": {"ff": self.ff, "limit": self.limit}, "router": router}
        if self.shared_ff is not None:
            values["shared"] = {"ff": self.shared_ff, "limit": self.shared_limit}
        return values

    def validate(self, where: str) -> None:
        if self.ff <= 0 or (self.shared_ff is not None and self.shared_ff <= 0):
            raise invalid_manifest(f"{where}: the widths of a feed-forward must be positive")
        if self.experts is None:
            return
        if not 0 < self.top <= self.experts:
            raise invalid_manifest(f"{where}: router.top must lie between 1 and router.experts")
        if not self.limit > 0 or (self.shared_ff is not None and not self.shared_limit > 0):
            raise invalid_manifest(f"{where}: the limit of an expert must be positive")
        if self.groups <= 0 or self.experts % self.groups or not 0 < self.keep_groups <= self.groups:
            raise invalid_manifest(f"{where}: router.groups must split the experts into equal groups and keep some of them")
        if self.keep_groups * (self.experts // self.groups) < self.top:
            raise invalid_manifest(f"{where}: the kept groups must hold at least router.top experts")


@dataclasses.dataclass(frozen=True)
class BimolixLayer:
    mixer: Union[Retention, Attention]
    mlp: Optional[BimolixFeedForward] = None
    weights_of: Optional[int] = None      # the layer whose tensors this one runs with

    def to_dict(self) -> dict:
        values = {"type": self.mixer.kind, "mixer": self.mixer.to_dict(),
                  "mlp": self.mlp.to_dict() if self.mlp is not None else None}
        if self.weights_of is not None:
            values["weights_of"] = self.weights_of
        return values


@dataclasses.dataclass(frozen=True)
class BimolixConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[BimolixLayer, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_ids: Tuple[int, ...] = ()

    architecture = "Bimolix"

    @classmethod
    def from_dict(cls, values: Mapping[str, Any]) -> "BimolixConfig":
        reader = ConfigReader(values)
        name = reader.string("architecture", cls.architecture)
        if name != cls.architecture:
            raise invalid_manifest(f"expected architecture '{cls.architecture}', found '{name}'")
        norm = reader.child("norm")
        if norm is None:
            raise invalid_manifest("config.json: 'norm' must be an object")
        raw_layers = reader.raw("layers")
        if not isinstance(raw_layers, (list, tuple)) or not raw_layers:
            raise invalid_manifest("config.json: 'layers' must be a non-empty list")
        layers = []
        for index, raw in enumerate(raw_layers):
            where = f"config.json:layers[{index}]"
            layer = ConfigReader(raw, where)
            kind, mixer, mlp = layer.string("type"), layer.child("mixer"), layer.child("mlp")
            if kind not in (RETENTION, ATTENTION):
                raise unsupported(f"layers[{index}]: layer type '{kind}' is not supported")
            if mixer is None:
                raise invalid_manifest(f"{where}: 'mixer' must be an object")
            layers.append(BimolixLayer(
                mixer=(Retention if kind == RETENTION else Attention).read(mixer, where + ":mixer"),
                mlp=BimolixFeedForward.read(mlp, where) if mlp is not None else None,
                weights_of=layer.integer("weights_of") if layer.has("weights_of") else None))
        eos = reader.raw("eos_token_id")
        if eos is None:
            eos_ids: Tuple[int, ...] = ()
        elif isinstance(eos, int) and not isinstance(eos, bool):
            eos_ids = (eos,)
        elif isinstance(eos, (list, tuple)) and all(isinstance(e, int) and not isinstance(e, bool) for e in eos):
            eos_ids = tuple(eos)
        else:
            raise invalid_manifest("'eos_token_id' must be an integer or a list of integers")
        config = cls(vocab=reader.integer("vocab"), width=reader.integer("width"), norm_eps=norm.number("eps"),
                     layers=tuple(layers), max_positions=reader.integer("max_positions", DEFAULT_MAX_POSITIONS),
                     eos_token_ids=eos_ids)
        config.validate()
        return config

    def owner(self, index: int) -> int:
        """The layer whose tensors layer `index` runs with (itself, unless it names another one)."""
        seen = []
        while self.layers[index].weights_of is not None:
            seen.append(index)
            index = self.layers[index].weights_of
            if not 0 <= index < len(self.layers) or index in seen:
                raise invalid_manifest(f"layers[{seen[0]}]: weights_of leads to no layer with tensors of its own")
        return index

    def validate(self) -> None:
        if min(self.vocab, self.width, self.max_positions) <= 0:
            raise invalid_manifest("invalid Bimolix dimensions: every size must be positive")
        if not self.norm_eps > 0:
            raise invalid_manifest("invalid Bimolix configuration: norm.eps must be positive")
        for index, layer in enumerate(self.layers):
            where = f"layers[{index}]"
            layer.mixer.validate(where)
            if layer.mlp is not None:
                layer.mlp.validate(where)
            owner = self.layers[self.owner(index)]
            if (layer.mixer, layer.mlp) != (owner.mixer, owner.mlp):
                raise invalid_manifest(f"{where}: a layer that runs with another layer's tensors is described as that layer is")
        if any(token < 0 or token >= self.vocab for token in self.eos_token_ids):
            raise invalid_manifest("eos_token_id lies outside the vocabulary")

    def to_dict(self) -> dict:
        """The config.json that `from_dict` reads back to an equal configuration."""
        values: dict = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                        "norm": {"eps": self.norm_eps}, "layers": [layer.to_dict() for layer in self.layers]}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            values["max_positions"] = self.max_positions
        if self.eos_token_ids:
            values["eos_token_id"] = list(self.eos_token_ids) if len(self.eos_token_ids) > 1 else self.eos_token_ids[0]
        return values
