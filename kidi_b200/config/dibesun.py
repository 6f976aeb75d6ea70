"""Typed configuration of Dibesun, read from the model's own config.json keys.

    architecture: "Dibesun"        vocab, width, embedding: {scale}, norm: {eps, groups}
    layers: [{type: "parallel", mixer: {left, right, left_scale, right_scale}, mlp: null | {...}}, ...]

`left` is an attention with sigmoid weights (heads, kv_heads, dim, vdim, scale and, each optional, softcap and mask:
{size}: runs of positions that see each other; absent: every earlier token), `right` a linear attention (heads, dim,
vdim, decay: one number per head). `mlp` is {kind: "dense", ff} or {kind: "moe", expert: {ff}, router: {experts, top},
shared: {ff}} with `shared` optional. `embedding.scale` and `norm.groups` default to 1. `max_positions` is optional (the
longest sequence that is served; default 65,536). A missing or ill-typed key is INVALID_MANIFEST naming the key.
"""
from __future__ import annotations

import dataclasses
import math
from typing import Any, Mapping, Optional, Tuple

from ..errors import invalid_manifest, unsupported
from .reader import ConfigReader

PARALLEL = "parallel"
DEFAULT_MAX_POSITIONS = 65536


@dataclasses.dataclass(frozen=True)
class SigmoidAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: Optional[float] = None
    chunk: Optional[int] = None           # None: every earlier token is seen

    @classmethod
    def read(cls, mixer: ConfigReader) -> "SigmoidAttention":
        mask = mixer.child("mask")
        return cls(heads=mixer.integer("heads"), kv_heads=mixer.integer("kv_heads"), dim=mixer.integer("dim"),
                   vdim=mixer.integer("vdim"), scale=mixer.number("scale"),
                   softcap=mixer.number("softcap") if mixer.has("softcap") else None,
                   chunk=mask.integer("size") if mask is not None and mask.has("size") else None)

    def to_dict(self) -> dict:
        values: dict = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                        "scale": self.scale}
        if self.softcap is not None:
            values["softcap"] = self.softcap
        if self.chunk is not None:
            values["mask"] = {"size": self.chunk}
        return values

    def validate(self, where: str) -> None:
        if min(self.heads, self.kv_heads, self.dim, self.vdim) <= 0 or self.heads % self.kv_heads:
            raise invalid_manifest(f"{where}: sizes must be positive and heads a multiple of kv_heads")
        if self.softcap is not None and not self.softcap > 0:
            raise invalid_manifest(f"{where}: softcap must be positive")
        if self.chunk is not None and self.chunk <= 0:
            raise invalid_manifest(f"{where}: mask.size must be positive")


@dataclasses.dataclass(frozen=True)
class LinearAttention:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]

    @classmethod
    def read(cls, mixer: ConfigReader, where: str) -> "LinearAttention":
        decay = mixer.raw("decay")
        if not isinstance(decay, (list, tuple)) or any(isinstance(value, bool) or not isinstance(value, (int, float))
                                                       for value in decay):
            raise invalid_manifest(f"{where}: 'decay' must be a list of numbers")
        return cls(heads=mixer.integer("heads"), dim=mixer.integer("dim"), vdim=mixer.integer("vdim"),
                   decay=tuple(float(value) for value in decay))

    def to_dict(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}

    def validate(self, where: str) -> None:
        if min(self.heads, self.dim, self.vdim) <= 0:
            raise invalid_manifest(f"{where}: every size must be positive")
        if len(self.decay) != self.heads or not all(math.isfinite(value) and 0.0 <= value <= 1.0 for value in self.decay):
            raise invalid_manifest(f"{where}: decay must hold a number between 0 and 1 for every head")


@dataclasses.dataclass(frozen=True)
class DibesunFeedForward:
    ff: int                               # of the dense layer, or of an expert
    experts: Optional[int] = None         # None: a dense layer
    top: int = 0
    shared_ff: Optional[int] = None

    @classmethod
    def read(cls, mlp: ConfigReader, where: str) -> "DibesunFeedForward":
        kind = mlp.string("kind")
        if kind == "dense":
            return cls(ff=mlp.integer("ff"))
        if kind != "moe":
            raise unsupported(f"{where}: feed-forward kind '{kind}' is not supported")
        expert, router, shared = mlp.child("expert"), mlp.child("router"), mlp.child("shared")
        if expert is None or router is None:
            raise invalid_manifest(f"{where}:mlp: 'expert' and 'router' must be objects")
        return cls(ff=expert.integer("ff"), experts=router.integer("experts"), top=router.integer("top"),
                   shared_ff=shared.integer("ff") if shared is not None else None)

    def to_dict(self) -> dict:
        if self.experts is None:
            return {"kind": "dense", "ff": self.ff}
        values: dict = {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}
        if self.shared_ff is not None:
            values["shared"] = {"ff": self.shared_ff}
        return values

    def validate(self, where: str) -> None:
        if self.ff <= 0 or (self.shared_ff is not None and self.shared_ff <= 0):
            raise invalid_manifest(f"{where}: the widths of a feed-forward must be positive")
        if self.experts is not None and not 0 < self.top <= self.experts:
            raise invalid_manifest(f"{where}: router.top must lie between 1 and router.experts")


@dataclasses.dataclass(frozen=True)
class DibesunLayer:
    left: SigmoidAttention
    right: LinearAttention
    left_scale: float
    right_scale: float
    mlp: Optional[DibesunFeedForward] = None

    def to_dict(self) -> dict:
        return {"type": PARALLEL, "mixer": {"left": self.left.to_dict(), "right": self.right.to_dict(),
                                            "left_scale": self.left_scale, "right_scale": self.right_scale},
                "mlp": self.mlp.to_dict() if self.mlp is not None else None}


@dataclasses.dataclass(frozen=True)
class DibesunConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[DibesunLayer, ...]
    norm_groups: int = 1
    embedding_scale: float = 1.0
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_ids: Tuple[int, ...] = ()

    architecture = "Dibesun"

    @classmethod
    def from_dict(cls, values: Mapping[str, Any]) -> "DibesunConfig":
        reader = ConfigReader(values)
        name = reader.string("architecture", cls.architecture)
        if name != cls.architecture:
            raise invalid_manifest(f"expected architecture '{cls.architecture}', found '{name}'")
        norm, embedding = reader.child("norm"), reader.child("embedding")
        if norm is None:
            raise invalid_manifest("config.json: 'norm' must be an object")
        raw_layers = reader.raw("layers")
        if not isinstance(raw_layers, (list, tuple)) or not raw_layers:
            raise invalid_manifest("config.json: 'layers' must be a non-empty list")
        layers = []
        for index, raw in enumerate(raw_layers):
            where = f"config.json:layers[{index}]"
            layer = ConfigReader(raw, where)
            kind = layer.string("type")
            if kind != PARALLEL:
                raise unsupported(f"layers[{index}]: layer type '{kind}' is not supported")
            mixer, mlp = layer.child("mixer"), layer.child("mlp")
            left = mixer.child("left") if mixer is not None else None
            right = mixer.child("right") if mixer is not None else None
            if left is None or right is None:
                raise invalid_manifest(f"{where}: 'mixer', 'mixer.left' and 'mixer.right' must be objects")
            layers.append(DibesunLayer(
                left=SigmoidAttention.read(left), right=LinearAttention.read(right, where + ":mixer:right"),
                left_scale=mixer.number("left_scale"), right_scale=mixer.number("right_scale"),
                mlp=DibesunFeedForward.read(mlp, where) if mlp is not None else None))
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
                     layers=tuple(layers), norm_groups=norm.integer("groups", 1),
                     embedding_scale=embedding.number("scale", 1.0) if embedding is not None else 1.0,
                     max_positions=reader.integer("max_positions", DEFAULT_MAX_POSITIONS), eos_token_ids=eos_ids)
        config.validate()
        return config

    def validate(self) -> None:
        if min(self.vocab, self.width, self.max_positions) <= 0:
            raise invalid_manifest("invalid Dibesun dimensions: every size must be positive")
        if not self.norm_eps > 0:
            raise invalid_manifest("invalid Dibesun configuration: norm.eps must be positive")
        if self.norm_groups <= 0 or self.width % self.norm_groups:
            raise invalid_manifest("invalid Dibesun configuration: the width must be a multiple of norm.groups")
        for index, layer in enumerate(self.layers):
            where = f"layers[{index}]"
            layer.left.validate(where + ":left")
            layer.right.validate(where + ":right")
            if layer.mlp is not None:
                layer.mlp.validate(where)
        if any(token < 0 or token >= self.vocab for token in self.eos_token_ids):
            raise invalid_manifest("eos_token_id lies outside the vocabulary")

    def to_dict(self) -> dict:
        """The config.json that `from_dict` reads back to an equal configuration."""
        values: dict = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                        "embedding": {"scale": self.embedding_scale},
                        "norm": {"eps": self.norm_eps, "groups": self.norm_groups},
                        "layers": [layer.to_dict() for layer in self.layers]}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            values["max_positions"] = self.max_positions
        if self.eos_token_ids:
            values["eos_token_id"] = list(self.eos_token_ids) if len(self.eos_token_ids) > 1 else self.eos_token_ids[0]
        return values
