"""Typed configuration of the Pevazen design, read from its own ``config.json`` keys.

The file lists the layers one by one: each entry names its mixer (``type``) with the mixer's sizes and
constants (``mixer``) and its feed-forward (``mlp``, or null for none).  Every size and constant that can
differ between two models of the design is a field here; nothing is assumed equal between layers.
"""

from __future__ import annotations

import copy
import dataclasses
from dataclasses import dataclass, field
from typing import Any, Mapping

from .logesun_config import _positive_int
from .model_config import ConfigError, _require
from .tabisun_config import RotaryConfig, _heads, _positive

SCALING_KEYS = ("factor",)  # every frequency is divided by it


@dataclass(frozen=True)
class ChunkedAttentionConfig:
    """Softmax attention with grouped heads, rotary positions on the leading dimensions and a chunked mask.
    ``kv_from``: the layer whose keys and values are read (the layer has none of its own)."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: RotaryConfig | None
    chunk: int | None
    kv_from: int | None = None

    @classmethod
    def from_raw(cls, where: str, raw: Mapping[str, Any]) -> "ChunkedAttentionConfig":
        heads, kv_heads = _heads(where, raw)
        dim = _positive_int(where, raw, "dim")
        mask, rot = raw.get("mask") or {}, raw.get("rot")
        source = raw.get("kv_from")
        return cls(heads=heads, kv_heads=kv_heads, dim=dim, vdim=_positive_int(where, raw, "vdim"),
                   scale=_positive(where, raw, "scale"),
                   rot=RotaryConfig.from_raw(where + ".rot", rot, SCALING_KEYS, dim) if rot else None,
                   chunk=_positive_int(where + ".mask", mask, "size") if mask else None,
                   kv_from=int(source) if source is not None else None)

    def to_raw(self) -> dict[str, Any]:
        out: dict[str, Any] = dict(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim,
                                   scale=self.scale)
        if self.rot is not None:
            out["rot"] = self.rot.to_raw()
        if self.chunk is not None:
            out["mask"] = dict(size=self.chunk)
        if self.kv_from is not None:
            out["kv_from"] = self.kv_from
        return out


@dataclass(frozen=True)
class DeltaConfig:
    """The gated delta rule.  ``decay_rank`` and ``gate_rank``: the row counts of the stored low-rank products,
    zero until they are read (``PevazenConfig.with_tensor_shapes``)."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: int = 0
    gate_rank: int = 0

    @classmethod
    def from_raw(cls, where: str, raw: Mapping[str, Any]) -> "DeltaConfig":
        heads, kv_heads = _heads(where, raw)
        return cls(heads=heads, kv_heads=kv_heads, dim=_positive_int(where, raw, "dim"),
                   vdim=_positive_int(where, raw, "vdim"), conv=_positive_int(where, raw, "conv"))

    def to_raw(self) -> dict[str, Any]:
        return dict(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, conv=self.conv)


@dataclass(frozen=True)
class SideBySideConfig:
    """``parallel``: attention with turned values beside the delta rule, both on the same input."""

    left: ChunkedAttentionConfig
    right: DeltaConfig

    @classmethod
    def from_raw(cls, where: str, raw: Mapping[str, Any]) -> "SideBySideConfig":
        left = ChunkedAttentionConfig.from_raw(where + ".left", _require(raw, "left"))
        if left.rot is None or left.vdim % 2 or left.kv_from is not None:
            raise ConfigError(f"{where}.left: turned values need rot.base, an even vdim and keys of their own")
        return cls(left=left, right=DeltaConfig.from_raw(where + ".right", _require(raw, "right")))

    def to_raw(self) -> dict[str, Any]:
        return dict(left=self.left.to_raw(), right=self.right.to_raw())


MIXER_CONFIGS = {"attention": ChunkedAttentionConfig, "parallel": SideBySideConfig}


@dataclass(frozen=True)
class PevazenLayerConfig:
    type: str
    mixer: Any
    ff: int | None  # width of the dense gated feed-forward; None: the layer has none


@dataclass(frozen=True)
class PevazenConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[PevazenLayerConfig, ...]
    extra: dict = field(default_factory=dict, compare=False, repr=False)

    architecture = "Pevazen"

    def __post_init__(self) -> None:
        if self.vocab < 1 or self.width < 1 or not self.layers:
            raise ConfigError("vocab, width and the number of layers must be positive")
        if not self.norm_eps > 0:
            raise ConfigError(f"norm.eps must be positive, got {self.norm_eps!r}")
        for i, layer in enumerate(self.layers):
            source = getattr(layer.mixer, "kv_from", None)
            if source is None:
                continue
            owner = self.layers[source].mixer if 0 <= source < i else None
            if not isinstance(owner, ChunkedAttentionConfig) or owner.kv_from is not None:
                raise ConfigError(f"layer {i}: kv_from={source} must be an earlier attention layer with keys of its own")
            for name in ("heads", "kv_heads", "dim", "vdim", "rot"):
                if getattr(owner, name) != getattr(layer.mixer, name):
                    raise ConfigError(f"layer {i}: {name} differs from layer {source}'s, whose keys and values it reads")

    @classmethod
    def from_hf_config(cls, raw: Mapping[str, Any]) -> "PevazenConfig":
        names = [raw.get("architecture"), *(raw.get("architectures") or [])]
        if cls.architecture not in names:
            raise ConfigError(f"unsupported architecture: {names}")
        layers = []
        for i, entry in enumerate(_require(raw, "layers")):
            kind = _require(entry, "type")
            if kind not in MIXER_CONFIGS:
                raise ConfigError(f"layer {i}: unknown layer type {kind!r} (known: {sorted(MIXER_CONFIGS)})")
            mixer = MIXER_CONFIGS[kind].from_raw(f"layer {i} mixer", _require(entry, "mixer"))
            mlp = entry.get("mlp")
            ff = None
            if mlp:
                if _require(mlp, "kind") != "dense":
                    raise ConfigError(f"layer {i} mlp: unknown feed-forward kind {mlp['kind']!r}")
                ff = _positive_int(f"layer {i} mlp", mlp, "ff")
            layers.append(PevazenLayerConfig(kind, mixer, ff))
        return cls(vocab=int(_require(raw, "vocab")), width=int(_require(raw, "width")),
                   norm_eps=float(_require(_require(raw, "norm"), "eps")), layers=tuple(layers))

    def to_hf_config(self) -> dict[str, Any]:
        """The ``config.json`` dictionary that :meth:`from_hf_config` reads back."""
        out: dict[str, Any] = dict(architecture=self.architecture, vocab=self.vocab, width=self.width,
                                   norm=dict(eps=self.norm_eps))
        out["layers"] = [dict(type=layer.type, mixer=layer.mixer.to_raw(),
                              mlp=dict(kind="dense", ff=layer.ff) if layer.ff else None) for layer in self.layers]
        return copy.deepcopy(out)

    def with_tensor_shapes(self, shape_of) -> "PevazenConfig":
        """The sizes that only the stored tensors give: ``shape_of(name)`` is a tensor's shape.  The delta rule's decay
        and output gate go through low-rank products whose ranks are the row counts of ``a1`` and ``g1``."""
        layers = []
        for i, layer in enumerate(self.layers):
            if isinstance(layer.mixer, SideBySideConfig):
                right = layer.mixer.right
                if not right.decay_rank or not right.gate_rank:
                    right = dataclasses.replace(right, decay_rank=int(shape_of(f"l{i}.mix.right.a1")[0]),
                                                gate_rank=int(shape_of(f"l{i}.mix.right.g1")[0]))
                    layer = dataclasses.replace(layer, mixer=dataclasses.replace(layer.mixer, right=right))
            layers.append(layer)
        return dataclasses.replace(self, layers=tuple(layers))
