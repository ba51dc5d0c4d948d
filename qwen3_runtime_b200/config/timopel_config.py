"""Typed configuration of the Timopel design, read from its own ``config.json`` keys.

The file lists the layers one by one: each entry names its mixer (``type``: ``attention``) with the mixer's sizes and
constants (``mixer``) and its feed-forward (``mlp``: ``kind`` ``dense`` or ``moe``, or null for none).  ``embedding.scale``
multiplies the token rows, ``residual_mult`` every sublayer's normed output, ``norm.eps`` belongs to every norm.  Every
size and constant that can differ between two models of the design is a field here; nothing is assumed equal between
layers, except that layers which mix values must agree in what they mix.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from .logesun_config import ExpertConfig, _positive_int
from .model_config import ConfigError, _require


@dataclass(frozen=True)
class TemperatureConfig:
    """The query of position p is multiplied by 1 + coef * ln(floor((p + 1) / every) + 1)."""

    coef: float
    every: int

    @classmethod
    def from_raw(cls, where: str, raw: Mapping[str, Any]) -> "TemperatureConfig":
        return cls(coef=float(_require(raw, "coef")), every=_positive_int(where, raw, "every"))


@dataclass(frozen=True)
class MixedValueAttentionConfig:
    """Causal attention with grouped key/value heads, normed q and k, a learned sink per head, no positions but a query
    temperature (``q_temp`` None: none); ``v_mix``: the layer's values take a learned share of the values of the first
    layer that has the flag."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    q_temp: TemperatureConfig | None = None
    v_mix: bool = False

    @classmethod
    def from_raw(cls, where: str, raw: Mapping[str, Any]) -> "MixedValueAttentionConfig":
        temp = raw.get("q_temp")
        cfg = cls(heads=_positive_int(where, raw, "heads"), kv_heads=_positive_int(where, raw, "kv_heads"),
                  dim=_positive_int(where, raw, "dim"), vdim=_positive_int(where, raw, "vdim"),
                  scale=float(_require(raw, "scale")),
                  q_temp=TemperatureConfig.from_raw(where + ".q_temp", temp) if temp else None,
                  v_mix=bool(raw.get("v_mix", False)))
        if cfg.heads % cfg.kv_heads:
            raise ConfigError(f"{where}: heads={cfg.heads} is no multiple of kv_heads={cfg.kv_heads}")
        if not cfg.scale > 0:
            raise ConfigError(f"{where}: scale must be positive")
        return cfg

    def to_raw(self) -> dict[str, Any]:
        out = dict(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, scale=self.scale,
                   v_mix=self.v_mix)
        if self.q_temp is not None:
            out["q_temp"] = dict(coef=self.q_temp.coef, every=self.q_temp.every)
        return out


@dataclass(frozen=True)
class DenseConfig:
    """One gated layer of width ``ff`` with gelu (tanh form)."""

    ff: int

    def to_raw(self) -> dict[str, Any]:
        return dict(kind="dense", ff=self.ff)


@dataclass(frozen=True)
class MoeConfig:
    """``experts`` clamped gated layers of which a token uses ``top``, weighted by the softmax over all router outputs
    at the chosen ones, made to sum to ``scale``; an optional shared one that every token uses."""

    experts: int
    top: int
    expert: ExpertConfig
    scale: float = 1.0
    shared: ExpertConfig | None = None

    def to_raw(self) -> dict[str, Any]:
        out: dict[str, Any] = dict(kind="moe", router=dict(experts=self.experts, top=self.top, scale=self.scale),
                                   expert=dict(ff=self.expert.ff, limit=self.expert.limit))
        if self.shared is not None:
            out["shared"] = dict(ff=self.shared.ff, limit=self.shared.limit)
        return out


def _mlp_from_raw(where: str, raw: Mapping[str, Any] | None):
    if not raw:
        return None
    kind = _require(raw, "kind")
    if kind == "dense":
        return DenseConfig(ff=_positive_int(where, raw, "ff"))
    if kind == "moe":
        router = _require(raw, "router")
        cfg = MoeConfig(experts=_positive_int(where + ".router", router, "experts"),
                        top=_positive_int(where + ".router", router, "top"), scale=float(router.get("scale", 1.0)),
                        expert=ExpertConfig.from_raw(where + ".expert", _require(raw, "expert")),
                        shared=ExpertConfig.from_raw(where + ".shared", raw["shared"]) if raw.get("shared") else None)
        if cfg.top > cfg.experts:
            raise ConfigError(f"{where}: top={cfg.top} exceeds experts={cfg.experts}")
        return cfg
    raise ConfigError(f"{where}: unknown feed-forward kind {kind!r} (dense or moe)")


@dataclass(frozen=True)
class TimopelLayerConfig:
    type: str
    mixer: MixedValueAttentionConfig
    mlp: DenseConfig | MoeConfig | None


@dataclass(frozen=True)
class TimopelConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[TimopelLayerConfig, ...]
    embed_scale: float = 1.0
    residual_mult: float = 1.0

    architecture = "Timopel"

    def __post_init__(self) -> None:
        if self.vocab < 1 or self.width < 1 or not self.layers:
            raise ConfigError("vocab, width and the number of layers must be positive")
        if not self.norm_eps > 0:
            raise ConfigError(f"norm.eps must be positive, got {self.norm_eps!r}")
        mixing = [(i, l.mixer.kv_heads, l.mixer.vdim) for i, l in enumerate(self.layers) if l.mixer.v_mix]
        for i, kv_heads, vdim in mixing[1:]:
            if (kv_heads, vdim) != mixing[0][1:]:
                raise ConfigError(f"layer {i} mixes {kv_heads} value heads of {vdim} with layer {mixing[0][0]}'s "
                                  f"{mixing[0][1]} of {mixing[0][2]}")

    @classmethod
    def from_hf_config(cls, raw: Mapping[str, Any]) -> "TimopelConfig":
        names = [raw.get("architecture"), *(raw.get("architectures") or [])]
        if cls.architecture not in names:
            raise ConfigError(f"unsupported architecture: {names}")
        layers = []
        for i, entry in enumerate(_require(raw, "layers")):
            kind = _require(entry, "type")
            if kind != "attention":
                raise ConfigError(f"layer {i}: unknown mixer type {kind!r} (known: attention)")
            layers.append(TimopelLayerConfig(
                kind, MixedValueAttentionConfig.from_raw(f"layer {i} mixer", _require(entry, "mixer")),
                _mlp_from_raw(f"layer {i} mlp", entry.get("mlp"))))
        return cls(vocab=_positive_int("config", raw, "vocab"), width=_positive_int("config", raw, "width"),
                   norm_eps=float(_require(_require(raw, "norm"), "eps")), layers=tuple(layers),
                   embed_scale=float((raw.get("embedding") or {}).get("scale", 1.0)),
                   residual_mult=float(raw.get("residual_mult", 1.0)))

    def to_hf_config(self) -> dict[str, Any]:
        """The ``config.json`` dictionary that :meth:`from_hf_config` reads back."""
        return dict(architecture=self.architecture, vocab=self.vocab, width=self.width, norm=dict(eps=self.norm_eps),
                    embedding=dict(scale=self.embed_scale), residual_mult=self.residual_mult,
                    layers=[dict(type=l.type, mixer=l.mixer.to_raw(), mlp=l.mlp.to_raw() if l.mlp else None)
                            for l in self.layers])

    def first_mixing_layer(self) -> int | None:
        """The layer whose values the later mixing layers take a share of."""
        return next((i for i, l in enumerate(self.layers) if l.mixer.v_mix), None)
