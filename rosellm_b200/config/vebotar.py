"""Vebotar's typed configuration, read from the keys of its own ``config.json``.

Top level: ``vocab``, ``width``, ``norm.eps``, ``embedding.scale`` (the token rows' factor), ``streams`` (copies of the
residual stream) and ``layers``.  A layer gives ``type`` (``attention``, the design's one mixer), the mixer's sizes and
constants under ``mixer`` and its feed-forward under ``mlp`` (null for none).

Mixer: ``heads``, ``kv_heads``, ``dim`` (of a query or key vector of one map), ``vdim``, ``scale``, ``diff``, ``mask.size``
(the chunks' size; absent: all earlier keys), ``rot`` (``dims``, ``base`` and optionally ``scaling`` with ``factor``,
``original``, ``fast`` and ``slow``; absent: no positions) and ``kv_from`` (an earlier layer whose cached keys and values
this one reads; absent: its own).  Feed-forward: ``{"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"},
"shared": {"ff"}}`` (``shared`` may be absent).  Every size and constant comes from there; layers may differ from one
another in all of them.  The design has no position limit of its own: ``max_positions``, where a folder gives it, bounds
the sequences the engine plans for, else ``DEFAULT_MAX_POSITIONS``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, ClassVar

from .base import ConfigError, ModelConfig, optional, require

DEFAULT_MAX_POSITIONS = 131072
MIXER_TYPES = ("attention",)
MLP_KINDS = ("moe",)
SCALING_KEYS = ("factor", "original", "fast", "slow")


def _object(raw: Any, where: str) -> dict:
    if not isinstance(raw, dict):
        raise ConfigError(f"config.json: {where} must be an object")
    return raw


def _positive(where: str, **values) -> None:
    for name, v in values.items():
        if v <= 0:
            raise ConfigError(f"config.json: {where}.{name} must be positive")


@dataclass(frozen=True)
class RampRotationConfig:
    """``rot``: ``dims`` turned entries a vector, ``base``, and the ramp's constants (``None``: plain frequencies)."""

    dims: int
    base: float
    scaling: tuple[tuple[str, float], ...] | None = None

    @classmethod
    def from_dict(cls, raw: Any, where: str) -> "RampRotationConfig":
        raw = _object(raw, where)
        dims, base, sc = require(raw, "dims", int), require(raw, "base", float), raw.get("scaling")
        if dims < 0 or dims % 2 or base <= 0:
            raise ConfigError(f"config.json: {where}: dims must be even and not negative, base positive")
        values = None
        if sc is not None:
            sc = _object(sc, where + ".scaling")
            values = tuple((k, require(sc, k, float)) for k in SCALING_KEYS)
            _positive(where + ".scaling", **dict(values))
            if base == 1.0:
                raise ConfigError(f"config.json: {where}: a ramp needs a base other than 1")
        return cls(dims, base, values)

    def scaling_params(self) -> dict | None:
        """What ``RotaryPositions(scaling=...)`` takes."""
        return None if self.scaling is None else dict(self.scaling, kind="ramp")

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"dims": self.dims, "base": self.base}
        if self.scaling is not None:
            sc = dict(self.scaling)
            out["scaling"] = {k: int(v) if k == "original" and float(v).is_integer() else v for k, v in sc.items()}
        return out


@dataclass(frozen=True)
class DifferentialAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    chunk: int | None = None
    rot: RampRotationConfig | None = None
    kv_from: int | None = None

    @classmethod
    def from_dict(cls, raw: Any, where: str) -> "DifferentialAttentionConfig":
        raw = _object(raw, where)
        heads, dim = require(raw, "heads", int), require(raw, "dim", int)
        mask, rot = raw.get("mask"), raw.get("rot")
        out = cls(heads=heads, kv_heads=optional(raw, "kv_heads", int, heads), dim=dim, vdim=optional(raw, "vdim", int, dim),
                  scale=require(raw, "scale", float), diff=require(raw, "diff", float),
                  chunk=None if mask is None else require(_object(mask, where + ".mask"), "size", int),
                  rot=None if rot is None else RampRotationConfig.from_dict(rot, where + ".rot"),
                  kv_from=optional(raw, "kv_from", int, None))
        _positive(where, heads=out.heads, kv_heads=out.kv_heads, dim=out.dim, vdim=out.vdim)
        if out.heads % out.kv_heads:
            raise ConfigError(f"config.json: {where}: {out.heads} heads are not a multiple of {out.kv_heads} kv_heads")
        if out.chunk is not None and out.chunk <= 0:
            raise ConfigError(f"config.json: {where}.mask.size must be positive")
        if out.rot is not None and out.rot.dims > out.dim:
            raise ConfigError(f"config.json: {where}.rot.dims={out.rot.dims} exceeds dim={out.dim}")
        return out

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                               "scale": self.scale, "diff": self.diff}
        if self.chunk is not None:
            out["mask"] = {"size": self.chunk}
        if self.rot is not None:
            out["rot"] = self.rot.to_dict()
        if self.kv_from is not None:
            out["kv_from"] = self.kv_from
        return out


@dataclass(frozen=True)
class ExpertsConfig:
    """``experts`` feed-forwards of inner size ``ff`` of which a token uses ``top``; ``shared_ff``: the inner size of the
    one that every token passes (0: none)."""

    ff: int
    experts: int
    top: int
    shared_ff: int = 0

    @classmethod
    def from_dict(cls, raw: Any, where: str) -> "ExpertsConfig":
        raw = _object(raw, where)
        kind = require(raw, "kind", str)
        if kind not in MLP_KINDS:
            raise ConfigError(f"config.json: {where}.kind={kind!r}; the design's feed-forwards: {MLP_KINDS}")
        router, shared = _object(raw.get("router"), where + ".router"), raw.get("shared")
        out = cls(ff=require(_object(raw.get("expert"), where + ".expert"), "ff", int),
                  experts=require(router, "experts", int), top=require(router, "top", int),
                  shared_ff=0 if shared is None else require(_object(shared, where + ".shared"), "ff", int))
        _positive(where, ff=out.ff, experts=out.experts, top=out.top)
        if shared is not None:
            _positive(where + ".shared", ff=out.shared_ff)
        if out.top > out.experts:
            raise ConfigError(f"config.json: {where}.router: top={out.top} of {out.experts} experts")
        return out

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}
        if self.shared_ff:
            out["shared"] = {"ff": self.shared_ff}
        return out


@dataclass(frozen=True)
class VebotarLayerConfig:
    type: str
    mixer: DifferentialAttentionConfig
    mlp: ExpertsConfig | None

    def to_dict(self) -> dict[str, Any]:
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass(frozen=True)
class VebotarConfig(ModelConfig):
    architecture: ClassVar[str] = "Vebotar"

    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    streams: int
    layers: tuple[VebotarLayerConfig, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_id: int | None = None

    def __post_init__(self) -> None:
        if self.vocab <= 0 or self.width <= 0 or self.max_positions <= 0 or not self.layers:
            raise ConfigError("config.json: vocab, width and max_positions must be positive and layers non-empty")
        if self.width % 8:
            raise ConfigError(f"config.json: width={self.width}: the products read rows in 16-byte pieces, so the "
                              "width must be a multiple of 8")
        if self.norm_eps <= 0:
            raise ConfigError("config.json: norm.eps must be positive")
        if self.streams <= 0:
            raise ConfigError("config.json: streams must be positive")
        for i, lc in enumerate(self.layers):
            j, m = lc.mixer.kv_from, lc.mixer
            if j is None:
                continue
            if not 0 <= j < i or self.layers[j].mixer.kv_from is not None:
                raise ConfigError(f"config.json: layers[{i}].mixer.kv_from={j}: an earlier layer with keys and values of its own")
            src = self.layers[j].mixer
            if (src.kv_heads, src.dim, src.vdim) != (m.kv_heads, m.dim, m.vdim):
                raise ConfigError(f"config.json: layers[{i}] reads the keys and values of layer {j}, which have other sizes")

    @classmethod
    def from_dict(cls, raw: dict[str, Any]) -> "VebotarConfig":
        norm = _object(raw.get("norm"), "norm")
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list):
            raise ConfigError("config.json: layers must be a list")
        layers = []
        for i, lr in enumerate(layers_raw):
            where = f"layers[{i}]"
            lr = _object(lr, where)
            kind = require(lr, "type", str)
            if kind not in MIXER_TYPES:
                raise ConfigError(f"config.json: {where}.type={kind!r}; the design's mixers: {MIXER_TYPES}")
            mlp = lr.get("mlp")
            layers.append(VebotarLayerConfig(kind, DifferentialAttentionConfig.from_dict(lr.get("mixer"), where + ".mixer"),
                                             None if mlp is None else ExpertsConfig.from_dict(mlp, where + ".mlp")))
        embedding = raw.get("embedding")
        return cls(
            vocab=require(raw, "vocab", int), width=require(raw, "width", int), norm_eps=require(norm, "eps", float),
            embedding_scale=1.0 if embedding is None else optional(_object(embedding, "embedding"), "scale", float, 1.0),
            streams=require(raw, "streams", int), layers=tuple(layers),
            max_positions=optional(raw, "max_positions", int, DEFAULT_MAX_POSITIONS),
            eos_token_id=optional(raw, "eos_token_id", int, None),
        )

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {
            "architecture": self.architecture, "vocab": self.vocab, "width": self.width,
            "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale}, "streams": self.streams,
            "layers": [l.to_dict() for l in self.layers],
        }
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            out["max_positions"] = self.max_positions
        if self.eos_token_id is not None:
            out["eos_token_id"] = self.eos_token_id
        return out
