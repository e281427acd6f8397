"""Kugadra's typed configuration, read from the keys of its own ``config.json``.

Top level: ``vocab``, ``width``, ``norm.eps``, ``embedding.scale`` (the token rows' factor), ``logit_softcap`` (the smooth
bound of the logits) and ``layers``.  A layer gives ``type`` (its mixer: ``lightning`` or ``latent_attention``), the mixer's
sizes and constants under ``mixer`` and its feed-forward under ``mlp`` (null for none; ``{"kind": "dense", "ff"}``; or
``{"kind": "moe", "expert": {"ff"}, "router": {"experts", "top", "scale"}, "shared": {"ff"}}``, ``shared`` may be absent).

Mixer keys.  ``lightning``: ``heads``, ``dim``, ``vdim``, ``decay`` (a factor per head).  ``latent_attention``: ``heads``,
``dim``, ``rot_dim``, ``vdim``, ``kv_rank``, ``q_rank``, ``scale``, ``rot`` (``base``, optionally ``scaling`` with ``factor``,
``original``, ``fast`` and ``slow``; its ``dims`` is ``rot_dim``) and ``kv_from`` (an earlier layer whose cached latents and
turned key parts this one reads; absent: its own).  Every size and constant comes from there; layers may differ from one
another in all of them.  The design has no position limit of its own: ``max_positions``, where a folder gives it, bounds
the sequences the engine plans for, else ``DEFAULT_MAX_POSITIONS``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, ClassVar

from .base import ConfigError, ModelConfig, optional, require

DEFAULT_MAX_POSITIONS = 131072
MIXER_TYPES = ("lightning", "latent_attention")
MLP_KINDS = ("dense", "moe")
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
class LightningConfig:
    """``lightning``: linear attention whose state decays by one factor a head."""

    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]

    kv_from: ClassVar[int | None] = None

    @classmethod
    def from_dict(cls, raw: Any, where: str) -> "LightningConfig":
        raw = _object(raw, where)
        heads, decay = require(raw, "heads", int), raw.get("decay")
        if not isinstance(decay, list) or len(decay) != heads or any(
                isinstance(d, bool) or not isinstance(d, (int, float)) or not 0.0 <= d <= 1.0 for d in decay):
            raise ConfigError(f"config.json: {where}.decay: a list of {heads} factors between 0 and 1, one a head")
        out = cls(heads=heads, dim=require(raw, "dim", int), vdim=optional(raw, "vdim", int, require(raw, "dim", int)),
                  decay=tuple(float(d) for d in decay))
        _positive(where, heads=out.heads, dim=out.dim, vdim=out.vdim)
        return out

    def to_dict(self) -> dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}


@dataclass(frozen=True)
class LatentConfig:
    """``latent_attention``: per head ``dim`` plain and ``rot_dim`` turned query/key entries and values of ``vdim``; a
    key/value latent of ``kv_rank`` and a query latent of ``q_rank``.  ``rot_scaling``: the ramp's constants (``None``: plain
    frequencies)."""

    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    rot_base: float
    rot_scaling: tuple[tuple[str, float], ...] | None = None
    kv_from: int | None = None

    @classmethod
    def from_dict(cls, raw: Any, where: str) -> "LatentConfig":
        raw = _object(raw, where)
        dim, rot_dim = require(raw, "dim", int), optional(raw, "rot_dim", int, 0)
        base, scaling = 10000.0, None
        if rot_dim < 0 or rot_dim % 2:
            raise ConfigError(f"config.json: {where}.rot_dim must be even and not negative")
        if rot_dim:
            rot = _object(raw.get("rot"), where + ".rot")
            base, sc = require(rot, "base", float), rot.get("scaling")
            if optional(rot, "dims", int, rot_dim) != rot_dim:
                raise ConfigError(f"config.json: {where}.rot.dims={rot['dims']}: the turned part of {rot_dim} entries is turned whole")
            if base <= 0:
                raise ConfigError(f"config.json: {where}.rot.base must be positive")
            if sc is not None:
                sc = _object(sc, where + ".rot.scaling")
                scaling = tuple((k, require(sc, k, float)) for k in SCALING_KEYS)
                _positive(where + ".rot.scaling", **dict(scaling))
                if base == 1.0:
                    raise ConfigError(f"config.json: {where}.rot: a ramp needs a base other than 1")
        out = cls(heads=require(raw, "heads", int), dim=dim, rot_dim=rot_dim, vdim=optional(raw, "vdim", int, dim),
                  kv_rank=require(raw, "kv_rank", int), q_rank=require(raw, "q_rank", int), scale=require(raw, "scale", float),
                  rot_base=base, rot_scaling=scaling, kv_from=optional(raw, "kv_from", int, None))
        _positive(where, heads=out.heads, dim=out.dim, vdim=out.vdim, kv_rank=out.kv_rank, q_rank=out.q_rank)
        return out

    def scaling_params(self) -> dict | None:
        """What ``RotaryPositions(scaling=...)`` takes."""
        return None if self.rot_scaling is None else dict(self.rot_scaling, kind="ramp")

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim,
                               "kv_rank": self.kv_rank, "q_rank": self.q_rank, "scale": self.scale}
        if self.rot_dim:
            out["rot"] = {"dims": self.rot_dim, "base": self.rot_base}
            if self.rot_scaling is not None:
                out["rot"]["scaling"] = {k: int(v) if k == "original" and float(v).is_integer() else v for k, v in self.rot_scaling}
        if self.kv_from is not None:
            out["kv_from"] = self.kv_from
        return out


MIXER_CONFIGS = {"lightning": LightningConfig, "latent_attention": LatentConfig}


@dataclass(frozen=True)
class FeedForwardConfig:
    """``dense``: inner size ``ff``; ``moe``: ``experts`` of inner size ``ff`` of which a token uses ``top``, their weights'
    factor ``scale``, and the inner size ``shared_ff`` of the one that every token passes (0: none)."""

    kind: str
    ff: int
    experts: int = 0
    top: int = 0
    scale: float = 1.0
    shared_ff: int = 0

    @classmethod
    def from_dict(cls, raw: Any, where: str) -> "FeedForwardConfig":
        raw = _object(raw, where)
        kind = require(raw, "kind", str)
        if kind == "dense":
            out = cls("dense", require(raw, "ff", int))
            _positive(where, ff=out.ff)
        elif kind == "moe":
            router, shared = _object(raw.get("router"), where + ".router"), raw.get("shared")
            out = cls("moe", require(_object(raw.get("expert"), where + ".expert"), "ff", int),
                      experts=require(router, "experts", int), top=require(router, "top", int),
                      scale=optional(router, "scale", float, 1.0),
                      shared_ff=0 if shared is None else require(_object(shared, where + ".shared"), "ff", int))
            _positive(where, ff=out.ff, experts=out.experts, top=out.top, scale=out.scale)
            if shared is not None:
                _positive(where + ".shared", ff=out.shared_ff)
            if out.top > out.experts:
                raise ConfigError(f"config.json: {where}.router: top={out.top} of {out.experts} experts")
        else:
            raise ConfigError(f"config.json: {where}.kind={kind!r}; the design's feed-forwards: {MLP_KINDS}")
        return out

    def to_dict(self) -> dict[str, Any]:
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff}
        out: dict[str, Any] = {"kind": "moe", "expert": {"ff": self.ff},
                               "router": {"experts": self.experts, "top": self.top, "scale": self.scale}}
        if self.shared_ff:
            out["shared"] = {"ff": self.shared_ff}
        return out


@dataclass(frozen=True)
class KugadraLayerConfig:
    type: str
    mixer: "LightningConfig | LatentConfig"
    mlp: FeedForwardConfig | None

    def to_dict(self) -> dict[str, Any]:
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass(frozen=True)
class KugadraConfig(ModelConfig):
    architecture: ClassVar[str] = "Kugadra"

    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    logit_softcap: float
    layers: tuple[KugadraLayerConfig, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_id: int | None = None

    def __post_init__(self) -> None:
        if self.vocab <= 0 or self.width <= 0 or self.max_positions <= 0 or not self.layers:
            raise ConfigError("config.json: vocab, width and max_positions must be positive and layers non-empty")
        if self.width % 8:
            raise ConfigError(f"config.json: width={self.width}: the products read rows in 16-byte pieces, so the "
                              "width must be a multiple of 8")
        if self.norm_eps <= 0 or self.logit_softcap <= 0:
            raise ConfigError("config.json: norm.eps and logit_softcap must be positive")
        for i, lc in enumerate(self.layers):
            j, m = lc.mixer.kv_from, lc.mixer
            if j is None:
                continue
            if not 0 <= j < i or self.layers[j].type != "latent_attention" or self.layers[j].mixer.kv_from is not None:
                raise ConfigError(f"config.json: layers[{i}].mixer.kv_from={j}: an earlier layer of latent attention with a "
                                  "latent of its own")
            src = self.layers[j].mixer
            if (src.kv_rank, src.rot_dim) != (m.kv_rank, m.rot_dim) or \
                    (m.rot_dim and (src.rot_base, src.rot_scaling) != (m.rot_base, m.rot_scaling)):
                raise ConfigError(f"config.json: layers[{i}] reads the latents of layer {j}, which have other sizes or another rotation")

    @classmethod
    def from_dict(cls, raw: dict[str, Any]) -> "KugadraConfig":
        norm, embedding, layers_raw = _object(raw.get("norm"), "norm"), raw.get("embedding"), raw.get("layers")
        if not isinstance(layers_raw, list):
            raise ConfigError("config.json: layers must be a list")
        layers = []
        for i, lr in enumerate(layers_raw):
            where = f"layers[{i}]"
            lr = _object(lr, where)
            kind = require(lr, "type", str)
            if kind not in MIXER_CONFIGS:
                raise ConfigError(f"config.json: {where}.type={kind!r}; the design's mixers: {MIXER_TYPES}")
            mlp = lr.get("mlp")
            layers.append(KugadraLayerConfig(kind, MIXER_CONFIGS[kind].from_dict(lr.get("mixer"), where + ".mixer"),
                                             None if mlp is None else FeedForwardConfig.from_dict(mlp, where + ".mlp")))
        return cls(
            vocab=require(raw, "vocab", int), width=require(raw, "width", int), norm_eps=require(norm, "eps", float),
            embedding_scale=1.0 if embedding is None else optional(_object(embedding, "embedding"), "scale", float, 1.0),
            logit_softcap=require(raw, "logit_softcap", float), layers=tuple(layers),
            max_positions=optional(raw, "max_positions", int, DEFAULT_MAX_POSITIONS),
            eos_token_id=optional(raw, "eos_token_id", int, None),
        )

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {
            "architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
            "embedding": {"scale": self.embedding_scale}, "logit_softcap": self.logit_softcap,
            "layers": [l.to_dict() for l in self.layers],
        }
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            out["max_positions"] = self.max_positions
        if self.eos_token_id is not None:
            out["eos_token_id"] = self.eos_token_id
        return out
