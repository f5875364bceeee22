"""Typed configuration of the Refolix decoder.

``config.json`` gives the vocabulary, the width, the norms' epsilon, the factor on the stream inside every norm, the
embedding's scale, the scale and the soft cap of the logits and the list of layers; each layer names the type of its mixer
(``parallel`` or ``retention``), the mixer's sizes and constants, and its feed-forward (a mixture of experts, or ``null``).  Every
size and constant is read from there; nothing about a particular model is written in the code.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from ..errors import ConfigError
from .fields import optional, required

NUMBER = (int, float)


@dataclass(frozen=True)
class RotationScaling:
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class Rotation:
    base: float
    dims: int
    scaling: RotationScaling | None = None


@dataclass(frozen=True)
class CappedAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float | None
    window: int | None
    rot: Rotation | None


@dataclass(frozen=True)
class DeltaRule:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class Parallel:
    left: CappedAttention
    right: DeltaRule


@dataclass(frozen=True)
class Retention:
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]
    rot: Rotation | None


@dataclass(frozen=True)
class Experts:
    experts: int
    top: int
    ff: int
    groups: int
    keep: int
    shared_ff: int | None


@dataclass(frozen=True)
class RefolixLayer:
    type: str
    mixer: Parallel | Retention
    mlp: Experts | None


def _positive(raw: Mapping[str, Any], name: str, where: str) -> int:
    value = required(raw, name, int)
    if value <= 0:
        raise ConfigError(f"{where}.{name} must be positive, got {value}")
    return value


def _positive_number(raw: Mapping[str, Any], name: str, where: str) -> float:
    value = float(required(raw, name, NUMBER))
    if value <= 0:
        raise ConfigError(f"{where}.{name} must be positive, got {value}")
    return value


def _cap(raw: Mapping[str, Any], name: str, where: str) -> float | None:
    value = optional(raw, name, (*NUMBER, type(None)), None)
    if value is not None and value <= 0:
        raise ConfigError(f"{where}.{name} must be positive, got {value}")
    return None if value is None else float(value)


def _rotation(mixer: Mapping[str, Any], dim: int, where: str) -> Rotation | None:
    rot = optional(mixer, "rot", (dict, type(None)), None)
    if rot is None:
        return None
    dims = required(rot, "dims", int)
    if dims < 0 or dims % 2 or dims > dim:
        raise ConfigError(f"{where}.rot.dims must be even and at most dim {dim}, got {dims}")
    base = _positive_number(rot, "base", f"{where}.rot")
    raw = optional(rot, "scaling", (dict, type(None)), None)
    scaling = None
    if raw is not None:
        if base <= 1.0:
            raise ConfigError(f"{where}.rot.base must exceed 1 where the rotation is scaled, got {base}")
        scaling = RotationScaling(*(_positive_number(raw, name, f"{where}.rot.scaling") for name in ("factor", "original", "fast", "slow")))
    return Rotation(base, dims, scaling) if dims else None


def _heads(raw: Mapping[str, Any], where: str) -> tuple[int, int]:
    heads = _positive(raw, "heads", where)
    kv_heads = _positive(raw, "kv_heads", where) if "kv_heads" in raw else heads
    if heads % kv_heads:
        raise ConfigError(f"{where}: heads {heads} is not a multiple of kv_heads {kv_heads}")
    return heads, kv_heads


def _sizes(raw: Mapping[str, Any], where: str) -> tuple[int, int]:
    dim = _positive(raw, "dim", where)
    return dim, _positive(raw, "vdim", where) if "vdim" in raw else dim


def _attention(raw: Mapping[str, Any], where: str) -> CappedAttention:
    heads, kv_heads = _heads(raw, where)
    dim, vdim = _sizes(raw, where)
    mask = optional(raw, "mask", (dict, type(None)), None) or {}
    size = optional(mask, "size", (int, type(None)), None)
    if size is not None and size <= 0:
        raise ConfigError(f"{where}.mask.size must be positive, got {size}")
    return CappedAttention(heads, kv_heads, dim, vdim, float(required(raw, "scale", NUMBER)), _cap(raw, "softcap", where), size,
                           _rotation(raw, dim, where))


def _mixer(kind: str, mixer: Mapping[str, Any], where: str) -> Parallel | Retention:
    if kind == "parallel":
        right = required(mixer, "right", dict)
        at = f"{where}.right"
        return Parallel(_attention(required(mixer, "left", dict), f"{where}.left"),
                        DeltaRule(*_heads(right, at), *_sizes(right, at), _positive(right, "conv", at)))
    if kind == "retention":
        heads = _positive(mixer, "heads", where)
        dim, vdim = _sizes(mixer, where)
        decay = required(mixer, "decay", list)
        if len(decay) != heads or any(isinstance(d, bool) or not isinstance(d, NUMBER) for d in decay):
            raise ConfigError(f"{where}.decay must hold one number per head ({heads}), got {decay}")
        return Retention(heads, dim, vdim, tuple(float(d) for d in decay), _rotation(mixer, dim, where))
    raise ConfigError(f"{where}: type {kind!r} is not a layer of this design; expected parallel or retention")


def _experts(raw: Mapping[str, Any], where: str) -> Experts:
    kind = required(raw, "kind", str)
    if kind != "moe":
        raise ConfigError(f"{where}.kind {kind!r} is not a feed-forward of this design; expected moe")
    router, expert = required(raw, "router", dict), required(raw, "expert", dict)
    experts, top = _positive(router, "experts", f"{where}.router"), _positive(router, "top", f"{where}.router")
    groups_raw = optional(router, "groups", (dict, type(None)), None)
    groups = keep = 1
    if groups_raw is not None:
        groups, keep = (_positive(groups_raw, name, f"{where}.router.groups") for name in ("count", "keep"))
    if experts % groups or keep > groups:
        raise ConfigError(f"{where}.router.groups: {groups} groups of which {keep} are kept do not fit {experts} experts")
    if top > keep * (experts // groups):
        raise ConfigError(f"{where}.router: top {top} exceeds the {keep * (experts // groups)} experts of the kept groups")
    shared = optional(raw, "shared", (dict, type(None)), None)
    return Experts(experts, top, _positive(expert, "ff", f"{where}.expert"), groups, keep,
                   _positive(shared, "ff", f"{where}.shared") if shared is not None else None)


def _layer(raw: Any, index: int) -> RefolixLayer:
    where = f"layers[{index}]"
    if not isinstance(raw, dict):
        raise ConfigError(f"{where} must be an object")
    kind = required(raw, "type", str)
    typed = _mixer(kind, required(raw, "mixer", dict), f"{where}.mixer")
    mlp = optional(raw, "mlp", (dict, type(None)), None)
    return RefolixLayer(kind, typed, None if mlp is None else _experts(mlp, f"{where}.mlp"))


@dataclass(frozen=True)
class RefolixConfig:
    vocab: int
    width: int
    eps: float
    postln_alpha: float
    embedding_scale: float
    logit_scale: float
    logit_softcap: float | None
    layers: tuple[RefolixLayer, ...]

    ARCHITECTURE = "Refolix"
    MODEL_TYPE = "refolix"
    # positions enter through rotations and masks only; the engine still wants a bound for its own bookkeeping
    MAX_POSITIONS = 1 << 24

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "RefolixConfig":
        eps = _positive_number(required(raw, "norm", dict), "eps", "norm")
        layers_raw = required(raw, "layers", list)
        if not layers_raw:
            raise ConfigError("layers must not be empty")
        layers = tuple(_layer(item, i) for i, item in enumerate(layers_raw))
        embedding = optional(raw, "embedding", (dict, type(None)), None) or {}
        return cls(_positive(raw, "vocab", "config"), _positive(raw, "width", "config"), eps,
                   float(required(raw, "postln_alpha", NUMBER)), float(optional(embedding, "scale", NUMBER, 1.0)),
                   float(optional(raw, "logit_scale", NUMBER, 1.0)), _cap(raw, "logit_softcap", "config"), layers)

    def validate_context_length(self, max_seq_len: int) -> None:
        if max_seq_len <= 0:
            raise ConfigError(f"max_seq_len must be positive, got {max_seq_len}")
        if max_seq_len > self.MAX_POSITIONS:
            raise ConfigError(f"max_seq_len {max_seq_len} exceeds the engine's bound {self.MAX_POSITIONS}")
