"""Typed configuration of the Fumolorn decoder.

``config.json`` gives the vocabulary, the width, the norms' epsilon, the factor on every sublayer's output, the embedding's
scale and bigram hash, the soft cap on the logits and the list of layers; each layer names the type of its mixer
(``latent_attention``, ``mlstm`` or ``gla``), the mixer's sizes and constants, and its feed-forward (dense, or ``null``).  Every
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
class LatentAttention:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    q_rank: int          # 0: not in config.json; the stored shape of ``dq`` gives it
    scale: float
    rot_base: float
    rot_dims: int
    rot_scaling: RotationScaling | None


@dataclass(frozen=True)
class MatrixMemory:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class GatedLinear:
    heads: int
    dim: int
    vdim: int
    tau: float


@dataclass(frozen=True)
class Dense:
    ff: int


@dataclass(frozen=True)
class FumolornLayer:
    type: str
    mixer: LatentAttention | MatrixMemory | GatedLinear
    mlp: Dense | None


@dataclass(frozen=True)
class Bigram:
    buckets: int
    mul_prev: int
    mul_cur: int


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


def _rotation(mixer: Mapping[str, Any], rot_dim: int, where: str) -> tuple[float, int, RotationScaling | None]:
    rot = optional(mixer, "rot", (dict, type(None)), None)
    if rot is None:
        if rot_dim > 0:
            raise ConfigError(f"{where}: rot_dim {rot_dim} needs a rot entry with base and dims")
        return 1.0, 0, None
    dims = required(rot, "dims", int)
    if dims < 0 or dims % 2 or dims > rot_dim:
        raise ConfigError(f"{where}.rot.dims must be even and at most rot_dim {rot_dim}, got {dims}")
    base = _positive_number(rot, "base", f"{where}.rot")
    raw = optional(rot, "scaling", (dict, type(None)), None)
    scaling = None
    if raw is not None:
        sw = f"{where}.rot.scaling"
        scaling = RotationScaling(*(_positive_number(raw, name, sw) for name in ("factor", "original", "fast", "slow")))
        if base <= 1.0:
            raise ConfigError(f"{where}.rot.base must exceed 1 where the rotation is scaled, got {base}")
    return base, dims, scaling


def _mixer(kind: str, mixer: Mapping[str, Any], where: str):
    if kind not in ("latent_attention", "mlstm", "gla"):
        raise ConfigError(f"{where}: type {kind!r} is not a layer of this design; expected latent_attention, mlstm or gla")
    heads, dim = _positive(mixer, "heads", where), _positive(mixer, "dim", where)
    vdim = _positive(mixer, "vdim", where) if "vdim" in mixer else dim
    if kind == "mlstm":
        return MatrixMemory(heads, dim, vdim, _positive_number(mixer, "gate_cap", where))
    if kind == "gla":
        return GatedLinear(heads, dim, vdim, _positive_number(mixer, "tau", where))
    rot_dim = required(mixer, "rot_dim", int)
    if rot_dim < 0:
        raise ConfigError(f"{where}.rot_dim must not be negative, got {rot_dim}")
    base, rot_dims, scaling = _rotation(mixer, rot_dim, where)
    return LatentAttention(heads, dim, rot_dim, vdim, _positive(mixer, "kv_rank", where),
                           _positive(mixer, "q_rank", where) if "q_rank" in mixer else 0, float(required(mixer, "scale", NUMBER)),
                           base, rot_dims, scaling)


def _layer(raw: Any, index: int) -> FumolornLayer:
    where = f"layers[{index}]"
    if not isinstance(raw, dict):
        raise ConfigError(f"{where} must be an object")
    kind = required(raw, "type", str)
    typed = _mixer(kind, required(raw, "mixer", dict), f"{where}.mixer")
    mlp_raw = optional(raw, "mlp", (dict, type(None)), None)
    mlp = None
    if mlp_raw is not None:
        mlp_kind = required(mlp_raw, "kind", str)
        if mlp_kind != "dense":
            raise ConfigError(f"{where}.mlp.kind {mlp_kind!r} is not a feed-forward of this design; expected dense")
        mlp = Dense(_positive(mlp_raw, "ff", f"{where}.mlp"))
    return FumolornLayer(kind, typed, mlp)


@dataclass(frozen=True)
class FumolornConfig:
    vocab: int
    width: int
    eps: float
    residual_mult: float
    embedding_scale: float
    bigram: Bigram | None
    logit_softcap: float | None
    layers: tuple[FumolornLayer, ...]

    ARCHITECTURE = "Fumolorn"
    MODEL_TYPE = "fumolorn"
    # positions enter through rotations and the causal mask only; the engine still wants a bound for its own bookkeeping
    MAX_POSITIONS = 1 << 24

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "FumolornConfig":
        eps = _positive_number(required(raw, "norm", dict), "eps", "norm")
        layers_raw = required(raw, "layers", list)
        if not layers_raw:
            raise ConfigError("layers must not be empty")
        layers = tuple(_layer(item, i) for i, item in enumerate(layers_raw))
        embedding = optional(raw, "embedding", (dict, type(None)), None) or {}
        bigram_raw = optional(embedding, "bigram", (dict, type(None)), None)
        bigram = None
        if bigram_raw is not None:
            bigram = Bigram(_positive(bigram_raw, "buckets", "embedding.bigram"), required(bigram_raw, "mul_prev", int),
                            required(bigram_raw, "mul_cur", int))
            if bigram.mul_prev < 0 or bigram.mul_cur < 0:
                raise ConfigError("embedding.bigram: the multipliers must not be negative")
        softcap = optional(raw, "logit_softcap", (*NUMBER, type(None)), None)
        if softcap is not None and softcap <= 0:
            raise ConfigError(f"logit_softcap must be positive, got {softcap}")
        return cls(_positive(raw, "vocab", "config"), _positive(raw, "width", "config"), eps,
                   float(required(raw, "residual_mult", NUMBER)), float(optional(embedding, "scale", NUMBER, 1.0)), bigram,
                   None if softcap is None else float(softcap), layers)

    def validate_context_length(self, max_seq_len: int) -> None:
        if max_seq_len <= 0:
            raise ConfigError(f"max_seq_len must be positive, got {max_seq_len}")
        if max_seq_len > self.MAX_POSITIONS:
            raise ConfigError(f"max_seq_len {max_seq_len} exceeds the engine's bound {self.MAX_POSITIONS}")
