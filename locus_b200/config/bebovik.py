"""Typed configuration of the Bebovik design.

config.json of this design is nested: the model's ``width``, ``vocab``, ``norm.eps`` (of the norms on queries and keys),
``embedding.scale`` (a factor on the embedding), ``logit_scale`` and ``logit_softcap`` (a factor on the logits and the bound
of the tanh behind it) and a list ``layers`` whose entries each give the ``type`` of their mixer, the mixer's sizes and
constants (``mixer``) and their feed-forward (``mlp``, or null for none).  Layers may differ from each other in everything.
Every size and constant is read here; nothing about a particular model is fixed in code.

Mixer ``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``mask.size`` (the chunk of positions that a
query sees; without a mask: every earlier key), ``rot`` = {``base``, ``dims``, ``scaling`` = {``factor``, ``low``, ``high``,
``original``}} (absent: no rotation, no scaling).
Feed-forward ``dense``: ``ff``, ``limit``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError, take
from .lalepel import _num, _pos, _sub


@dataclass(frozen=True)
class WavelengthScaling:
    factor: float
    low: float
    high: float
    original: float


@dataclass(frozen=True)
class ScaledRotation:
    base: float
    dims: int
    scaling: Optional[WavelengthScaling]


@dataclass(frozen=True)
class ChunkedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int                       # 0: no mask of chunks
    rot: Optional[ScaledRotation]

    kind = "attention"


@dataclass(frozen=True)
class ClampedMlpConfig:
    ff: int
    limit: float

    kind = "dense"


@dataclass(frozen=True)
class BebovikLayer:
    mixer: ChunkedAttentionConfig
    mlp: Optional[ClampedMlpConfig]


def _positive(raw: Dict[str, Any], key: str, where: str) -> float:
    v = _num(raw, key, where)
    if not v > 0:
        raise ConfigError(f"config.json: {where}{key} must be positive, got {v}")
    return v


def _rotation(m: Dict[str, Any], where: str, dim: int) -> Optional[ScaledRotation]:
    rot = _sub(m, "rot", where, optional=True)
    if rot is None:
        return None
    w = where + "rot."
    dims = _pos(rot, "dims", w)
    if dims % 2 or dims > dim:
        raise ConfigError(f"config.json: {w}dims {dims} must be even and at most {dim}")
    sc = _sub(rot, "scaling", w, optional=True)
    scaling = None
    if sc is not None:
        s = w + "scaling."
        scaling = WavelengthScaling(factor=_positive(sc, "factor", s), low=_positive(sc, "low", s),
                                    high=_positive(sc, "high", s), original=_positive(sc, "original", s))
        if scaling.high < scaling.low:
            raise ConfigError(f"config.json: {s}high {scaling.high} must not be below low {scaling.low}")
    return ScaledRotation(base=_positive(rot, "base", w), dims=dims, scaling=scaling)


def _attention(m: Dict[str, Any], where: str) -> ChunkedAttentionConfig:
    heads, kv = _pos(m, "heads", where), _pos(m, "kv_heads", where)
    if heads % kv:
        raise ConfigError(f"config.json: {where}heads {heads} must be a multiple of kv_heads {kv}")
    dim = _pos(m, "dim", where)
    mask = _sub(m, "mask", where, optional=True)
    return ChunkedAttentionConfig(heads=heads, kv_heads=kv, dim=dim, vdim=_pos(m, "vdim", where), scale=_num(m, "scale", where),
                                  chunk=_pos(mask, "size", where + "mask.") if mask is not None else 0,
                                  rot=_rotation(m, where, dim))


def _mlp(raw: Any, where: str) -> Optional[ClampedMlpConfig]:
    if raw is None:
        return None
    if not isinstance(raw, dict):
        raise ConfigError(f"config.json: {where[:-1]} must be an object or null")
    if raw.get("kind") != "dense":
        raise ConfigError(f"config.json: {where}kind must be 'dense', got {raw.get('kind')!r}")
    return ClampedMlpConfig(ff=_pos(raw, "ff", where), limit=_positive(raw, "limit", where))


@dataclass(frozen=True)
class BebovikConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    logit_scale: float
    logit_softcap: float
    layers: Tuple[BebovikLayer, ...]

    architecture = "Bebovik"

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "BebovikConfig":
        layers_raw = take(raw, "layers", list)
        if not layers_raw:
            raise ConfigError("config.json: layers must not be empty")
        layers = []
        for i, lr in enumerate(layers_raw):
            where = f"layers[{i}]."
            if not isinstance(lr, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            if lr.get("type") != "attention":
                raise ConfigError(f"config.json: {where}type must be 'attention', got {lr.get('type')!r}")
            layers.append(BebovikLayer(mixer=_attention(_sub(lr, "mixer", where), where + "mixer."),
                                       mlp=_mlp(lr.get("mlp"), where + "mlp.")))
        return cls(vocab=_pos(raw, "vocab", ""), width=_pos(raw, "width", ""), eps=_num(_sub(raw, "norm", ""), "eps", "norm."),
                   embedding_scale=_num(_sub(raw, "embedding", ""), "scale", "embedding."),
                   logit_scale=_num(raw, "logit_scale", ""), logit_softcap=_positive(raw, "logit_softcap", ""),
                   layers=tuple(layers))
