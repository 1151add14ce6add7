"""Typed configuration of the Megovik design.

config.json of this design is nested: the model's ``width``, ``vocab``, ``max_positions`` (rows of the table of learned
position vectors: the longest context), ``norm.eps``, ``embedding.scale`` (a factor on the token's row), ``logit_scale``,
``loop`` = {``start``, ``stop``, ``times``} (layers start .. stop - 1 run ``times`` times in a row; absent: every layer
once) and a list ``layers`` whose entries each give the ``type`` of their mixer, the mixer's sizes and constants (``mixer``)
and their feed-forward (``mlp``, or null for none).  Layers may differ from each other in everything.  Every size and
constant is read here; nothing about a particular model is fixed in code.

Mixer ``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim`` (the values are the keys: equal to ``dim``), ``scale``,
``q_temp`` = {``coef``, ``every``} (a factor on q by position; absent: none).
Mixer ``latent_attention``: ``heads``, ``dim``, ``vdim``, ``kv_rank``, ``scale``.  Mixer ``latent_attention_2``: also
``q_rank``, the size of the queries' own latent.
Feed-forward ``dense``: ``ff``.  ``moe``: ``router`` = {``experts``, ``top``, ``scale`` (absent: 1), ``groups`` =
{``count``, ``keep``} (absent: one group)}, ``expert.ff``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError, take
from .lalepel import DenseFfConfig, _num, _pos, _sub
from .pozozen import _groups, _loop


@dataclass(frozen=True)
class QueryTemperature:
    coef: float
    every: float


@dataclass(frozen=True)
class BiasedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    q_temp: Optional[QueryTemperature]

    kind = "attention"


@dataclass(frozen=True)
class PlainLatentConfig:
    heads: int
    dim: int
    vdim: int
    q_rank: int                      # 0: the queries have no latent
    kv_rank: int
    scale: float

    kind = "latent_attention"


@dataclass(frozen=True)
class SigmoidMoeConfig:
    experts: int
    top: int
    group_count: int
    group_keep: int
    scale: float
    expert_ff: int

    kind = "moe"


@dataclass(frozen=True)
class MegovikLayer:
    mixer: Any                       # BiasedAttentionConfig | PlainLatentConfig
    mlp: Any                         # DenseFfConfig | SigmoidMoeConfig | None


def _attention(m: Dict[str, Any], where: str) -> BiasedAttentionConfig:
    heads, kv = _pos(m, "heads", where), _pos(m, "kv_heads", where)
    if heads % kv:
        raise ConfigError(f"config.json: {where}heads {heads} must be a multiple of kv_heads {kv}")
    dim = _pos(m, "dim", where)
    vdim = take(m, "vdim", int, dim)
    if vdim != dim:
        raise ConfigError(f"config.json: {where}vdim {vdim} must equal dim {dim} (the values are the keys)")
    temp = _sub(m, "q_temp", where, optional=True)
    q_temp = None
    if temp is not None:
        w = where + "q_temp."
        q_temp = QueryTemperature(coef=_num(temp, "coef", w), every=_num(temp, "every", w))
        if not q_temp.every > 0:
            raise ConfigError(f"config.json: {w}every must be positive, got {q_temp.every}")
    return BiasedAttentionConfig(heads=heads, kv_heads=kv, dim=dim, scale=_num(m, "scale", where), q_temp=q_temp)


def _latent(m: Dict[str, Any], where: str, q_latent: bool) -> PlainLatentConfig:
    return PlainLatentConfig(heads=_pos(m, "heads", where), dim=_pos(m, "dim", where), vdim=_pos(m, "vdim", where),
                             q_rank=_pos(m, "q_rank", where) if q_latent else 0, kv_rank=_pos(m, "kv_rank", where),
                             scale=_num(m, "scale", where))


def _mlp(raw: Any, where: str):
    if raw is None:
        return None
    if not isinstance(raw, dict):
        raise ConfigError(f"config.json: {where[:-1]} must be an object or null")
    kind = raw.get("kind")
    if kind == "dense":
        return DenseFfConfig(ff=_pos(raw, "ff", where))
    if kind != "moe":
        raise ConfigError(f"config.json: {where}kind must be 'dense' or 'moe', got {kind!r}")
    router, rw = _sub(raw, "router", where), where + "router."
    experts, top = _pos(router, "experts", rw), _pos(router, "top", rw)
    if top > experts:
        raise ConfigError(f"config.json: {rw}top {top} exceeds {rw}experts {experts}")
    count, keep = _groups(router, rw, experts, top)
    return SigmoidMoeConfig(experts=experts, top=top, group_count=count, group_keep=keep, scale=take(router, "scale", float, 1.0),
                            expert_ff=_pos(_sub(raw, "expert", where), "ff", where + "expert."))


@dataclass(frozen=True)
class MegovikConfig:
    vocab: int
    width: int
    max_positions: int
    eps: float
    embedding_scale: float
    logit_scale: float
    loop: Optional[Tuple[int, int, int]]   # (start, stop, times)
    layers: Tuple[MegovikLayer, ...]

    architecture = "Megovik"

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "MegovikConfig":
        layers_raw = take(raw, "layers", list)
        if not layers_raw:
            raise ConfigError("config.json: layers must not be empty")
        layers = []
        for i, lr in enumerate(layers_raw):
            where = f"layers[{i}]."
            if not isinstance(lr, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            kind, m, w = lr.get("type"), _sub(lr, "mixer", where), where + "mixer."
            if kind == "attention":
                mixer = _attention(m, w)
            elif kind in ("latent_attention", "latent_attention_2"):
                mixer = _latent(m, w, kind == "latent_attention_2")
            else:
                raise ConfigError(f"config.json: {where}type must be 'attention', 'latent_attention' or 'latent_attention_2', "
                                  f"got {kind!r}")
            layers.append(MegovikLayer(mixer=mixer, mlp=_mlp(lr.get("mlp"), where + "mlp.")))
        return cls(vocab=_pos(raw, "vocab", ""), width=_pos(raw, "width", ""), max_positions=_pos(raw, "max_positions", ""),
                   eps=_num(_sub(raw, "norm", ""), "eps", "norm."),
                   embedding_scale=_num(_sub(raw, "embedding", ""), "scale", "embedding."),
                   logit_scale=_num(raw, "logit_scale", ""), loop=_loop(raw, len(layers)), layers=tuple(layers))
