"""The Bebovik design as a plan of parts.

A decoder whose norm is Dynamic Tanh (elementwise, no statistics) in front of and behind every sublayer, with a layer
scale on what a sublayer adds: x <- x + ls1 * D1b(mixer(D1(x))); x <- x + ls2 * D2b(ff(D2(x))).  The scaled embedding passes
such a norm too.  The mixer is grouped-query attention within chunks of positions: an RMS norm with a shared weight on every
query and key head, a rotation of adjacent pairs of part of each head with frequencies scaled by wavelength, a sigmoid gate
on the heads' outputs.  The feed-forward is a clamped gated unit.  The logits are scaled and softly capped.  Tensor names:
``embed``, ``embed.norm``, ``l<i>.norm1|norm1b|norm2|norm2b``, ``l<i>.ls1|ls2``, ``l<i>.mix.*``, ``l<i>.mlp.gate|up|down``,
``final.norm``, ``head``; a norm's bias and scalar stand beside its weight as ``.b`` and ``.alpha``.
"""
from __future__ import annotations

from ..config.base import ArchEntry, register_arch
from ..config.bebovik import BebovikConfig, ChunkedAttentionConfig
from ..parts.base import LayerCall, LayerSpec, ModelPlan, PartSpec

# positions enter the rotation's angle as float32: exact up to 2^24
MAX_POSITIONS = 1 << 24

_ATTN_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm", "gate": "g"}
_MLP_NAMES = {"gate": "gate", "up": "up", "down": "down"}
_NORM_SUFFIXES = {"tensor": "", "bias_tensor": ".b", "alpha_tensor": ".alpha"}


def _named_norm(width: int, name: str) -> dict:
    return {"width": width, **{arg: name + suffix for arg, suffix in _NORM_SUFFIXES.items()}}


def _position(rot) -> dict:
    args = {"theta": rot.base, "rot_dim": rot.dims, "interleaved": True}
    if rot.scaling is not None:
        s = rot.scaling
        args["scaling"] = {"factor": s.factor, "original": s.original, "high": s.high, "low": s.low}
    return args


def _mixer(cfg: BebovikConfig, m: ChunkedAttentionConfig) -> PartSpec:
    position = PartSpec("none") if m.rot is None else PartSpec("rotary", {"head_dim": m.dim, **_position(m.rot)})
    return PartSpec("attention", {
        "hidden": cfg.width, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim, "v_dim": m.vdim,
        "qkv_bias": False, "qk_norm": "head", "qk_norm_eps": cfg.eps, "softmax_scale": m.scale, "position": position,
        "chunk": m.chunk, "out_gate": True, "names": _ATTN_NAMES})


def _feed_forward(cfg: BebovikConfig, f) -> PartSpec:
    if f is None:
        return PartSpec("none")
    return PartSpec("dense_mlp", {"hidden": cfg.width, "intermediate": f.ff, "activation": "glu_clamp", "limit": f.limit,
                                  "names": _MLP_NAMES})


def build_plan(cfg: BebovikConfig) -> ModelPlan:
    arrangement = PartSpec("sandwich_norm", {"hidden": cfg.width, "scale_names": ("ls1", "ls2"),
                                             "tensor_suffixes": _NORM_SUFFIXES})
    layers = [LayerSpec(prefix=f"l{i}", arrangement=arrangement, norm=PartSpec("dynamic_tanh", {"width": cfg.width}),
                        mixer=_mixer(cfg, layer.mixer), feed_forward=_feed_forward(cfg, layer.mlp))
              for i, layer in enumerate(cfg.layers)]
    return ModelPlan(
        architecture=cfg.architecture, hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS,
        eos_token_id=-1,
        embedding=PartSpec("embedding", {"vocab": cfg.vocab, "hidden": cfg.width, "prefix": "embed", "tensor": "embed",
                                         "scale": cfg.embedding_scale,
                                         "norm": PartSpec("dynamic_tanh", _named_norm(cfg.width, "embed.norm"))}),
        layers=layers, order=[LayerCall(i) for i in range(len(layers))],
        final_norm=PartSpec("dynamic_tanh", {"prefix": "final.norm", **_named_norm(cfg.width, "final.norm")}),
        head=PartSpec("linear", {"vocab": cfg.vocab, "hidden": cfg.width, "prefix": "head", "tensor": "head",
                                 "scale": cfg.logit_scale, "softcap": cfg.logit_softcap}),
        config=cfg,
    )


register_arch(ArchEntry(
    name="Bebovik",
    description="Bebovik: Dynamic Tanh norms around every sublayer and behind the scaled embedding, layer scales; grouped-query "
                "attention within chunks of positions with q/k head norms, an interleaved rotation scaled by wavelength and an "
                "output gate; clamped gated feed-forward; scaled, softly capped logits",
    parse_config=BebovikConfig.from_dict,
    build_plan=build_plan,
))
