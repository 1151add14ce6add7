"""The Megovik design as a plan of parts.

A decoder of parallel blocks: one RMS norm, whose output both sublayers read, x <- x + (mixer(h) + ff(h)).  The residual
stream starts from the scaled embedding plus a learned vector per position; a stretch of layers may run several times in a
row with the same weights (a cache for every pass), and what the embedding gave is added once more in front of every pass
but the first.  Mixers: ``attention``, grouped queries with weighted head norms, a factor on q by position, a linear
distance bias per head and values that are the keys as projected; ``latent_attention`` and ``latent_attention_2``, keys and
values of all heads from one cached latent without positions, the queries projected directly or through a latent of their
own.  Feed-forwards: a rectified gate with biases, or routed SwiGLU experts with sigmoid scores chosen within the best
groups.  Tensor names: ``embed``, ``pos``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.gate|up|down`` (+ ``.b``),
``l<i>.mlp.router|e<j>.gate|up|down``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from typing import List

from ..config.base import ArchEntry, register_arch
from ..config.lalepel import DenseFfConfig
from ..config.megovik import BiasedAttentionConfig, MegovikConfig, PlainLatentConfig, SigmoidMoeConfig
from ..parts.base import LayerCall, LayerSpec, ModelPlan, PartSpec

_ATTN_NAMES = {"q": "q", "k": "k", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm"}
_DENSE_NAMES = {"gate": "gate", "up": "up", "down": "down", "gate_bias": "gate.b", "up_bias": "up.b", "down_bias": "down.b"}
_MOE_NAMES = {"router": "router", "expert_gate": "e{e}.gate", "expert_up": "e{e}.up", "expert_down": "e{e}.down"}


def head_slopes(heads: int) -> tuple:
    """The distance bias's slope of every head, 2^(-8 (h + 1) / heads)."""
    return tuple(2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads))


def _mixer(cfg: MegovikConfig, m) -> PartSpec:
    if isinstance(m, BiasedAttentionConfig):
        return PartSpec("attention", {
            "hidden": cfg.width, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim, "qkv_bias": False,
            "qk_norm": "head", "qk_norm_eps": cfg.eps, "softmax_scale": m.scale, "position": PartSpec("none"), "values": "keys",
            "q_temp": (m.q_temp.coef, m.q_temp.every) if m.q_temp is not None else None, "slopes": head_slopes(m.heads),
            "names": _ATTN_NAMES})
    if isinstance(m, PlainLatentConfig):
        return PartSpec("latent_attention", {
            "hidden": cfg.width, "n_heads": m.heads, "nope_dim": m.dim, "rot_dim": 0, "v_dim": m.vdim, "q_rank": m.q_rank,
            "kv_rank": m.kv_rank, "scale": m.scale, "eps": cfg.eps})
    raise TypeError(m)


def _feed_forward(cfg: MegovikConfig, f) -> PartSpec:
    if f is None:
        return PartSpec("none")
    if isinstance(f, DenseFfConfig):
        return PartSpec("dense_mlp", {"hidden": cfg.width, "intermediate": f.ff, "activation": "reglu", "bias": True,
                                      "names": _DENSE_NAMES})
    if isinstance(f, SigmoidMoeConfig):
        return PartSpec("sparse_moe", {
            "hidden": cfg.width, "n_experts": f.experts, "top_k": f.top, "norm_topk": True, "expert_intermediate": f.expert_ff,
            "shared_gate": False, "score_fn": "sigmoid", "weight_scale": f.scale, "n_group": f.group_count,
            "n_group_used": f.group_keep, "names": _MOE_NAMES})
    raise TypeError(f)


def run_order(cfg: MegovikConfig) -> List[LayerCall]:
    n = len(cfg.layers)
    if cfg.loop is None:
        return [LayerCall(i) for i in range(n)]
    a, b, times = cfg.loop
    order = [LayerCall(i) for i in range(a)]
    for k in range(times):
        order += [LayerCall(i, add_embedding=k > 0 and i == a) for i in range(a, b)]
    return order + [LayerCall(i) for i in range(b, n)]


def build_plan(cfg: MegovikConfig) -> ModelPlan:
    norm = PartSpec("rmsnorm", {"width": cfg.width, "eps": cfg.eps})
    layers = [LayerSpec(prefix=f"l{i}", arrangement=PartSpec("parallel_pre_norm", {"hidden": cfg.width}), norm=norm,
                        mixer=_mixer(cfg, layer.mixer), feed_forward=_feed_forward(cfg, layer.mlp))
              for i, layer in enumerate(cfg.layers)]
    return ModelPlan(
        architecture=cfg.architecture, hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=cfg.max_positions,
        eos_token_id=-1,
        embedding=PartSpec("embedding", {"vocab": cfg.vocab, "hidden": cfg.width, "prefix": "embed", "tensor": "embed",
                                         "scale": cfg.embedding_scale,
                                         "positions": {"tensor": "pos", "count": cfg.max_positions}}),
        layers=layers, order=run_order(cfg),
        final_norm=PartSpec("rmsnorm", {"width": cfg.width, "eps": cfg.eps, "prefix": "final.norm", "tensor": "final.norm"}),
        head=PartSpec("linear", {"vocab": cfg.vocab, "hidden": cfg.width, "prefix": "head", "tensor": "head",
                                 "scale": cfg.logit_scale}),
        config=cfg,
    )


register_arch(ArchEntry(
    name="Megovik",
    description="Megovik: parallel blocks on one RMS norm, learned position vectors, looped layers that the embedding enters "
                "again; grouped-query attention with values that are the keys, q/k head norms, a factor on q by position and a "
                "distance bias; latent attention without positions, queries direct or through a latent; dense rectified gates "
                "with biases or routed SwiGLU experts with grouped sigmoid scores",
    parse_config=MegovikConfig.from_dict,
    build_plan=build_plan,
))
