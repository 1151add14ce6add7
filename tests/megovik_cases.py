"""Tiny Megovik configurations, random model folders with weights shaped so that faults show, and the helpers that the
host tests (plain twins of the kernels, CPU) and the gpu tests share to run schedules against the plain implementation of
``plain_megovik``.

Random weights of standard deviation 0.02 hide faults: attention is nearly uniform, the position vectors and biases are
lost beside the embedding, every router is near 1/2 and the experts give nothing.  ``sharpen`` spreads all of them.
``beacon`` makes one token's key stand out for every later query, however far away."""
import copy
import json
import os

import torch

import plain_megovik as plain
import pozozen_cases
from lalepel_cases import cuts, make_runner, schedules, tokens  # noqa: F401  (shared schedule helpers)
from pozozen_cases import compare, compare_together, run_steps  # noqa: F401


def attention(heads, kv_heads, dim, scale=None, temp=None):
    """``temp`` = (coef, every)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale if scale is not None else dim ** -0.5}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": m}


def latent(heads, dim, vdim, kv_rank, q_rank=0, scale=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale if scale is not None else dim ** -0.5}
    if q_rank:
        m["q_rank"] = q_rank
    return {"type": "latent_attention_2" if q_rank else "latent_attention", "mixer": m}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, groups=None, scale=1.5):
    router = {"experts": experts, "top": top, "scale": scale}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "router": router, "expert": {"ff": ff}}


def with_mlp(layer, mlp):
    return {**layer, "mlp": mlp}


def model(width, vocab, layers, loop=None, eps=1e-5, emb=4.0, logit_scale=0.8, positions=1024):
    cfg = {"architecture": "Megovik", "width": width, "vocab": vocab, "max_positions": positions, "norm": {"eps": eps},
           "embedding": {"scale": emb}, "logit_scale": logit_scale, "layers": layers}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


CONFIGS = {
    # layers that differ in everything, the middle of them run three times
    "mix": model(72, 89, [
        with_mlp(latent(3, 24, 16, 40, scale=0.21), moe(8, 3, 24, groups=(4, 2), scale=2.5)),
        with_mlp(attention(6, 2, 24, scale=0.3, temp=(0.4, 9)), dense(56)),
        with_mlp(latent(2, 16, 40, 24, q_rank=32), dense(40)),
        with_mlp(attention(4, 4, 16, temp=(0.15, 50)), None),
        with_mlp(attention(5, 1, 32, scale=0.12), moe(6, 2, 16, groups=(2, 1), scale=0.7)),
    ], loop=(1, 4, 3), emb=3.0),
    # nothing a multiple of 8 or 4; one head; groups of one expert, no groups, every expert picked; a factor of 1
    "odd": model(50, 61, [
        with_mlp(attention(3, 3, 10, temp=(1.0, 1)), moe(3, 2, 7, groups=(3, 2), scale=1.0)),
        with_mlp(latent(1, 7, 13, 9), dense(9)),
        with_mlp(latent(5, 6, 5, 10, q_rank=11, scale=0.5), moe(5, 5, 6)),
        with_mlp(attention(1, 1, 18, scale=0.4, temp=(0.25, 7)), moe(4, 1, 12, scale=3.0)),
    ], loop=(0, 4, 2), eps=1e-6, emb=1.0, logit_scale=1.0),
    "attention_only": model(48, 50, [with_mlp(attention(4, 2, 16, scale=0.4, temp=(0.3, 20)), None)]),
    "latents_only": model(48, 50, [with_mlp(latent(4, 16, 16, 32), None), with_mlp(latent(2, 24, 8, 24, q_rank=16), None)]),
    "dense_only": model(40, 45, [with_mlp(attention(1, 1, 8), dense(48))], loop=(0, 1, 2)),
    "moe_only": model(40, 45, [with_mlp(latent(1, 8, 8, 8), moe(12, 4, 16, groups=(3, 2)))], loop=(0, 1, 1)),
    # larger heads and latents: four query heads to a key/value head of 128, rows of 256 and 96
    "wide": model(128, 211, [
        with_mlp(attention(8, 2, 128, scale=0.07, temp=(0.5, 30)), dense(160)),
        with_mlp(latent(4, 64, 32, 256, scale=0.11), moe(8, 2, 64, groups=(4, 3), scale=2.0)),
        with_mlp(latent(6, 32, 64, 96, q_rank=64), dense(96)),
        with_mlp(attention(8, 4, 64, scale=0.1), None),
    ], loop=(1, 3, 2), emb=2.0, logit_scale=0.5),
}
SEEDS = {n: 331 + i for i, n in enumerate(CONFIGS)}


def sharpen(name, w, strength=1.0):
    """Weights (name -> float32 tensor) changed in place so that every mechanism matters.  ``strength`` < 1 moves the factors
    on the projections towards 1 (deep bfloat16 models, whose rounding sharp scores amplify)."""
    g = torch.Generator().manual_seed(23)
    f = lambda m: 1.0 + (m - 1.0) * strength
    width = w["embed"].shape[1]
    for n in list(w):
        t = w[n]
        if n.endswith((".norm1", ".norm")):
            w[n] = 0.5 + torch.rand(t.shape, generator=g)
        elif n.endswith(".b"):
            w[n] = (torch.rand(t.shape, generator=g) - 0.5) * 0.8
        elif n == "embed":
            w[n] = t * 15.0
        elif n == "pos":
            w[n] = t * 40.0
        elif n.endswith((".mix.q", ".mix.uq", ".mix.uk")):
            w[n] = t * f(8.0)
        elif n.endswith((".mix.k", ".mix.uv", ".mix.o")):
            w[n] = t * f(7.0)
        elif n.endswith(".router"):
            w[n] = t * 8.0
        elif n.endswith((".gate", ".up", ".down")):
            w[n] = t * f(9.0)
        elif n == "head":
            w[n] = t * 40.0 * (48.0 / width) ** 0.5


BEACON = 7


def beacon(name, w):
    """One token (``BEACON``) whose key stands out for every later query of the model's one attention layer: every query
    carries a fixed direction (from a channel of the residual stream that every embedding sets alike), and the beacon's key
    has that direction (from a channel that only its embedding sets), so its score lies many units above all others'
    wherever it stands."""
    sharpen(name, w)
    w["pos"] *= 0.1
    w["pos"][:, :2] = 0.0
    w["embed"][:, 0] = 1.0
    w["embed"][:, 1] = 0.0
    w["embed"][BEACON, 1] = 3.0
    w["l0.norm1"][:2] = 1.0
    into = (("l0.mix.q", 0), ("l0.mix.k", 1)) if "l0.mix.k" in w else (("l0.mix.q" if "l0.mix.q" in w else "l0.mix.dq", 0), ("l0.mix.dkv", 1))
    for n, channel in into:
        w[n] *= 0.2 if n == "l0.mix.k" else 1.0
        w[n][:, channel] = 0.0
    if "l0.mix.k" in w:
        d = w["l0.mix.q.norm"].numel()
        w["l0.mix.q.norm"][:] = 1.0
        w["l0.mix.k.norm"][:] = 1.0
        for n, channel in into:
            heads = w[n].view(-1, d, w[n].shape[1])
            heads[:, d - 2:, channel] = 6.0
        return
    # the latents: one dimension of each carries the direction, and every head's first query and key dimension reads it
    w["l0.mix.dkv"][0, 1] = 8.0
    w["l0.mix.dkv.norm"][0] = 1.0
    q = "l0.mix.q"
    if "l0.mix.dq" in w:
        w["l0.mix.dq"][0, 0] = 6.0
        w["l0.mix.dq.norm"][0] = 1.0
        q = "l0.mix.uq"
        w[q][:, 0] = 0.0
    w["l0.mix.uk"][:, 0] = 0.0
    d = w["l0.mix.uk"].shape[0] // BEACON_HEADS
    for h in range(BEACON_HEADS):
        w[q][h * d] = 0.0
        w[q][h * d, 0] = 4.0
        w["l0.mix.uk"][h * d] = 0.0
        w["l0.mix.uk"][h * d, 0] = 4.0


BEACON_HEADS = 4


def make_dir(tmp_path, name, store_dtype=torch.bfloat16, raw=None, tweak=sharpen, seed=None):
    """A model folder of configuration ``name`` (or ``raw``): seeded random weights, then ``tweak``, stored in
    ``store_dtype``.  Returns (folder, config dict, weights as stored, float32)."""
    from locus_b200.weights.loader import write_random_model
    from locus_b200.weights.safetensors_io import ModelFiles, write_safetensors
    import locus_b200.models  # noqa: F401

    cfg = copy.deepcopy(raw if raw is not None else CONFIGS[name])
    d = os.path.join(str(tmp_path), f"megovik_{name}_{str(store_dtype).split('.')[-1]}")
    write_random_model(cfg, SEEDS.get(name, 5) if seed is None else seed, d, torch.float32)
    mf = ModelFiles(d)
    w = {n: mf.tensor(n).clone().float() for n in mf.names()}
    mf.close()
    if tweak is not None:
        tweak(name, w)
    w = {n: t.to(store_dtype) for n, t in w.items()}
    write_safetensors(os.path.join(d, "model.safetensors"), [(n, tuple(t.shape), store_dtype) for n, t in w.items()],
                      lambda n: w[n], metadata={"format": "pt"})
    with open(os.path.join(d, "config.json"), "w", encoding="utf-8") as f:
        json.dump(cfg, f)
    return d, cfg, {n: t.float() for n, t in w.items()}


class Case(pozozen_cases.Case):
    """With ``ref`` and ``ref_following`` (the plain logits, with the engine's picks at a router's near-ties)."""

    def __init__(self, name, tmp_path, store_dtype=torch.bfloat16, raw=None, requests=(), tweak=sharpen, seed=None):
        self.name = name
        self.dir, self.cfg, self.weights = make_dir(tmp_path, name, store_dtype, raw=raw, tweak=tweak, seed=seed)
        self.tokens = {f"r{i}": tokens(n, self.cfg["vocab"], 1000 * (i + 1) + n) for i, n in enumerate(requests)}
        self.order = [i for i, _ in plain.run_order(self.cfg)]
        self._ref = {}

    def ref(self, rid, picks=None):
        if picks is None and rid in self._ref:
            return self._ref[rid]
        aux = {}
        lg = plain.forward(self.cfg, self.weights, self.tokens[rid], picks=picks, aux=aux)
        if picks is None:
            self._ref[rid] = (lg, aux)
        return lg, aux


def errors(out, ref):
    """Per row: the largest difference of the logits (mean taken off) over the largest logit of the request."""
    d = out - ref
    d = d - d.mean(-1, keepdim=True)
    top = float((ref - ref.mean(-1, keepdim=True)).abs().max())
    return d.abs().max(-1).values / top, float(d.abs().mean()) / top


def random_config(seed):
    """A configuration drawn from the ranges a small model of this design may have: widths, head counts and sizes, latents,
    temperatures, feed-forwards, routers, groups, the loop and constants all vary, layer by layer."""
    import random

    r = random.Random(seed)

    def ff():
        kind = r.random()
        if kind < 0.15:
            return None
        if kind < 0.5:
            return dense(r.choice([64, 96, 160, 320]))
        experts = r.choice([4, 6, 8, 12, 16])
        count = r.choice([c for c in (1, 2, 3, 4, 8) if experts % c == 0])
        keep = r.randint(1, count)
        top = r.randint(1, min(5, keep * (experts // count)))
        return moe(experts, top, r.choice([32, 64, 96]), groups=(count, keep) if count > 1 or r.random() < 0.5 else None,
                   scale=r.choice([1.0, 0.5, 2.5]))

    def mixer():
        heads = r.choice([1, 2, 3, 4, 6, 8, 12])
        kind = r.random()
        if kind < 0.4:
            dim = r.choice([16, 32, 48, 64, 80, 128])
            return attention(heads, r.choice([k for k in (1, 2, 3, 4, 6, 8) if heads % k == 0]), dim, round(r.uniform(0.03, 0.2), 3),
                             r.choice([None, (0.1, 64), (0.5, 100), (0.3, 31)]))
        return latent(heads, r.choice([16, 24, 32, 64]), r.choice([16, 32, 48, 64]), r.choice([32, 48, 64, 96, 128, 160, 192]),
                      q_rank=r.choice([48, 64, 96]) if kind > 0.7 else 0)

    n = r.randint(2, 5)
    layers = [with_mlp(mixer(), ff()) for _ in range(n)]
    loop = None
    if r.random() < 0.75:
        a = r.randint(0, n - 1)
        loop = (a, r.randint(a + 1, n), r.randint(1, 3))
    return model(r.choice([64, 96, 128, 192]), r.randint(100, 700), layers, loop=loop, eps=r.choice([1e-5, 1e-6]), emb=r.choice([1.0, 4.0, 8.0]),
                 logit_scale=r.choice([1.0, 0.25, 2.0]))
