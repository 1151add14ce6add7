"""Tiny Bebovik configurations, random model folders with weights shaped so that faults show, and the helpers that the
host tests (plain twins of the kernels, CPU) and the gpu tests share to run schedules against the plain implementation
of ``plain_bebovik``.

Random weights of standard deviation 0.02 hide faults: attention is nearly uniform, every tanh is nearly linear, the
feed-forward's clamps and the cap on the logits are never reached and the layer scales are all 1.  ``sharpen`` spreads the
norms' scalars, weights and biases, the layer scales, the head norms' weights, the gates and the feed-forward's inputs.
``beacon`` makes one token's key stand out for every query of its chunk, however far away."""
import copy
import json
import os

import torch

import plain_bebovik as plain
from lalepel_cases import cuts, make_runner, run_steps, schedules, tokens  # noqa: F401  (shared schedule helpers)


def attention(heads, kv_heads, dim, vdim, chunk=None, rot=None, base=10000.0, scaling=None, scale=None):
    """``scaling`` = (factor, low, high, original)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5}
    if chunk:
        m["mask"] = {"size": chunk}
    if rot:
        m["rot"] = {"base": base, "dims": rot}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return m


def layer(mixer, ff=0, limit=1.25):
    """``ff`` 0: no feed-forward."""
    return {"type": "attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff else None}


def model(width, vocab, layers, eps=1e-5, emb=6.0, logit_scale=1.5, cap=9.0):
    return {"architecture": "Bebovik", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": emb},
            "logit_scale": logit_scale, "logit_softcap": cap, "layers": layers}


CONFIGS = {
    # layers that differ in everything: head counts and sizes, values of other sizes than keys, chunks of 20, 33 and 7
    # positions and none, a rotated part with and without scaled frequencies and none, a layer without a feed-forward
    "mix": model(72, 89, [
        layer(attention(4, 2, 24, 24, chunk=20, rot=12, base=3000.0, scaling=(4.0, 1.0, 3.0, 60), scale=0.31), 56, 1.25),
        layer(attention(6, 3, 16, 32, chunk=33, rot=16, base=900.0, scale=0.4), 40, 0.75),
        layer(attention(2, 2, 40, 8, scale=0.27), 0),
        layer(attention(5, 1, 32, 32, chunk=7, rot=8, base=77.0, scaling=(16.0, 0.5, 2.0, 300)), 24, 2.5),
    ], emb=5.0, logit_scale=0.75, cap=6.0),
    # nothing a multiple of 16, 8 or 4; one head; a factor of 1 on embedding and logits; a chunk of one position
    "odd": model(50, 61, [
        layer(attention(3, 3, 10, 6, chunk=13, rot=6), 9, 0.5),
        layer(attention(1, 1, 7, 13, chunk=1), 5, 2.0),
        layer(attention(2, 1, 6, 14, chunk=9, rot=2, base=50.0, scaling=(2.0, 1.0, 4.0, 20), scale=0.6), 0),
        layer(attention(4, 2, 18, 18, chunk=1000, rot=18), 11, 3.0),
    ], eps=1e-6, emb=1.0, logit_scale=1.0, cap=3.5),
    "attention_only": model(48, 50, [layer(attention(4, 2, 16, 16, chunk=16, rot=8), 0)]),
    "mlp_only": model(40, 45, [layer(attention(1, 1, 8, 8, chunk=1), 48, 1.0)]),
    # larger heads: heads of 128 with values of 96 (the kernels' head size above the values'), four query heads to a
    # key/value head, chunks of 48 and 66
    "wide": model(128, 211, [
        layer(attention(4, 1, 128, 96, chunk=48, rot=96, base=5e5, scaling=(6.0, 1.0, 5.0, 200), scale=0.12), 160, 1.5),
        layer(attention(4, 2, 64, 64, chunk=66, rot=24, base=1e4, scale=0.2), 96, 2.0),
    ], emb=9.0, logit_scale=2.5, cap=14.0),
}
SEEDS = {n: 231 + i for i, n in enumerate(CONFIGS)}


def sharpen(name, w, strength=1.0):
    """Weights (name -> float32 tensor) changed in place so that every mechanism matters.  ``strength`` < 1 moves the factors on
    the projections towards 1 (deep bfloat16 models, whose rounding sharp scores amplify)."""
    g = torch.Generator().manual_seed(19)
    f = lambda m: 1.0 + (m - 1.0) * strength
    width = w["embed"].shape[1]
    for n in list(w):
        t = w[n]
        if n.endswith(".alpha"):
            w[n] = 0.4 + 0.9 * torch.rand(t.shape, generator=g)
        elif n.endswith((".norm1", ".norm1b", ".norm2", ".norm2b")) or n in ("embed.norm", "final.norm"):
            w[n] = 0.5 + torch.rand(t.shape, generator=g)
        elif n.endswith(".b"):
            w[n] = (torch.rand(t.shape, generator=g) - 0.5) * 0.6
        elif n.endswith((".ls1", ".ls2")):
            w[n] = 0.3 + 0.9 * torch.rand(t.shape, generator=g)
        elif n.endswith((".q.norm", ".k.norm")):
            w[n] = 0.5 + torch.rand(t.shape, generator=g)
        elif n.endswith((".mix.q", ".mix.k")):
            w[n] = t * 8.0                     # (normed per head: only the ratio to eps matters)
        elif n.endswith((".mix.v", ".mix.o", ".mix.g")):
            w[n] = t * f(9.0)
        elif n.endswith((".gate", ".up")):
            w[n] = t * f(15.0)                 # the clamps are reached
        elif n.endswith(".down"):
            w[n] = t * f(6.0)
        elif n == "head":
            w[n] = t * 50.0 * (48.0 / width) ** 0.5   # the cap is reached
        elif n == "embed":
            w[n] = t * 9.0


BEACON = 7


def beacon(name, w):
    """One token (``BEACON``) whose key stands out for every query of its chunk: every query carries a fixed direction in the
    head's last, unrotated elements (from a constant channel of the normed stream), and the beacon's key has that direction
    (from a channel that only its embedding sets), so its score lies many units above all others wherever it stands."""
    sharpen(name, w)
    w["embed"][:, 1] = 0.0
    w["embed"][BEACON, 1] = 3.0
    w["embed.norm.b"][1] = 0.0
    w["l0.norm1.b"][1] = 0.0
    w["l0.norm1"][0] = 0.0
    w["l0.norm1.b"][0] = 1.0
    d = w["l0.mix.q.norm"].numel()
    for proj, channel in (("l0.mix.q", 0), ("l0.mix.k", 1)):
        heads = w[proj].view(-1, d, w[proj].shape[1])
        heads[:, :, channel] = 0.0
        heads[:, d - 4:, channel] = 6.0


def make_dir(tmp_path, name, store_dtype=torch.bfloat16, raw=None, tweak=sharpen, seed=None):
    """A model folder of configuration ``name`` (or ``raw``): seeded random weights, then ``tweak``, stored in
    ``store_dtype``.  Returns (folder, config dict, weights as stored, float32)."""
    from locus_b200.weights.loader import write_random_model
    from locus_b200.weights.safetensors_io import ModelFiles, write_safetensors
    import locus_b200.models  # noqa: F401

    cfg = copy.deepcopy(raw if raw is not None else CONFIGS[name])
    d = os.path.join(str(tmp_path), f"bebovik_{name}_{str(store_dtype).split('.')[-1]}")
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


class Case:
    def __init__(self, name, tmp_path, store_dtype=torch.bfloat16, raw=None, requests=(), tweak=sharpen, seed=None):
        self.name = name
        self.dir, self.cfg, self.weights = make_dir(tmp_path, name, store_dtype, raw=raw, tweak=tweak, seed=seed)
        self.tokens = {f"r{i}": tokens(n, self.cfg["vocab"], 1000 * (i + 1) + n) for i, n in enumerate(requests)}
        self._ref = {}

    def ref(self, rid):
        """The plain logits [T, vocab] (float64)."""
        if rid not in self._ref:
            self._ref[rid] = plain.forward(self.cfg, self.weights, self.tokens[rid])
        return self._ref[rid]


def errors(out, ref):
    """Per row: the largest difference of the logits (mean taken off) over the largest logit of the request."""
    d = out - ref
    d = d - d.mean(-1, keepdim=True)
    top = float((ref - ref.mean(-1, keepdim=True)).abs().max())
    return d.abs().max(-1).values / top, float(d.abs().mean()) / top


def compare(case, got, tol_max, tol_mean):
    for rid, out in got.items():
        ref = case.ref(rid)
        assert out.shape == ref.shape, rid
        assert bool(torch.isfinite(out).all()), f"{case.name}/{rid}: logits that are not numbers (a page read stale?)"
        err, mean = errors(out, ref)
        worst = int(err.argmax())
        assert float(err.max()) <= tol_max, f"{case.name}/{rid}: position {worst} is off by {float(err.max()):.2e} of the largest logit"
        assert mean <= tol_mean, f"{case.name}/{rid}: mean error {mean:.2e}"


def random_config(seed):
    """A configuration drawn from the ranges a small model of this design may have: widths, head counts and sizes, chunks,
    rotated parts, scaled frequencies, feed-forwards and constants all vary, layer by layer."""
    import random

    r = random.Random(seed)
    layers = []
    for _ in range(r.randint(2, 6)):
        heads = r.choice([1, 2, 4, 6, 8])
        kv = r.choice([k for k in (1, 2, 3, 4, 8) if heads % k == 0])
        dim = r.choice([16, 32, 48, 64, 80, 128])
        rot = r.choice([0, dim // 4 * 2, dim])
        scaling = r.choice([None, (r.choice([2.0, 4.0, 32.0]), 1.0, r.choice([2.0, 4.0]), r.choice([64, 256, 8192]))])
        mixer = attention(heads, kv, dim, r.choice([dim, 32, 64, 80]), chunk=r.choice([None, 5, 16, 50, 64, 100, 128, 200]), rot=rot,
                          base=r.choice([1e4, 5e5]), scaling=scaling if rot else None, scale=round(r.uniform(0.05, 0.25), 3))
        layers.append(layer(mixer, r.choice([0, 64, 160, 320]), r.choice([0.75, 1.5, 4.0])))
    return model(r.choice([64, 96, 128, 192]), r.randint(100, 700), layers, eps=r.choice([1e-5, 1e-6]), emb=r.choice([1.0, 4.0, 10.0]),
                 logit_scale=r.choice([1.0, 0.5, 3.0]), cap=r.choice([8.0, 20.0, 50.0]))
