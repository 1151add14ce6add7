"""The Megovik design, plainly: float64, whole sequences, one function per mechanism, written from the equations.

Nothing here is shared with ``locus_b200``: the configuration is the raw nested dictionary of config.json and the weights
a dictionary of tensors by their stored names.  ``forward`` runs one sequence from its first token.

Notation: x [T, width] the residual stream, p a position counted from 0, rms(z; w) = z / sqrt(mean(z^2) + eps) * w.

* embedding: e_p = embed[token] * scale + pos[p]; x starts as e;
* order: the layers in turn; the stretch start .. stop - 1 runs ``times`` times in a row with the same weights, and in
  front of every pass but the first e is added to x once;
* layer: one norm for both sublayers, h = rms(x; norm1), x <- x + (mixer(h) + ff(h));
* mixer ``attention``: grouped queries; the values are the keys as projected; q and k take an rms norm per head with a
  shared weight, q then a factor that grows with the logarithm of its position; a head-wise slope times the distance is
  taken off every score;
* mixers ``latent_attention`` and ``latent_attention_2``: c = rms(W_dkv h; dkv.norm), keys W_uk c and values W_uv c head by
  head; the queries are W_q h, or W_uq rms(W_dq h; dq.norm);
* feed-forward ``dense``: W_down (relu(W_gate h + b) * (W_up h + b)) + b; ``moe``: sigmoid scores, the groups with the
  largest sums of two scores stay eligible, the largest scores among them are picked and their sum is brought to ``scale``;
* output: logits = logit_scale * head rms(x; final.norm).
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def _w(weights, name):
    return weights[name].to(F64)


def rms(z, w, eps):
    return z / torch.sqrt((z * z).mean(-1, keepdim=True) + eps) * w


def embedding(cfg, weights, tokens):
    return _w(weights, "embed")[torch.tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"] + _w(weights, "pos")[: len(tokens)]


def slopes(heads):
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def temperature(p, t):
    """The factor on a query at position p."""
    return 1.0 + t["coef"] * math.log(math.floor((p + 1) / t["every"]) + 1) if t else 1.0


def causal_softmax(q, k, v, scale, slope=0.0):
    """One head: q, k [T, d], v [T, dv]."""
    T = q.shape[0]
    at = torch.arange(T, dtype=F64)
    s = (q @ k.T) * scale - slope * (at[:, None] - at[None, :])
    s = s.masked_fill(at[None, :] > at[:, None], -math.inf)
    return torch.softmax(s, -1) @ v


def attention(m, weights, pre, h, eps):
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    k_raw = (h @ _w(weights, pre + "k").T).view(T, G, d)
    q = rms((h @ _w(weights, pre + "q").T).view(T, H, d), _w(weights, pre + "q.norm"), eps)
    q = q * torch.tensor([temperature(p, m.get("q_temp")) for p in range(T)], dtype=F64)[:, None, None]
    k = rms(k_raw, _w(weights, pre + "k.norm"), eps)
    out = [causal_softmax(q[:, i], k[:, i // (H // G)], k_raw[:, i // (H // G)], m["scale"], s) for i, s in enumerate(slopes(H))]
    return torch.cat(out, -1) @ _w(weights, pre + "o").T


def latent_attention(m, weights, pre, h, eps):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    if "q_rank" in m:
        q = rms(h @ _w(weights, pre + "dq").T, _w(weights, pre + "dq.norm"), eps) @ _w(weights, pre + "uq").T
    else:
        q = h @ _w(weights, pre + "q").T
    c = rms(h @ _w(weights, pre + "dkv").T, _w(weights, pre + "dkv.norm"), eps)
    q, k, v = q.view(T, H, d), (c @ _w(weights, pre + "uk").T).view(T, H, d), (c @ _w(weights, pre + "uv").T).view(T, H, dv)
    return torch.cat([causal_softmax(q[:, i], k[:, i], v[:, i], m["scale"]) for i in range(H)], -1) @ _w(weights, pre + "o").T


def dense_ff(weights, pre, h):
    part = lambda n, z: z @ _w(weights, pre + n).T + _w(weights, pre + n + ".b")
    return part("down", torch.relu(part("gate", h)) * part("up", h))


def choose(r, scores):
    """(picked experts, groups' scores, scores with the closed groups' experts at -inf) of one token's scores [experts]
    (python floats)."""
    n, groups = len(scores), r.get("groups") or {"count": 1, "keep": 1}
    per = n // groups["count"]
    of_group = [sum(sorted(scores[g * per:(g + 1) * per])[-2:]) for g in range(groups["count"])]
    kept = sorted(range(groups["count"]), key=lambda g: -of_group[g])[: groups["keep"]]
    masked = [s if e // per in kept else -math.inf for e, s in enumerate(scores)]
    return sorted(range(n), key=lambda e: -masked[e])[: r["top"]], of_group, masked


def shares(r, scores, picked):
    """The picked experts' weights."""
    total = sum(scores[e] for e in picked) + 1e-20
    return [scores[e] / total * r.get("scale", 1.0) for e in picked]


def moe_ff(f, weights, pre, h, picks=None, aux=None):
    s = torch.sigmoid(h @ _w(weights, pre + "router").T)
    out = torch.zeros_like(h)
    seen = [choose(f["router"], row) for row in s.tolist()]
    if aux is not None:
        aux.update(own=torch.tensor([c[0] for c in seen]), groups=torch.tensor([c[1] for c in seen]),
                   masked=torch.tensor([c[2] for c in seen]), choice=s)
    for t in range(h.shape[0]):
        picked = seen[t][0] if picks is None else picks[t]
        for e, w in zip(picked, shares(f["router"], s[t].tolist(), picked)):
            g, u = (_w(weights, f"{pre}e{e}.{n}") @ h[t] for n in ("gate", "up"))
            out[t] += w * (_w(weights, f"{pre}e{e}.down") @ (g * torch.sigmoid(g) * u))
    return out


def run_order(cfg):
    """(layer, whether the embedding is added in front of it) in the order of the run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    body = range(loop["start"], loop["stop"])
    order = [(i, False) for i in range(loop["start"])]
    for k in range(loop["times"]):
        order += [(i, k > 0 and i == loop["start"]) for i in body]
    return order + [(i, False) for i in range(loop["stop"], n)]


MIXERS = {"attention": attention, "latent_attention": latent_attention, "latent_attention_2": latent_attention}


def forward(cfg, weights, tokens, layers_out=None, picks=None, aux=None):
    """Logits [T, vocab] of one sequence; ``layers_out``: a list that receives the residual stream after every layer run.
    ``picks`` {index in the run order: experts of every token}: taken in the place of the router's own choice; ``aux``
    receives {index in the run order: what the router saw}."""
    eps = cfg["norm"]["eps"]
    e = embedding(cfg, weights, tokens)
    x = e
    for call, (i, add) in enumerate(run_order(cfg)):
        layer = cfg["layers"][i]
        if add:
            x = x + e
        h = rms(x, _w(weights, f"l{i}.norm1"), eps)
        y = MIXERS[layer["type"]](layer["mixer"], weights, f"l{i}.mix.", h, eps)
        f = layer.get("mlp")
        if f is not None and f["kind"] == "dense":
            y = y + dense_ff(weights, f"l{i}.mlp.", h)
        elif f is not None:
            seen = aux.setdefault(call, {}) if aux is not None else None
            y = y + moe_ff(f, weights, f"l{i}.mlp.", h, None if picks is None else picks.get(call), seen)
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return (rms(x, _w(weights, "final.norm"), eps) @ _w(weights, "head").T) * cfg["logit_scale"]
