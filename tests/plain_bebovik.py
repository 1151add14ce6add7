"""The Bebovik design, plainly: float64, whole sequences, one function per mechanism, written from the equations.

Nothing here is shared with ``locus_b200``: the configuration is the raw nested dictionary of config.json and the weights
a dictionary of tensors by their stored names.  ``forward`` runs one sequence from its first token.

Notation: x [T, width] the residual stream, p a position counted from 0, D_n(z) = tanh(alpha_n z) * w_n + b_n the norm of
name n (a scalar alpha_n, vectors w_n and b_n; no statistics).

* embedding: x = D_embed(embed[token] * scale);
* layer: x <- x + ls1 * D_1b(mixer(D_1(x))); x <- x + ls2 * D_2b(ff(D_2(x)));
* mixer ``attention``: grouped queries; q and k divided by their root mean square per head and weighted, then their
  first ``dims`` elements rotated in adjacent pairs, the slow pairs' frequencies divided by a factor; a query sees the
  keys of its own chunk of ``size`` positions up to itself; the heads' outputs are multiplied by sigmoid(W_g h);
* feed-forward: W_down (g sigmoid(1.702 g) (u + 1)) with g = min(W_gate h, limit), u = clamp(W_up h, -limit, limit);
* output: z = logit_scale * head D_final(x); logits = cap * tanh(z / cap).
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def _w(weights, name):
    return weights[name].to(F64)


def dyt(weights, name, z):
    return torch.tanh(_w(weights, name + ".alpha") * z) * _w(weights, name) + _w(weights, name + ".b")


def head_rms(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def frequencies(rot):
    """The angle per position of every pair: base^(-2i/dims); with ``scaling``, a pair whose wavelength 2 pi / f is
    longer than original / low turns ``factor`` times slower, one that is shorter than original / high as before, and
    between them the two rates are blended linearly in original / wavelength."""
    fs = [float(rot["base"]) ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)]
    sc = rot.get("scaling")
    if not sc:
        return fs
    out = []
    for f in fs:
        turns = sc["original"] * f / (2.0 * math.pi)      # how often the pair turns over the original length
        if turns > sc["high"]:
            out.append(f)
        elif turns < sc["low"]:
            out.append(f / sc["factor"])
        else:
            s = (turns - sc["low"]) / (sc["high"] - sc["low"])
            out.append((1.0 - s) * f / sc["factor"] + s * f)
    return out


def rotate_adjacent(v, positions, rot):
    """v [T, heads, d]: the pairs (2i, 2i + 1) of the first ``dims`` elements turned by p * f_i, the rest as they are."""
    n = rot["dims"]
    ang = positions.to(F64)[:, None] * torch.tensor(frequencies(rot), dtype=F64)[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    out = v.clone()
    a, b = v[..., 0:n:2], v[..., 1:n:2]
    out[..., 0:n:2] = a * c - b * s
    out[..., 1:n:2] = b * c + a * s
    return out


def first_visible(p, mask):
    """The first key in sight of a query at position p."""
    return (p // mask["size"]) * mask["size"] if mask else 0


def attention(m, weights, pre, h, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = head_rms((h @ _w(weights, pre + "q").T).view(T, H, d), _w(weights, pre + "q.norm"), eps)
    k = head_rms((h @ _w(weights, pre + "k").T).view(T, G, d), _w(weights, pre + "k.norm"), eps)
    v = (h @ _w(weights, pre + "v").T).view(T, G, dv)
    rot = m.get("rot")
    if rot:
        q, k = rotate_adjacent(q, pos, rot), rotate_adjacent(k, pos, rot)
    out = torch.zeros(T, H, dv, dtype=F64)
    for i in range(T):
        lo = first_visible(i, m.get("mask"))
        for hd in range(H):
            g = hd // (H // G)
            s = (k[lo:i + 1, g] @ q[i, hd]) * m["scale"]
            out[i, hd] = torch.softmax(s, 0) @ v[lo:i + 1, g]
    gate = torch.sigmoid(h @ _w(weights, pre + "g").T)
    return (out.reshape(T, H * dv) * gate) @ _w(weights, pre + "o").T


def clamped_ff(f, weights, pre, h):
    lim = f["limit"]
    g = torch.clamp(h @ _w(weights, pre + "gate").T, max=lim)
    u = torch.clamp(h @ _w(weights, pre + "up").T, min=-lim, max=lim)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ _w(weights, pre + "down").T


def softcap(z, cap):
    return cap * torch.tanh(z / cap)


def forward(cfg, weights, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out``: a list that receives the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = _w(weights, "embed")[torch.tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    x = dyt(weights, "embed.norm", x)
    for i, layer in enumerate(cfg["layers"]):
        if layer["type"] != "attention":
            raise ValueError(layer["type"])
        y = attention(layer["mixer"], weights, f"l{i}.mix.", dyt(weights, f"l{i}.norm1", x), eps)
        x = x + dyt(weights, f"l{i}.norm1b", y) * _w(weights, f"l{i}.ls1")
        if layer.get("mlp") is not None:
            y = clamped_ff(layer["mlp"], weights, f"l{i}.mlp.", dyt(weights, f"l{i}.norm2", x))
            x = x + dyt(weights, f"l{i}.norm2b", y) * _w(weights, f"l{i}.ls2")
        if layers_out is not None:
            layers_out.append(x.clone())
    z = (dyt(weights, "final.norm", x) @ _w(weights, "head").T) * cfg["logit_scale"]
    return softcap(z, cfg["logit_softcap"])
