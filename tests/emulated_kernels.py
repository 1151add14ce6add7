"""Plain torch versions of every function of ``locus_b200.kernels``, same signatures.

Two uses.  (1) ``install()`` swaps them in so that the engine's host logic -- paging,
portions, mixed batches, scheduling, graphs of parts -- runs on the CPU in the ``not gpu``
tests.  (2) The ``gpu`` tests call them on copies of a kernel's inputs as that kernel's
plain reference.  They compute in float32 (or float64 when ``PRECISE`` is set), with plain
loops; they are not a product path and nothing in ``locus_b200`` imports them.
"""
from __future__ import annotations


import torch

import locus_b200.kernels as K

PRECISE = False


def _f(t: torch.Tensor) -> torch.Tensor:
    return t.to(torch.float64 if PRECISE else torch.float32)


def embed_rows(tokens, table, out, copies=1, scale=1.0, dyt_norm=None, positions=None, pos_table=None, keep=None):
    rows = _f(table[tokens.long()]) * scale
    if pos_table is not None:
        rows = rows + _f(pos_table[positions[: len(tokens)].long()])
    if dyt_norm is not None:
        rows = _dyt(rows, dyt_norm)
    out.copy_(rows.to(out.dtype).repeat(1, copies))
    if keep is not None:
        keep.copy_(rows.to(keep.dtype))


def add_rows(x, y):
    x += y.to(x.dtype)


def _dyt(z, norm):
    alpha, w, b = norm
    return torch.tanh(_f(alpha) * z) * _f(w) + _f(b)


def dyt(x, norm=None, out=None, rows=None, add=None):
    n = x.shape[0] if out is None else out.shape[0]
    pick = slice(0, n) if rows is None else rows.long()
    u = _f(x[pick])
    if add is not None:
        y, y_norm, scale = add
        u = u + (1.0 if scale is None else _f(scale)) * _dyt(_f(y[pick]), y_norm)
        if rows is None:
            x[:n] = u.to(x.dtype)
    if out is not None:
        out.copy_(_dyt(u, norm).to(out.dtype))


def attn_chunk_tc_takes(q, head_dim, page_tokens, n_tokens, max_ctx=0):
    return False


def rmsnorm_adds(x):
    return x.dtype == torch.float32 and x.shape[-1] % 4 == 0


def rmsnorm(x, w, eps, out, rows=None, add=None, add_rows=None):
    if rows is not None and (add is not None or add_rows is not None):
        x = x.clone()
    if add is not None:
        moe_combine(x if rows is not None else x[: out.shape[0]], add[0], add[1], add[2])
    if add_rows is not None:
        x += add_rows.to(x.dtype)
    xs = _f(x if rows is None else x[rows.long()])[: out.shape[0]]
    ss = (xs * xs).sum(-1, keepdim=True)
    out.copy_((xs * (1.0 / torch.sqrt(ss / xs.shape[-1] + eps)) * _f(w)).to(out.dtype))


class ExpertLayout(K.ExpertLayout):
    pass


def linear(x, w, out, *, w2=None, bias=None, accumulate=False, row_scale=None, scale_rows=None, x_rows=None, lists_ready=False,
           second_tiles=False,
           x_row_div=1, layout=None, n_rows=None, act=None, act_limit=0.0, act_scale=1.0):
    assert act in (None, "relu2", "glu_clamp", "softcap", "reglu") and not (act == "relu2" and w2 is not None)
    assert act != "reglu" or w2 is not None
    assert act != "glu_clamp" or (w2 is not None and act_limit > 0)
    assert act != "softcap" or (w2 is None and act_limit > 0)
    M = out.shape[0] if n_rows is None else n_rows
    if M == 0:
        return
    rs_all = None
    if row_scale is not None:
        rs_all = _f(row_scale[scale_rows[:M].long()] if scale_rows is not None else row_scale[:M])[:, None]

    def unit(g, u, rows):
        """Two products of the same rows into one: SwiGLU, the rectified gate with its two biases, or the clamped gated unit
        with the rows' scale in front."""
        if act == "reglu":
            b, b2 = (_f(bias[: g.shape[1]]), _f(bias[g.shape[1]:])) if bias is not None else (0.0, 0.0)
            return torch.clamp(g + b, min=0.0) * (u + b2)
        if act != "glu_clamp":
            return g / (1.0 + torch.exp(-g)) * u
        s = rs_all[rows] if rs_all is not None else 1.0
        g = torch.clamp(g * s, max=act_limit)
        u = torch.clamp(u * s, min=-act_limit, max=act_limit)
        return g / (1.0 + torch.exp(-1.702 * g)) * (u + 1.0)

    if x_rows is not None:
        xin = _f(x)[(x_rows[:M].long() // x_row_div)]
    else:
        xin = _f(x)[:M]
    if layout is None:
        y = xin @ _f(w).T
        if w2 is not None:
            y = unit(y, xin @ _f(w2).T, slice(0, M))
    else:
        y = torch.zeros(M, w.shape[1], dtype=xin.dtype)
        off = layout.offsets.tolist()
        for e in range(w.shape[0]):   # experts behind the weights have none: their rows are not this product's
            a, b = off[e], off[e + 1]
            if b > a:
                ye = xin[a:b] @ _f(w[e]).T
                if w2 is not None:
                    ye = unit(ye, xin[a:b] @ _f(w2[e]).T, slice(a, b))
                y[a:b] = ye
    if bias is not None and act != "reglu":
        y = y + _f(bias)
    if act == "relu2":
        y = torch.clamp(y, min=0.0) ** 2
    if rs_all is not None and act != "glu_clamp":
        y = y * rs_all
    if act == "softcap":
        y = act_limit * torch.tanh(y * act_scale / act_limit)
    if layout is not None:
        M = min(M, int(layout.offsets[w.shape[0]]))   # a grouped product writes the rows of its experts only
        y = y[:M]
    if accumulate:
        out[:M] += y.to(out.dtype)
    else:
        out[:M] = y.to(out.dtype)


def rope_kv_write(qkv, positions, inv_freq, q_out, pool, slots, *, n_heads, n_kv_heads, head_dim, rot_dim,
                  interleaved, page_tokens, write_kv=True):
    T = qkv.shape[0]
    x = _f(qkv).view(T, n_heads + 2 * n_kv_heads, head_dim).clone()
    if inv_freq is not None:
        ang = positions[:T].to(torch.float32)[:, None] * inv_freq[None, :].to(torch.float32)
        c, s = _f(torch.cos(ang))[:, None, :], _f(torch.sin(ang))[:, None, :]
        rot = x[:, : n_heads + n_kv_heads, :rot_dim]
        if interleaved:
            x0, x1 = rot[..., 0::2].clone(), rot[..., 1::2].clone()
            rot[..., 0::2] = x0 * c - x1 * s
            rot[..., 1::2] = x0 * s + x1 * c
        else:
            h = rot_dim // 2
            x0, x1 = rot[..., :h].clone(), rot[..., h:].clone()
            rot[..., :h] = x0 * c - x1 * s
            rot[..., h:] = x0 * s + x1 * c
    q_out[:T] = x[:, :n_heads].reshape(T, -1).to(q_out.dtype)
    if not write_kv:
        return
    for t in range(T):
        page, off = int(slots[t]) // page_tokens, int(slots[t]) % page_tokens
        pool[page, 0, :, off, :] = x[t, n_heads : n_heads + n_kv_heads].to(pool.dtype)
        pool[page, 1, :, off, :] = x[t, n_heads + n_kv_heads :].to(pool.dtype)


def _attend_one(q, pool, table, p, kvh, page_tokens, window, scale, keep_first=0, sink=False, head=0, chunk=0, slopes=None):
    lo = max(0, p - window + 1) if window > 0 else (p - p % chunk if chunk > 0 else 0)
    ts = list(range(0, min(keep_first, lo))) + list(range(lo, p + 1))
    pages = [int(table[t // page_tokens]) for t in ts]
    assert all(pg >= 0 for pg in pages), "attention reads a page that was given back"
    k = torch.stack([_f(pool[pg, 0, kvh, t % page_tokens]) for pg, t in zip(pages, ts)])
    v = torch.stack([_f(pool[pg, 1, kvh, t % page_tokens]) for pg, t in zip(pages, ts)])
    s = (k @ _f(q)) * scale
    if slopes is not None:
        s = s - _f(slopes)[head] * (p - torch.tensor(ts, dtype=s.dtype))
    if isinstance(sink, torch.Tensor):     # a learned score per head, as it is
        s = torch.cat([s, _f(sink)[head].view(1)])
        return torch.softmax(s, dim=0)[:-1] @ v
    if sink:
        s = torch.cat([s, s.new_zeros(1)])
        return torch.softmax(s, dim=0)[:-1] @ v
    a = torch.softmax(s, dim=0)
    return a @ v


def _attn(q, pool, out, seg_list, *, seg_q0, seg_qn, seg_ctx, block_table, n_heads, n_kv_heads, head_dim,
          page_tokens, window, scale, keep_first=0, sink=False, chunk=0, slopes=None):
    group = n_heads // n_kv_heads
    for seg in seg_list:
        q0, qn, ctx = int(seg_q0[seg]), int(seg_qn[seg]), int(seg_ctx[seg])
        for i in range(qn):
            for h in range(n_heads):
                qv = q[q0 + i].view(n_heads, head_dim)[h]
                o = _attend_one(qv, pool, block_table[seg], ctx + i, h // group, page_tokens, window, scale, keep_first, sink, head=h,
                                chunk=chunk, slopes=slopes)
                out[q0 + i].view(n_heads, head_dim)[h] = o.to(out.dtype)


def attn_chunk(q, pool, out, *, seg_q0, seg_qn, seg_ctx, block_table, items, n_items, n_heads, n_kv_heads,
               head_dim, page_tokens, window, scale, keep_first=0, sink=False, chunk=0, slopes=None):
    segs = sorted({int(items[i, 0]) for i in range(n_items)})
    _attn(q, pool, out, segs, seg_q0=seg_q0, seg_qn=seg_qn, seg_ctx=seg_ctx, block_table=block_table,
          n_heads=n_heads, n_kv_heads=n_kv_heads, head_dim=head_dim, page_tokens=page_tokens, window=window,
          scale=scale, keep_first=keep_first, sink=sink, chunk=chunk, slopes=slopes)


def attn_chunk_mma_splits(n_items, n_heads, max_ctx):
    return 1


def attn_chunk_mma(q, pool, out, *, seg_q0, seg_qn, seg_ctx, block_table, items, n_items, n_heads, n_kv_heads,
                   head_dim, page_tokens, window, scale, n_splits=1, part_o=None, part_ml=None, keep_first=0, sink=False, chunk=0,
                   slopes=None):
    attn_chunk(q, pool, out, seg_q0=seg_q0, seg_qn=seg_qn, seg_ctx=seg_ctx, block_table=block_table, items=items,
               n_items=n_items, n_heads=n_heads, n_kv_heads=n_kv_heads, head_dim=head_dim, page_tokens=page_tokens,
               window=window, scale=scale, keep_first=keep_first, sink=sink, chunk=chunk, slopes=slopes)


def attn_decode(q, pool, out, *, seg_q0, seg_qn, seg_ctx, block_table, items, n_items, n_heads, n_kv_heads,
                head_dim, page_tokens, window, scale, part_o, part_ml, counters, max_splits, keep_first=0, sink=False, chunk=0,
                slopes=None):
    segs = [int(items[i]) for i in range(n_items)]
    for s in segs:
        assert int(seg_ctx[s]) // K.DECODE_SPLIT + 1 <= max_splits
    _attn(q, pool, out, segs, seg_q0=seg_q0, seg_qn=seg_qn, seg_ctx=seg_ctx, block_table=block_table,
          n_heads=n_heads, n_kv_heads=n_kv_heads, head_dim=head_dim, page_tokens=page_tokens, window=window,
          scale=scale, keep_first=keep_first, sink=sink, chunk=chunk, slopes=slopes)


def _select(logits_row, top_k, renorm, scale, score_fn, sel_bias, n_group, n_group_used, group_score="top2"):
    """The selection rule of csrc/moe_route.cu (select_token) for one token."""
    E = logits_row.shape[0]
    r = logits_row
    if score_fn == "softmax":
        e = torch.exp(r - r.max())
        p = e / e.sum()
    else:
        p = 1.0 / (1.0 + torch.exp(-r))
    sel = p.clone() if sel_bias is None else p + sel_bias.to(p.dtype).cpu()
    if score_fn == "sigmoid" and sel_bias is None and n_group <= 1:
        sel = r.clone()     # ranked by the logits: the same order, no ties where the sigmoid rounds to one score
    sel = torch.clamp(torch.where(torch.isnan(sel), torch.full_like(sel, -3.0e38), sel), min=-3.0e38)
    if n_group > 1:
        per = E // n_group
        gs = []
        for g in range(n_group):
            top2 = torch.sort(torch.cat([sel[g * per : (g + 1) * per], torch.full((2,), -1e30, dtype=sel.dtype)]), descending=True).values
            gs.append(float(top2[0]) + (float(top2[1]) if per > 1 and group_score == "top2" else 0.0))
        keep = []
        for _ in range(n_group_used):
            keep.append(max((g for g in range(n_group) if g not in keep), key=lambda g: (gs[g], -g)))
        for x in range(E):
            if x // per not in keep:
                sel[x] = -1e30
    picked = []
    for _ in range(top_k):
        best = max((x for x in range(E) if x not in picked), key=lambda x: (float(sel[x]), -x))
        picked.append(best)
    wsum = sum(p[x] for x in picked) + (1e-20 if score_fn == "sigmoid" else 0.0) if renorm else 1.0
    return picked, [float(p[x] / wsum * scale) for x in picked]


def router_topk(h, w_router, w_gate, ids, wts, gamma, *, top_k, renorm, scale=1.0, scratch=None, score_fn="softmax",
                sel_bias=None, n_group=1, n_group_used=1, logit_bias=None, group_score="top2"):
    T = h.shape[0]
    r = _f(h) @ _f(w_router).T
    if logit_bias is not None:
        r = r + _f(logit_bias[: r.shape[1]])
    for t in range(T):
        picked, w = _select(r[t], top_k, renorm, scale, score_fn, sel_bias, n_group, n_group_used, group_score)
        for j, e in enumerate(picked):
            ids[t * top_k + j] = e
            wts[t * top_k + j] = w[j]
    if w_gate is not None:
        z = _f(h) @ _f(w_gate).reshape(-1)
        gamma[:T] = (1.0 / (1.0 + torch.exp(-z))).to(gamma.dtype)


def router_logits(h, w_all, logits, bias=None):
    T, n = h.shape[0], w_all.shape[0]
    z = _f(h) @ _f(w_all).T
    if bias is not None:
        z = z + _f(bias[:n])
    logits[:T, :n] = z.to(logits.dtype)


def router_select(logits, n_experts, has_gate, ids, wts, gamma, *, n_tokens, top_k, renorm, scale=1.0,
                  score_fn="softmax", sel_bias=None, n_group=1, n_group_used=1, group_score="top2"):
    lg = _f(logits[:n_tokens, :n_experts])
    for t in range(n_tokens):
        picked, w = _select(lg[t], top_k, renorm, scale, score_fn, sel_bias, n_group, n_group_used, group_score)
        for j, e in enumerate(picked):
            ids[t * top_k + j] = e
            wts[t * top_k + j] = w[j]
    if has_gate:
        z = _f(logits[:n_tokens, n_experts])
        gamma[:n_tokens] = (1.0 / (1.0 + torch.exp(-z))).to(gamma.dtype)


def route_small_takes(n_tokens, top_k, n_experts):
    return n_tokens <= 16 and n_tokens * top_k <= 1024 and n_experts <= 512


def route_small(logits, n_experts, has_gate, ids, wts, gamma, layout, *, n_tokens, top_k, renorm, scale=1.0,
                tile_m=None, **rule):
    router_select(logits, n_experts, has_gate, ids, wts, gamma, n_tokens=n_tokens, top_k=top_k, renorm=renorm,
                  scale=scale, **rule)
    moe_sort(ids, n_tokens * top_k, layout, tile_m)


def route_fused_small(h, w_all, logits, n_experts, has_gate, ids, wts, gamma, layout, counter, *, n_tokens, tile_m=None,
                      logit_bias=None, **rule):
    router_logits(h[:n_tokens], w_all, logits, bias=logit_bias)
    route_small(logits, n_experts, has_gate, ids, wts, gamma, layout, n_tokens=n_tokens, tile_m=tile_m, **rule)


def moe_sort(ids, n_pairs, layout, tile_m=None, tile2_m=0):
    if tile_m is not None:
        layout.tile_m = tile_m
    layout.tile2_m = tile2_m
    E, tm = layout.n_experts, layout.tile_m
    idl = ids[:n_pairs].tolist()
    pos = 0
    tile = tile2 = 0
    for e in range(E):
        mine = [p for p, x in enumerate(idl) if x == e]
        layout.counts[e] = len(mine)
        layout.offsets[e] = pos
        for i in range(0, len(mine), tm):
            layout.tile_expert[tile] = e
            layout.tile_row0[tile] = pos + i
            layout.tile_rows[tile] = min(tm, len(mine) - i)
            tile += 1
        for i in range(0, len(mine), tile2_m) if tile2_m else ():
            layout.tile2_expert[tile2] = e
            layout.tile2_row0[tile2] = pos + i
            layout.tile2_rows[tile2] = min(tile2_m, len(mine) - i)
            tile2 += 1
        for p in mine:
            layout.sorted_pair[pos] = p
            layout.pair_pos[p] = pos
            pos += 1
    layout.offsets[E] = pos
    layout.n_tiles[0] = tile
    if tile2_m:
        layout.n_tiles2[0] = tile2


def moe_combine(x, pair_out, pair_pos, top_k):
    T = x.shape[0]
    for t in range(T):
        acc = torch.zeros_like(x[t])
        for s in range(top_k):
            acc = acc + pair_out[int(pair_pos[t * top_k + s])].to(acc.dtype)
        x[t] += acc


def gather_rows(src, idx, div, out, n):
    out[:n] = src[(idx[:n].long() // div)]


def apply_penalties(logits, history, repeat, freq, presence):
    R, V = logits.shape
    for r in range(R):
        rp, fp, pp = float(repeat[r]), float(freq[r]), float(presence[r])
        if rp == 1.0 and fp == 0.0 and pp == 0.0:
            continue
        counts = {}
        for t in history[r].tolist():
            if 0 <= t < V:
                counts[t] = counts.get(t, 0) + 1
        for t, c in counts.items():
            l = float(logits[r, t])
            if rp != 1.0:
                l = l / rp if l > 0 else l * rp
            logits[r, t] = l - (fp * c + pp)


def sample(logits, *, temperature, top_k, top_p, min_p, seeds, counters, out, kept_count=None):
    """Greedy rows exactly; stochastic rows by torch's generator seeded from (seed, counter)
    over the same kept set (the device kernel has its own counter-based generator)."""
    R, V = logits.shape
    for r in range(R):
        row = logits[r].double()
        T = float(temperature[r])
        if not T > 0:
            out[r] = int(torch.argmax(row))  # first maximum
            continue
        keep = torch.ones(V, dtype=torch.bool)
        k = int(top_k[r])
        if 0 < k < V:
            thr = torch.sort(row, descending=True).values[k - 1]
            keep &= row >= thr
        w = torch.where(keep, torch.exp((row - row.max()) / T), torch.zeros_like(row))
        tp = float(top_p[r])
        if tp < 1.0:
            sw, _ = torch.sort(w, descending=True)
            cum = torch.cumsum(sw, 0)
            j = int(torch.nonzero(cum >= tp * w.sum())[0])
            keep &= w >= sw[j]
        mp = float(min_p[r])
        if mp > 0:
            keep &= w >= mp * w.max()
        w = torch.where(keep, w, torch.zeros_like(w))
        g = torch.Generator().manual_seed((int(seeds[r]) * 1000003 + int(counters[r])) & 0x7FFFFFFF)
        out[r] = int(torch.multinomial(w / w.sum(), 1, generator=g))
        if kept_count is not None:
            kept_count[r] = int(keep.sum())


def cast_rows(x, out):
    out.copy_(x.to(out.dtype))


def rmsnorm_add(y, w, eps, x):
    ys = _f(y)
    x += (ys / torch.sqrt((ys * ys).mean(-1, keepdim=True) + eps) * _f(w)).to(x.dtype)


def _turn(x, positions, freq, magnitude, rot_pairs, half_split=False):
    """x [T, ..., n]: interleaved pairs (2i, 2i + 1), i < rot_pairs, turned by positions[t] * freq[i]; ``half_split``:
    the pairs (i, i + rot_pairs)."""
    if rot_pairs == 0:
        return x
    if half_split:
        n = 2 * rot_pairs
        mixed = torch.stack([x[..., :rot_pairs], x[..., rot_pairs:n]], -1).reshape(*x.shape[:-1], n)
        t = _turn(torch.cat([mixed, x[..., n:]], -1), positions, freq, magnitude, rot_pairs)
        return torch.cat([t[..., 0:n:2], t[..., 1:n:2], t[..., n:]], -1)
    T = x.shape[0]
    ang = positions[:T].to(torch.float64)[:, None] * freq[:rot_pairs].to(torch.float64)[None, :]
    shape = [T] + [1] * (x.dim() - 2) + [rot_pairs]
    c = (torch.cos(ang) * magnitude).to(x.dtype).view(shape)
    s = (torch.sin(ang) * magnitude).to(x.dtype).view(shape)
    out = x.clone()
    u, v = x[..., 0:2 * rot_pairs:2], x[..., 1:2 * rot_pairs:2]
    out[..., 0:2 * rot_pairs:2] = u * c - v * s
    out[..., 1:2 * rot_pairs:2] = v * c + u * s
    return out


def latent_prep(dqkv, positions, freq, magnitude, w_q, w_kv, eps, cq_out, pool, slots, *, q_rank, kv_rank, rot_dim,
                rot_pairs, write=True, half_split=False):
    T = dqkv.shape[0]
    x = _f(dqkv)

    def unit(v):
        return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)

    if q_rank:
        cq_out[:T] = (unit(x[:, :q_rank]) * _f(w_q)).to(cq_out.dtype)
    if not write:
        return
    c = unit(x[:, q_rank:q_rank + kv_rank]) * _f(w_kv)
    kr = _turn(x[:, q_rank + kv_rank:q_rank + kv_rank + rot_dim], positions, freq, magnitude, rot_pairs, half_split)
    rows = torch.cat([c, kr], -1).to(pool.dtype)
    page_tokens = pool.shape[-2]
    for t in range(T):
        pool[int(slots[t]) // page_tokens, 0, 0, int(slots[t]) % page_tokens] = rows[t]


def latent_q_split(q, positions, freq, magnitude, q_nope_hm, q_rot, *, n_heads, nope_dim, rot_dim, rot_pairs, half_split=False):
    T = q.shape[0]
    x = _f(q).view(T, n_heads, nope_dim + rot_dim)
    q_nope_hm[: n_heads * T] = x[..., :nope_dim].transpose(0, 1).reshape(n_heads * T, nope_dim).to(q_nope_hm.dtype)
    q_rot[:T] = _turn(x[..., nope_dim:], positions, freq, magnitude, rot_pairs, half_split).reshape(T, -1).to(q_rot.dtype)


def latent_attn(q_abs_hm, q_rot, pool, sink, out_hm, *, seg_q0, seg_qn, seg_ctx, block_table, items, n_items, n_tokens,
                n_heads, kv_rank, rot_dim, page_tokens, window, scale):
    T = n_tokens
    done = set()
    for it in range(n_items):
        seg = int(items[it, 0])
        if seg in done:
            continue
        done.add(seg)
        q0, qn, ctx = int(seg_q0[seg]), int(seg_qn[seg]), int(seg_ctx[seg])
        for i in range(qn):
            p = ctx + i
            lo = max(0, p - window + 1) if window > 0 else 0
            pages = [int(block_table[seg, t // page_tokens]) for t in range(lo, p + 1)]
            assert all(pg >= 0 for pg in pages), "latent attention reads a page that was given back"
            rows = torch.stack([_f(pool[pg, 0, 0, t % page_tokens]) for pg, t in zip(pages, range(lo, p + 1))])
            for h in range(n_heads):
                qa = _f(q_abs_hm[h * T + q0 + i])
                qr = _f(q_rot[q0 + i]).view(n_heads, rot_dim)[h]
                s = (rows[:, :kv_rank] @ qa + rows[:, kv_rank:] @ qr) * scale
                big = s.max() if sink is None else torch.maximum(s.max(), _f(sink)[h])
                e = torch.exp(s - big)
                den = e.sum() + (torch.exp(_f(sink)[h] - big) if sink is not None else 0.0)
                out_hm[h * T + q0 + i] = ((e / den) @ rows[:, :kv_rank]).to(out_hm.dtype)


def latent_decode_takes(dtype, kv_rank, rot_dim):
    return False


def latent_decode_ranges(n_items, n_heads, max_keys):
    return 1


def latent_decode(q_abs_hm, q_rot, pool, sink, out_hm, *, seg_q0, seg_ctx, block_table, items, n_items, n_tokens, n_heads, kv_rank,
                  rot_dim, page_tokens, window, scale, n_ranges=1, part_o=None, part_ml=None):
    pairs = torch.stack([items[:n_items], torch.zeros_like(items[:n_items])], 1)
    latent_attn(q_abs_hm, q_rot, pool, sink, out_hm, seg_q0=seg_q0, seg_qn=torch.ones_like(seg_ctx), seg_ctx=seg_ctx, block_table=block_table,
                items=pairs, n_items=n_items, n_tokens=n_tokens, n_heads=n_heads, kv_rank=kv_rank, rot_dim=rot_dim, page_tokens=page_tokens,
                window=window, scale=scale)


def latent_gather(pool, out, *, segs, n_segs, row0, seg_qn, seg_ctx, block_table, page_tokens, longest):
    for i in range(n_segs):
        s = int(segs[i])
        n = int(seg_ctx[s]) + int(seg_qn[s])
        assert n <= longest
        for t in range(n):
            page = int(block_table[s, t // page_tokens])
            out[int(row0[s]) + t] = pool[page, 0, 0, t % page_tokens, : out.shape[1]] if page >= 0 else 0.0


def attn_chunk_tc_splits(n_items, n_heads, max_ctx, n_rows=0):
    return 1


def attn_chunk_tc_rows(q, k, v, out, *, seg_q0, seg_qn, seg_ctx, kv_row0, items, n_items, n_heads, n_kv_heads, head_dim, window, scale,
                       n_splits=1, part_o=None, part_ml=None, keep_first=0, sink=False, chunk=0, slopes=None):
    assert window == 0 and keep_first == 0 and chunk == 0
    group = n_heads // n_kv_heads
    for seg in sorted({int(items[i, 0]) for i in range(n_items)}):
        q0, qn, ctx, r0 = int(seg_q0[seg]), int(seg_qn[seg]), int(seg_ctx[seg]), int(kv_row0[seg])
        for i in range(qn):
            p = ctx + i
            for h in range(n_heads):
                cols = slice((h // group) * head_dim, (h // group + 1) * head_dim)
                s = (_f(k[r0:r0 + p + 1, cols]) @ _f(q[q0 + i].view(n_heads, head_dim)[h])) * scale
                if slopes is not None:
                    s = s - _f(slopes)[h] * (p - torch.arange(p + 1, dtype=s.dtype))
                if sink is not False:
                    s = torch.cat([s, (_f(sink)[h] if isinstance(sink, torch.Tensor) else s.new_zeros(())).view(1)])
                w = torch.softmax(s, 0)[: p + 1]
                out[q0 + i].view(n_heads, head_dim)[h] = (w @ _f(v[r0:r0 + p + 1, cols])).to(out.dtype)


def latent_attn_mma_takes(dtype, kv_rank, rot_dim):
    return False


def heads_to_rows(src_hm, out, *, n_tokens, n_heads):
    d = src_hm.shape[1]
    out[:n_tokens] = src_hm[: n_heads * n_tokens].view(n_heads, n_tokens, d).transpose(0, 1).reshape(n_tokens, n_heads * d)


def retention_scan(qkvg, state, state_slots, seg_q0, seg_qn, n_seg, decay, k_scale, o_raw, *, n_heads, dim, v_dim,
                   short=True, long=True, longest_new=0):
    H, d, dv = n_heads, dim, v_dim
    for seg in range(n_seg):
        q0, qn, slot = int(seg_q0[seg]), int(seg_qn[seg]), int(state_slots[seg])
        S = _f(state[slot])
        for t in range(q0, q0 + qn):
            row = _f(qkvg[t])
            q, k = row[: H * d].view(H, d), row[H * d:2 * H * d].view(H, d) * k_scale
            v = row[2 * H * d:2 * H * d + H * dv].view(H, dv)
            S = _f(decay).view(H, 1, 1) * S + k[:, :, None] * v[:, None, :]
            o_raw[t] = torch.einsum("hdv,hd->hv", S, q).reshape(-1).to(o_raw.dtype)
        state[slot] = S.to(state.dtype)


def retention_gate_norm(o_raw, qkvg, gate_offset, eps, out, *, n_heads, v_dim):
    T = out.shape[0]
    o = _f(o_raw[:T]).view(T, n_heads, v_dim)
    g = _f(qkvg[:T, gate_offset:gate_offset + n_heads * v_dim]).view(T, n_heads, v_dim)
    unit = o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps)
    out[:T] = (unit * (g / (1.0 + torch.exp(-g)))).reshape(T, -1).to(out.dtype)


def layernorm(x, w, b, eps, out, rows=None, n_streams=1, coef=None):
    n, H = out.shape
    xs = _f(x if rows is None else x[rows.long()])[:n].view(n, n_streams, H)
    c = _f(coef) if coef is not None else torch.ones(n_streams, dtype=xs.dtype)
    u = (xs * c[None, :, None]).sum(1)
    d = u - u.mean(-1, keepdim=True)
    out.copy_((d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * _f(w) + _f(b)).to(out.dtype))


def embed_pair(tokens, positions, table, pair, out, *, seg_q0, seg_qn, state_slots, last, n_seg, longest_new, mul_prev, mul_cur):
    buckets = pair.shape[0] - 1
    for seg in range(n_seg):
        q0, qn, slot = int(seg_q0[seg]), int(seg_qn[seg]), int(state_slots[seg])
        assert qn <= longest_new
        for i in range(qn):
            t = q0 + i
            tok = int(tokens[t])
            r = buckets
            if int(positions[t]) > 0:
                prev = int(tokens[t - 1]) if i > 0 else int(last[slot, 0])
                r = (prev * mul_prev + tok * mul_cur) % buckets
            out[t] = (_f(table[tok]) + _f(pair[r])).to(out.dtype)
    for seg in range(n_seg):
        if int(seg_qn[seg]) > 0:
            last[int(state_slots[seg]), 0] = int(tokens[int(seg_q0[seg]) + int(seg_qn[seg]) - 1])


def layernorm_post(x, y, alpha, w, b, eps, cast=None):
    n = x.shape[0]
    u = alpha * _f(x) + _f(y[:n])
    d = u - u.mean(-1, keepdim=True)
    x.copy_((d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * _f(w) + _f(b)).to(x.dtype))
    if cast is not None:
        cast[:n] = x.to(cast.dtype)


def span_rmsnorm(x, spans, eps):
    for off, n, w in spans:
        v = _f(x[:, off:off + n])
        x[:, off:off + n] = (v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps) * _f(w)).to(x.dtype)


def gla_decay(z, off, n, tau):
    v = _f(z[:, off:off + n])
    z[:, off:off + n] = (-torch.expm1(-torch.nn.functional.softplus(-v) / tau)).to(z.dtype)


def gla_scan(q, off_q, k, off_k, v, off_v, decay, off_a, state, state_offset, state_slots, seg_q0, seg_qn, n_seg, out, *,
             n_heads, dim, v_dim, q_scale):
    H, d, dv = n_heads, dim, v_dim
    for seg in range(n_seg):
        q0, qn, slot = int(seg_q0[seg]), int(seg_qn[seg]), int(state_slots[seg])
        S = _f(state[slot, state_offset:state_offset + H * d * dv]).view(H, d, dv).clone()
        for i in range(qn):
            r = q0 + i
            qv = _f(q[r, off_q:off_q + H * d]).view(H, d)
            kv = _f(k[r, off_k:off_k + H * d]).view(H, d)
            av = _f(decay[r, off_a:off_a + H * d]).view(H, d)
            vv = _f(v[r, off_v:off_v + H * dv]).view(H, dv)
            S = (S - av[:, :, None] * S) + kv[:, :, None] * vv[:, None, :]
            out[r] = (torch.einsum("hdv,hd->hv", S, qv) * q_scale).reshape(-1).to(out.dtype)
        state[slot, state_offset:state_offset + H * d * dv] = S.reshape(-1).to(state.dtype)


def stream_update(x, y, mix, out_coef, n_streams):
    n, H = y.shape
    old = _f(x[:n]).view(n, n_streams, H)
    new = torch.einsum("st,nsh->nth", _f(mix), old) + _f(out_coef)[None, :, None] * _f(y)[:, None, :]
    x[:n] = new.reshape(n, n_streams * H).to(x.dtype)


def moe_identity(h, wts, layout, pair_out, *, n_pairs, top_k, n_real):
    first = int(layout.offsets[n_real])
    for r in range(first, n_pairs):
        pair = int(layout.sorted_pair[r])
        pair_out[r] = (_f(wts[pair]) * _f(h[pair // top_k])).to(pair_out.dtype)
    for te, nt in ((layout.tile_expert, layout.n_tiles), (layout.tile2_expert, layout.n_tiles2)):
        if te is layout.tile2_expert and not layout.tile2_m:
            continue
        n = int(nt[0])
        cut = [i for i in range(n) if int(te[i]) >= n_real]
        if cut:
            nt[0] = cut[0]


def gated_recurrence(q, off_q, k, off_k, v, off_v, keep, take, state, state_offset, state_slots, seg_q0, seg_qn, n_seg,
                     out, *, n_heads, heads_per_group, dim, v_dim, ones=False, q_scale=1.0, short=True, long=True,
                     longest_new=0):
    H, d, dv = n_heads, dim, v_dim
    dvx = dv + (1 if ones else 0)
    G = H // heads_per_group
    grp = torch.arange(H) // heads_per_group
    for seg in range(n_seg):
        q0, qn, slot = int(seg_q0[seg]), int(seg_qn[seg]), int(state_slots[seg])
        S = _f(state[slot, state_offset:state_offset + H * d * dvx]).view(H, d, dvx).clone()
        for t in range(q0, q0 + qn):
            qq = _f(q[t, off_q:off_q + G * d]).view(G, d)[grp] * q_scale
            kk = _f(k[t, off_k:off_k + G * d]).view(G, d)[grp]
            vv = _f(v[t, off_v:off_v + H * dv]).view(H, dv)
            if ones:
                vv = torch.cat([vv, torch.ones(H, 1, dtype=vv.dtype)], 1)
            S = _f(keep[t]).view(H, 1, 1) * S + (_f(take[t]).view(H, 1) * kk)[:, :, None] * vv[:, None, :]
            out[t] = torch.einsum("hdv,hd->hv", S, qq).reshape(-1).to(out.dtype)
        state[slot, state_offset:state_offset + H * d * dvx] = S.reshape(-1).to(state.dtype)


def mlstm_gates(proj, off_i, off_f, cap, state, m_offset, state_slots, seg_q0, seg_qn, n_seg, keep, take, m_out, *, n_heads):
    H = n_heads
    for seg in range(n_seg):
        q0, qn, slot = int(seg_q0[seg]), int(seg_qn[seg]), int(state_slots[seg])
        m = _f(state[slot, m_offset:m_offset + H]).clone()
        for t in range(q0, q0 + qn):
            i = cap * torch.tanh(_f(proj[t, off_i:off_i + H]) / cap)
            f = torch.nn.functional.logsigmoid(cap * torch.tanh(_f(proj[t, off_f:off_f + H]) / cap))
            m_new = torch.maximum(f + m, i)
            keep[t] = torch.exp(f + m - m_new).to(keep.dtype)
            take[t] = torch.exp(i - m_new).to(take.dtype)
            m_out[t] = m_new.to(m_out.dtype)
            m = m_new
        state[slot, m_offset:m_offset + H] = m.to(state.dtype)


def mlstm_out(o_raw, m_t, proj, off_g, w, eps, out, *, n_heads, v_dim):
    T, H, dv = out.shape[0], n_heads, v_dim
    o = _f(o_raw[:T]).view(T, H, dv + 1)
    den = torch.maximum(o[..., dv].abs(), torch.exp(-_f(m_t[:T]))) + 1e-6
    u = o[..., :dv] / den[..., None]
    u = u / torch.sqrt((u * u).mean(-1, keepdim=True) + eps)
    g = _f(proj[:T, off_g:off_g + H * dv])
    out[:T] = (u.reshape(T, H * dv) * _f(w) * torch.sigmoid(g)).to(out.dtype)


def head_prep(proj, *, offsets, heads, dims, laid, state_slots, seg_q0, seg_qn, n_seg, longest_new, positions, q_out,
              k_out=None, v_out=None, pool=None, slots=None, page_tokens=0, write_kv=True, conv=None, state=None,
              conv_offset=0, move_state=True, act=False, inv_freq=None, rot=0, norm=None, eps=0.0, q_scale=1.0, gates=None,
              interleaved=False, norm_weights=None, n_rows=0, q_temp=None):
    widths = [h * d for h, d in zip(heads, dims)]
    C = sum(widths)
    taps = conv.shape[1] if conv is not None else 1
    for seg in range(n_seg):
        q0, qn, slot = int(seg_q0[seg]), int(seg_qn[seg]), int(state_slots[seg])
        if qn == 0:
            continue
        rows = slice(q0, q0 + qn)
        xin = torch.cat([_f(proj[rows, o:o + w]) for o, w in zip(offsets, widths)], 1)        # [qn, C]
        if conv is not None:
            if taps > 1:
                old = _f(state[slot, conv_offset:conv_offset + C * (taps - 1)]).view(C, taps - 1)
                full = torch.cat([old.T, xin], 0)
            else:
                full = xin
            y = torch.zeros_like(xin)
            for j in range(taps):
                y = y + full[j:j + qn] * _f(conv)[:, j]
            if taps > 1 and move_state:
                state[slot, conv_offset:conv_offset + C * (taps - 1)] = full[qn:].T.reshape(-1).to(state.dtype)
        else:
            y = xin
        if act:
            y = y / (1.0 + torch.exp(-y))
        at = 0
        for which in range(3):
            H, d, L = heads[which], dims[which], laid[which]
            x = y[:, at:at + H * d].reshape(qn, H, d).clone()
            at += H * d
            if H == 0 or (which > 0 and not write_kv):
                continue
            if which < 2 and norm == "head":
                x = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * _f(norm_weights[which])
            if which < 2 and inv_freq is not None and rot > 0:
                ang = positions[rows].to(torch.float32)[:, None] * inv_freq[None, :].to(torch.float32)
                c, s = _f(torch.cos(ang))[:, None, :], _f(torch.sin(ang))[:, None, :]
                half = rot // 2
                a, b = (slice(0, rot, 2), slice(1, rot, 2)) if interleaved else (slice(0, half), slice(half, rot))
                u, v = x[..., a].clone(), x[..., b].clone()
                x[..., a] = u * c - v * s
                x[..., b] = v * c + u * s
            if which < 2 and norm == "rms":
                x = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
            elif which < 2 and norm == "unit":
                x = x / torch.sqrt((x * x).sum(-1, keepdim=True) + eps)
            if which == 0:
                x = x * q_scale
                if q_temp is not None:
                    turns = torch.floor((positions[rows].double() + 1.0) / q_temp[1]) + 1.0
                    x = x * (1.0 + q_temp[0] * torch.log(_f(turns)))[:, None, None]
            padded = x.new_zeros(qn, H, L)
            padded[..., :d] = x
            if which == 0:
                q_out[rows] = padded.reshape(qn, H * L).to(q_out.dtype)
            elif pool is not None:
                for i in range(qn):
                    page, off = int(slots[q0 + i]) // page_tokens, int(slots[q0 + i]) % page_tokens
                    pool[page, which - 1, :, off, :] = padded[i].to(pool.dtype)
            else:
                (k_out if which == 1 else v_out)[rows] = padded.reshape(qn, H * L).to(q_out.dtype)
        if gates is not None:
            beta, decay, off_b, off_a, a_log, dt_bias = gates
            G = beta.shape[1]
            beta[rows] = torch.sigmoid(_f(proj[rows, off_b:off_b + G])).to(beta.dtype)
            dt = torch.nn.functional.softplus(_f(proj[rows, off_a:off_a + G]) + _f(dt_bias))
            decay[rows] = torch.exp(-torch.exp(_f(a_log)) * dt).to(decay.dtype)


def gate_rows(o, proj, off, *, n_heads, dim, laid):
    T = o.shape[0]
    g = torch.sigmoid(_f(proj[:T, off:off + n_heads * dim])).view(T, n_heads, dim)
    ov = o.view(T, n_heads, laid)
    ov[..., :dim] = (_f(ov[..., :dim]) * g).to(o.dtype)


def delta_rule(q, off_q, k, off_k, v, off_v, beta, decay, state, state_offset, state_slots, seg_q0, seg_qn, n_seg, out, *,
               n_heads, heads_per_group, dim, v_dim):
    H, d, dv = n_heads, dim, v_dim
    for seg in range(n_seg):
        q0, qn, slot = int(seg_q0[seg]), int(seg_qn[seg]), int(state_slots[seg])
        S = _f(state[slot, state_offset:state_offset + H * d * dv]).view(H, d, dv).clone()
        for i in range(qn):
            r = q0 + i
            for h in range(H):
                g = h // heads_per_group
                qv = _f(q[r, off_q + g * d: off_q + (g + 1) * d])
                kv = _f(k[r, off_k + g * d: off_k + (g + 1) * d])
                vv = _f(v[r, off_v + h * dv: off_v + (h + 1) * dv])
                S[h] = S[h] * _f(decay[r, h])
                u = _f(beta[r, h]) * (vv - S[h].T @ kv)
                S[h] = S[h] + kv[:, None] * u[None, :]
                out[r, h * dv:(h + 1) * dv] = (S[h].T @ qv).to(out.dtype)
        state[slot, state_offset:state_offset + H * d * dv] = S.reshape(-1).to(state.dtype)


def delta_out(o, proj, off_g, w, eps, out, *, n_heads, v_dim):
    T = out.shape[0]
    x = _f(o[:T]).view(T, n_heads, v_dim)
    x = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    wv = _f(w).view(-1, v_dim)     # [1, v_dim] (shared) or [heads, v_dim]
    z = _f(proj[:T, off_g:off_g + n_heads * v_dim]).view(T, n_heads, v_dim)
    out[:T] = (x * wv * (z / (1.0 + torch.exp(-z)))).reshape(T, -1).to(out.dtype)


def ssm_conv(proj, off_xbc, off_dt, conv_w, conv_b, dt_bias, a_log, state, conv_offset, state_slots, seg_q0, seg_qn, n_seg,
             act, keep, take, *, n_heads, longest_new=0):
    C, taps = conv_w.shape
    H = n_heads
    for seg in range(n_seg):
        q0, qn, slot = int(seg_q0[seg]), int(seg_qn[seg]), int(state_slots[seg])
        old = _f(state[slot, conv_offset:conv_offset + C * (taps - 1)]).view(C, taps - 1)
        xin = torch.cat([old.T, _f(proj[q0:q0 + qn, off_xbc:off_xbc + C])], 0)      # [taps - 1 + qn, C]
        acc = _f(conv_b)[None, :].repeat(qn, 1)
        for j in range(taps):
            acc = acc + xin[j:j + qn] * _f(conv_w)[:, j]
        act[q0:q0 + qn] = (acc / (1.0 + torch.exp(-acc))).to(act.dtype)
        state[slot, conv_offset:conv_offset + C * (taps - 1)] = xin[qn:].T.reshape(-1).to(state.dtype)
        dt = torch.nn.functional.softplus(_f(proj[q0:q0 + qn, off_dt:off_dt + H]) + _f(dt_bias))
        keep[q0:q0 + qn] = torch.exp(-torch.exp(_f(a_log)) * dt).to(keep.dtype)
        take[q0:q0 + qn] = dt.to(take.dtype)


def ssm_out(y, act, proj, off_z, d_skip, w, eps, out, *, parts, v_dim):
    T, inner = out.shape
    x = _f(act[:T, :inner])
    z = _f(proj[:T, off_z:off_z + inner])
    u = (_f(y[:T]) + _f(d_skip).repeat_interleave(v_dim)[None, :] * x) * (z / (1.0 + torch.exp(-z)))
    u = u.view(T, parts, inner // parts)
    u = u / torch.sqrt((u * u).mean(-1, keepdim=True) + eps)
    out[:T] = (u.reshape(T, inner) * _f(w)).to(out.dtype)


def head_tile(n_tokens, dtype, widths_ok):
    return 8 if (widths_ok and n_tokens <= 8) else 64


_NAMES = ["embed_rows", "rmsnorm", "rmsnorm_adds", "attn_chunk_tc_takes", "linear", "rope_kv_write", "attn_chunk", "attn_chunk_mma", "attn_decode", "router_topk", "router_logits", "router_select",
          "moe_sort", "route_small", "route_small_takes", "route_fused_small", "moe_combine", "gather_rows", "add_rows", "latent_gather", "latent_decode", "latent_decode_takes", "latent_decode_ranges", "attn_chunk_tc_splits", "attn_chunk_tc_rows", "apply_penalties", "sample",
          "cast_rows", "rmsnorm_add", "latent_prep", "latent_q_split", "latent_attn", "heads_to_rows", "retention_scan",
          "retention_gate_norm", "head_tile", "latent_attn_mma_takes", "layernorm", "stream_update", "moe_identity",
          "gated_recurrence", "mlstm_gates", "mlstm_out", "ssm_conv", "ssm_out", "head_prep", "gate_rows", "delta_rule", "delta_out",
          "embed_pair", "layernorm_post", "dyt", "span_rmsnorm", "gla_decay", "gla_scan"]


def install(monkeypatch) -> None:
    """Replace the CUDA entry points by the functions of this file (pytest monkeypatch)."""
    g = globals()
    for n in _NAMES:
        monkeypatch.setattr(K, n, g[n])
    from locus_b200.csrc import build
    monkeypatch.setattr(build, "ensure", lambda names, verbose=True: None)
