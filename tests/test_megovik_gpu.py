"""The Megovik design on the GPU against the plain implementation (float64), in float32 and in bfloat16: whole prompts,
decoding token by token, portions down to two tokens, mixed batches with pages that are used again; configurations drawn at
random on pages of 64; a key that stands out among hundreds, in prompts and while decoding; long decoding through CUDA
graphs; heads of 128 in long portions; the new kernels and the new forms of the others alone against their plain twins;
greedy generation through the engine's entry point and the command line; trace replay as a program.  Pages are filled with
NaN when they are made and when they go back."""
import functools
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import emulated_kernels as EK
import plain_megovik as plain
from megovik_cases import (Case, attention, compare, compare_together, dense, errors, latent, make_runner, model, moe, random_config,
                           run_steps, schedules, sharpen, with_mlp)

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEV = "cuda:0"

# max and mean |error| of the logits (their mean over the vocabulary taken off) relative to the largest |logit|
TOL = {torch.float32: (1e-4, 1e-5), torch.bfloat16: (5e-2, 8e-3)}
TIE = {torch.float32: 1e-4, torch.bfloat16: 8e-2}   # a router's near-tie, of the spread of its scores
DTYPES = [torch.float32, torch.bfloat16]
IDS = ["f32", "bf16"]
LENGTHS = {"mix": (1, 2, 37, 70, 45, 19, 130), "odd": (3, 90, 33, 16, 75), "wide": (150, 40, 260), "attention_only": (50, 23),
           "latents_only": (60, 5, 33), "dense_only": (20, 5), "moe_only": (40, 3)}


def _milder(dtype):
    """The factors on the projections nearer to 1 in bfloat16: with all of them a few positions amplify the rounding of the
    activations beyond what tells a fault from it."""
    return sharpen if dtype == torch.float32 else functools.partial(sharpen, strength=0.35)


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    made = {}

    def get(name, dtype):
        if (name, dtype) not in made:
            made[name, dtype] = Case(name, tmp_path_factory.mktemp("megovik"), torch.bfloat16, requests=LENGTHS[name], tweak=_milder(dtype))
        return made[name, dtype]

    return get


def _agree(case, got, routed, dtype):
    if dtype == torch.float32:
        compare(case, got, routed, *TOL[dtype], TIE[dtype])
    else:   # (eleven calls of sharpened layers: single rows amplify rounding)
        compare_together(case, got, routed, *TOL[dtype], TIE[dtype], cap=3.0)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("name", list(LENGTHS))
def test_every_schedule_agrees_with_plain(name, dtype, cases):
    case = cases(name, dtype)
    runner, cache = make_runner(case, dtype, DEV, page_tokens=16, n_pages=40, max_tokens=320)
    for sched_name, steps in schedules(case).items():
        got, routed = run_steps(runner, cache, case, steps)
        _agree(case, got, routed, dtype)
        assert cache.free_pages() == cache.total_pages() and cache.state_slots.free == cache.state_slots.total, sched_name


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("seed", list(range(6)))
def test_drawn_configurations_on_pages_of_64(seed, dtype, tmp_path_factory):
    """Configurations drawn at random: portions of changing size and mixed batches of four live requests on pages of 64
    whose pool only holds them when pages are used again."""
    case = Case(f"drawn{seed}", tmp_path_factory.mktemp("drawn"), torch.bfloat16, raw=random_config(700 + seed),
                requests=(230, 1, 150, 40, 97, 180), seed=seed, tweak=_milder(dtype))
    runner, cache = make_runner(case, dtype, DEV, page_tokens=64, n_pages=14, max_tokens=256, max_seq=512)
    sch = schedules(case)
    for name in ("mixed", "chunked"):
        got, routed = run_steps(runner, cache, case, sch[name])
        if dtype == torch.float32:
            compare(case, got, routed, 3e-4, 4e-5, TIE[dtype])
        else:
            compare_together(case, got, routed, *TOL[dtype], TIE[dtype], cap=3.0)
        assert cache.free_pages() == cache.total_pages()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("page_tokens", [8, 64])
def test_other_page_sizes_and_the_cuda_core_products(page_tokens, dtype, cases, monkeypatch):
    import locus_b200.kernels as K

    case = cases("mix", dtype)
    if page_tokens == 8:
        monkeypatch.setattr(K, "USE_TENSOR_CORES", False)   # bfloat16 on the CUDA-core products and attention
    runner, cache = make_runner(case, dtype, DEV, page_tokens=page_tokens, n_pages=24 if page_tokens == 64 else 90,
                                max_tokens=320, max_seq=1024)
    sch = schedules(case)
    for steps in (sch["mixed"], sch["chunked"]):
        got, routed = run_steps(runner, cache, case, steps)
        _agree(case, got, routed, dtype)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_heads_of_128_in_long_portions_on_pages_of_64(dtype, tmp_path_factory, monkeypatch):
    """Heads of 128, four query heads on every key/value head, latents of 512 and 320, portions of several hundred tokens (the
    kernels that long portions take), routed and dense feed-forwards over hundreds of rows."""
    import locus_b200.kernels as K

    raw = model(256, 301, [with_mlp(attention(8, 2, 128, scale=0.06, temp=(0.3, 64)), dense(192)),
                           with_mlp(latent(16, 64, 64, 512, scale=0.1), moe(16, 4, 96, groups=(4, 2), scale=2.0)),
                           with_mlp(latent(4, 128, 128, 320, q_rank=192, scale=0.06), None),
                           with_mlp(attention(4, 4, 128, scale=0.06), moe(8, 2, 128, scale=1.0))],
                loop=(1, 3, 2), emb=2.0, logit_scale=0.5)
    tweak = sharpen if dtype == torch.float32 else functools.partial(sharpen, strength=0.2)
    case = Case("big", tmp_path_factory.mktemp("big"), torch.bfloat16, raw=raw, requests=(700, 90), tweak=tweak)
    runner, cache = make_runner(case, dtype, DEV, page_tokens=64, n_pages=20, max_tokens=640, max_seq=1024)
    expanded = []
    rows = K.attn_chunk_tc_rows
    monkeypatch.setattr(K, "attn_chunk_tc_rows", lambda *a, **kw: (expanded.append(kw["n_items"]), rows(*a, **kw)))
    for steps in ([[("r0", 300), ("r1", 40)], [("r0", 399), ("r1", 1)], [("r0", 1), ("r1", 49)]],
                  [[("r0", 500), ("r1", 2)], [("r0", 72)], [("r0", 128), ("r1", 88)]]):
        got, routed = run_steps(runner, cache, case, steps)
        _agree(case, got, routed, dtype)
    # the second latent's keys and values (heads of 128) are expanded in portions of 64 tokens and more, in both passes
    assert expanded == ([5, 5, 7, 7, 8, 8, 2, 2, 4, 4] if dtype == torch.bfloat16 else [])


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("name", ["mix", "wide"])
def test_long_decoding_through_graphs(name, dtype, tmp_path):
    """Two requests decoded side by side for 200 tokens through CUDA graphs, past several pages and steps of the queries'
    factor: the replayed steps against the same steps launched kernel by kernel, and both against the plain implementation."""
    from locus_b200.engine.step import StepEntry

    case = Case(name, tmp_path, torch.bfloat16, requests=(230, 215), tweak=_milder(dtype))
    rows, picks = {}, {}
    for graphs in (False, True):
        runner, cache = make_runner(case, dtype, DEV, page_tokens=16, n_pages=40, max_tokens=64, use_graphs=graphs)
        seqs = {r: cache.open(r) for r in ("r0", "r1")}
        for r, n in (("r0", 30), ("r1", 15)):
            assert cache.ensure_capacity(seqs[r], n)
            runner.step([StepEntry(seqs[r], case.tokens[r][:n], [n - 1])])
        fed, got = {"r0": 30, "r1": 15}, []
        for _ in range(200):
            entries = []
            for r in ("r0", "r1"):
                assert cache.ensure_capacity(seqs[r], 1)
                entries.append(StepEntry(seqs[r], [case.tokens[r][fed[r]]], [0]))
                fed[r] += 1
            got.append(runner.step(entries).detach().cpu().double().clone())
        runner.check_device_errors()
        rows[graphs] = torch.stack(got)
        if graphs:
            assert runner.stats["graph_replays"] >= 190
    ref = torch.stack([case.ref("r0")[0][30:230], case.ref("r1")[0][15:215]], 1)
    tol = TOL[dtype]
    err, mean = errors(rows[True].reshape(400, -1), rows[False].reshape(400, -1))
    assert mean <= tol[1] and float(torch.quantile(err, 0.95)) <= tol[0], (float(err.max()), mean)
    # (the picks are not followed here: a router's near-tie may move a row, few rows may)
    err, mean = errors(rows[True].reshape(400, -1), ref.reshape(400, -1))
    assert mean <= 1.5 * tol[1] and float(torch.quantile(err, 0.9)) <= tol[0], (float(err.max()), mean)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("kind", ["attention", "latent", "latent2"])
def test_a_far_key_among_hundreds(kind, dtype, tmp_path_factory):
    """A key that stands out among up to hundreds of others: at the sequence's first position, at page borders and late; seen
    by queries in whole prompts, in portions, and decoded one by one."""
    from test_megovik_host import beacon_case, beacon_reach

    n, places = 420, (0, 15, 16, 255, 256, 390)
    case = beacon_case(tmp_path_factory.mktemp("beacon"), kind, n, places, torch.bfloat16)
    runner, cache = make_runner(case, dtype, DEV, page_tokens=16, n_pages=30, max_tokens=448, slots=1)
    for i, at in enumerate(places):
        r = f"r{i}"
        beacon_reach(case, r, at)
        for steps in ([[(r, n)]], [[(r, 396)]] + [[(r, 1)]] * 24, [[(r, 2)], [(r, 253)], [(r, 2)], [(r, 160)], [(r, 2)], [(r, 1)]]):
            got, routed = run_steps(runner, cache, case, steps)
            compare(case, got, routed, *TOL[dtype], TIE[dtype])


# ---------------------------------------------------------------------------
# the kernels alone against their plain twins (float64)


def _cmp(a, b, tol):
    a, b = a.double().cpu(), b.double().cpu()
    assert bool(torch.isfinite(a).all())
    assert float((a - b).abs().max()) <= tol * max(1.0, float(b.abs().max())), float((a - b).abs().max())


@pytest.fixture
def precise(monkeypatch):
    monkeypatch.setattr(EK, "PRECISE", True)


def test_the_embedding_with_position_vectors_and_kept_rows_against_its_twin(precise):
    import locus_b200.kernels as K

    g = torch.Generator().manual_seed(6)
    for dt, pdt in ((torch.float32, torch.float32), (torch.bfloat16, torch.bfloat16), (torch.bfloat16, torch.float32)):
        for H in (50, 640):
            table, pos_table = torch.randn(31, H, generator=g).to(dt), torch.randn(70, H, generator=g).to(pdt)
            toks, pos = (torch.randint(0, hi, (19,), generator=g, dtype=torch.int32) for hi in (31, 70))
            ref, kept = torch.zeros(19, H, dtype=torch.float64), torch.zeros(19, H, dtype=torch.float64)
            out, keep = torch.zeros(19, H, device=DEV), torch.zeros(19, H, device=DEV)
            EK.embed_rows(toks, table, ref, scale=3.5, positions=pos, pos_table=pos_table, keep=kept)
            K.embed_rows(toks.cuda(), table.cuda(), out, scale=3.5, positions=pos.cuda(), pos_table=pos_table.cuda(), keep=keep)
            _cmp(out, ref, 1e-6)
            assert torch.equal(out, keep)
            K.embed_rows(toks.cuda(), table.cuda(), out, scale=3.5, positions=pos.cuda(), pos_table=pos_table.cuda())
            assert torch.equal(out, keep)
    with pytest.raises(K.KernelError):
        K.embed_rows(toks.cuda(), table.cuda(), out, pos_table=pos_table.cuda())


@pytest.mark.parametrize("odt", DTYPES, ids=IDS)
@pytest.mark.parametrize("H,T,k", [(256, 1, 2), (2048, 70, 4), (4100, 9, 3), (20, 5, 1), (8192, 3, 2)])
def test_rmsnorm_with_rows_added_in_front(H, T, k, odt, precise):
    """The experts' sum and the rows, either alone and both, over all rows and over gathered ones; rows wider than the
    registers hold; the plain addition."""
    import locus_b200.kernels as K

    g = torch.Generator().manual_seed(H + T)
    x, y, w = torch.randn(T, H, generator=g), torch.randn(T, H, generator=g), torch.randn(H, generator=g).to(odt)
    pairs, pos = torch.randn(T * k, H, generator=g).to(torch.bfloat16), torch.randperm(T * k, generator=g).to(torch.int32)
    rows = torch.randint(0, T, (4,), generator=g, dtype=torch.int32)
    for add in (None, (pairs, pos, k)):
        for r in (None, rows):
            n = T if r is None else 4
            rx, ro = x.double(), torch.zeros(n, H, dtype=torch.float64)
            EK.rmsnorm(rx, w, 1e-5, ro, r, add=add, add_rows=y)
            dx, do = x.cuda(), torch.zeros(n, H, dtype=odt, device=DEV)
            K.rmsnorm(dx, w.cuda(), 1e-5, do, None if r is None else r.cuda(), add=None if add is None else (pairs.cuda(), pos.cuda(), k),
                      add_rows=y.cuda())
            _cmp(do, ro, 3e-6 if odt == torch.float32 else 6e-3)
            _cmp(dx, rx if r is None else x, 2e-6)
    dx = x.cuda()
    K.add_rows(dx, y.cuda())
    _cmp(dx, x.double() + y, 1e-6)
    odd = torch.randn(3, 7, generator=g)
    dx = odd.cuda()
    K.add_rows(dx, odd.cuda())
    assert torch.equal(dx.cpu(), 2 * odd)


@pytest.mark.parametrize("odt", DTYPES, ids=IDS)
@pytest.mark.parametrize("heads,dim,temp", [((6, 2), 64, (0.5, 37)), ((4, 4), 128, (0.25, 1)), ((3, 1), 10, (1.5, 12.5)), ((5, 5), 256, None),
                                            ((8, 2), 40, (0.1, 1000)), ((2, 1), 7, (-0.2, 3))])
def test_head_prep_with_values_from_the_keys_and_a_factor_by_position(heads, dim, temp, odt, precise):
    """Both kernels (a block per token, a warp per head), at one token and at hundreds; positions on both sides of every
    multiple of ``every``; the values are the keys in front of their norm."""
    import locus_b200.kernels as K

    H, G = heads
    laid, P = -(-dim // 16) * 16, 16
    g = torch.Generator().manual_seed(dim + H)
    nw = (torch.rand(dim, generator=g) + 0.5, torch.rand(dim, generator=g) + 0.5)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32)
    for T in (1, 45, 330):
        proj = torch.randn(T, -(-(H + G) * dim // 8) * 8, generator=g)
        pos, n_pages = torch.arange(30, 30 + T, dtype=torch.int32), -(-T // P) + 1
        ten = dict(state_slots=i32([0]), seg_q0=i32([0]), seg_qn=i32([T]), positions=pos,
                   slots=torch.randperm(n_pages * P, generator=g)[:T].to(torch.int32))
        kw = dict(offsets=(0, H * dim, H * dim), heads=(H, G, G), dims=(dim,) * 3, laid=(laid,) * 3, n_seg=1, longest_new=T, page_tokens=P,
                  norm="head", eps=1e-5, q_scale=0.7, q_temp=temp)
        rq, rp = torch.zeros(T, H * laid, dtype=torch.float64), torch.zeros(n_pages, 2, G, P, laid, dtype=torch.float64)
        EK.head_prep(proj, q_out=rq, pool=rp, norm_weights=nw, **ten, **kw)
        k0 = proj[0, H * dim:(H + G) * dim].view(G, dim).double()
        s0 = int(ten["slots"][0])
        assert torch.equal(rp[s0 // P, 1, :, s0 % P, :dim], k0)
        for n_rows in (T, 0):
            dq, dp = torch.full((T, H * laid), 7.0, dtype=odt, device=DEV), torch.zeros(*rp.shape, dtype=odt, device=DEV)
            K.head_prep(proj.cuda(), q_out=dq, pool=dp, norm_weights=tuple(t.cuda() for t in nw), n_rows=n_rows,
                        **{k: v.cuda() for k, v in ten.items()}, **kw)
            _cmp(dq, rq, 2e-6 if odt == torch.float32 else 6e-3)
            _cmp(dp, rp, 2e-6 if odt == torch.float32 else 6e-3)
    with pytest.raises(K.KernelError):
        K.head_prep(proj.cuda(), q_out=dq, pool=dp, norm_weights=tuple(t.cuda() for t in nw), n_rows=0,
                    **{k: v.cuda() for k, v in ten.items()}, **{**kw, "q_temp": (0.5, 0.0)})


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("M,tc", [(1, True), (5, True), (14, True), (100, True), (300, True), (40, False)])
def test_the_rectified_gate_on_every_product_kernel(M, tc, dtype, precise, monkeypatch):
    """max(x Wg + b, 0) (x Wu + b') as an epilogue of the row-streaming, the weight-streaming, the tcgen05 and the CUDA-core
    kernel, with biases of both element types and without; grouped rows with a scale behind it."""
    import locus_b200.kernels as K

    if not tc:
        monkeypatch.setattr(K, "USE_TENSOR_CORES", False)
    g = torch.Generator().manual_seed(M)
    for Kd, N in ((64, 300), (2048, 128), (36, 52)):
        x = torch.randn(M, Kd, generator=g).to(dtype)
        wg, wu = ((torch.randn(N, Kd, generator=g) * Kd ** -0.5).to(dtype) for _ in range(2))
        for bias in (None, torch.randn(2 * N, generator=g), torch.randn(2 * N, generator=g).to(torch.bfloat16)):
            ref, out = torch.zeros(M, N, dtype=torch.float64), torch.zeros(M, N, dtype=dtype, device=DEV)
            EK.linear(x, wg, ref, w2=wu, act="reglu", bias=bias)
            K.linear(x.cuda(), wg.cuda(), out, w2=wu.cuda(), act="reglu", bias=None if bias is None else bias.cuda())
            _cmp(out, ref, 5e-6 if dtype == torch.float32 else 8e-3)
            assert float((ref == 0).double().mean()) > 0.2
    with pytest.raises(K.KernelError):
        K.linear(x.cuda(), wg.cuda(), out, act="reglu")
    with pytest.raises(K.KernelError):
        K.linear(x.cuda(), wg.cuda(), out, w2=wu.cuda(), act="reglu", bias=torch.zeros(N, device=DEV))


def test_sigmoid_scores_in_groups_from_logits_far_from_zero(precise):
    """The weights' sum of grouped sigmoid scores: ordinary logits, logits so low that every score is tiny, and a token none of
    whose scores is above zero (its weights are zero, not NaN)."""
    import locus_b200.kernels as K

    g = torch.Generator().manual_seed(3)
    T, E, k = 9, 12, 3
    logits = torch.randn(T, E, generator=g) * 3
    logits[3] -= 30.0
    logits[4] -= 200.0
    kw = dict(n_tokens=T, top_k=k, renorm=True, scale=2.5, score_fn="sigmoid", n_group=4, n_group_used=2)
    ids, wts = torch.zeros(T * k, dtype=torch.int32), torch.zeros(T * k, dtype=torch.float64)
    EK.router_select(logits, E, False, ids, wts, None, **kw)
    di, dw = torch.zeros(T * k, dtype=torch.int32, device=DEV), torch.zeros(T * k, device=DEV)
    K.router_select(logits.cuda(), E, False, di, dw, None, **kw)
    keep = [t for t in range(T) if t != 4]
    assert torch.equal(di.cpu().view(T, k)[keep], ids.view(T, k)[keep])
    _cmp(dw.view(T, k)[keep], wts.view(T, k)[keep], 1e-5)
    assert float(dw.view(T, k)[4].abs().max()) <= 1e-6 and bool(torch.isfinite(dw).all())
    assert math.isclose(float(wts.view(T, k)[3].sum()), 2.5, rel_tol=1e-3)


@pytest.mark.parametrize("window,keep_first,sink", [(0, 0, False), (0, 0, "learned"), (90, 20, True)], ids=["causal", "sink", "window_kept_sink"])
@pytest.mark.parametrize("nh,nkv,hd,dtype", [(6, 2, 128, torch.bfloat16), (8, 2, 64, torch.bfloat16), (2, 2, 128, torch.bfloat16),
                                             (12, 1, 64, torch.bfloat16), (3, 1, 96, torch.bfloat16), (4, 2, 64, torch.float32),
                                             (2, 1, 16, torch.float32)],
                         ids=["6on2_128", "8on2_64", "2on2_128", "12on1_64", "3on1_96", "f32_4on2_64", "f32_2on1_16"])
def test_every_attention_kernel_with_a_distance_bias(nh, nkv, hd, dtype, window, keep_first, sink):
    """Portions (tcgen05 whole and with its keys cut into ranges, mma.sync in both forms, CUDA cores) and single tokens
    (streaming per head and per group of query heads in both variants, fixed ranges) against the twin in float64, with slopes
    from steep to flat, also beside a sink (where a bias by key alone would be another function) and within a window that
    keeps first tokens."""
    import locus_b200.kernels as K
    from test_mekizen_gpu import _close, _paged_attention_case

    P = 64
    tol = 1.5e-2 if dtype == torch.bfloat16 else 2e-5
    slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / nh) for h in range(nh)], dtype=torch.float32)
    kw = dict(n_heads=nh, n_kv_heads=nkv, head_dim=hd, page_tokens=P, window=window, scale=0.11, keep_first=keep_first)
    lsink = torch.linspace(-1.0, 2.0, nh) if sink == "learned" else sink
    cpu = dict(kw, slopes=slopes, sink=lsink)
    kw = dict(kw, slopes=slopes.cuda(), sink=lsink.cuda() if sink == "learned" else sink)

    def twin(pool, q, meta, T, items):
        ref = torch.zeros(T, nh * hd, dtype=torch.float64)
        EK.PRECISE = True
        try:
            EK.attn_chunk(q, pool, ref, items=items, n_items=len(items), **meta, **cpu)
        finally:
            EK.PRECISE = False
        return ref

    segs = [(0, 5), (33, 17), (100, 2), (64, 64), (190, 130), (331, 4), (600, 70)]
    pool, q, meta, T = _paged_attention_case(dtype, nh, nkv, hd, P, segs, window, keep_first, seed=nh + hd)
    items64 = torch.tensor([(s, o) for s, (c, n) in enumerate(segs) for o in range(0, n, K.MMA_QUERY_TILE)], dtype=torch.int32)
    items16 = torch.tensor([(s, o) for s, (c, n) in enumerate(segs) for o in range(0, n, 16)], dtype=torch.int32)
    ref = twin(pool, q, meta, T, items16)
    dev, dq, dpool = {k: v.cuda() for k, v in meta.items()}, q.cuda(), pool.cuda()

    def fresh():
        return torch.full((T, nh * hd), float("nan"), dtype=dtype, device="cuda")

    def scratch(n):
        return torch.full((n,), float("nan"), device="cuda")

    if K.attn_chunk_tc_takes(dq, hd, P, T, 2048):
        for n_splits in (1, 2, 7):
            extra = dict(n_splits=n_splits, part_o=scratch(T * nh * n_splits * hd), part_ml=scratch(T * nh * n_splits * 2)) if n_splits > 1 else {}
            out = fresh()
            K.attn_chunk_tc(dq, dpool, out, items=items64.cuda(), n_items=len(items64), **extra, **dev, **kw)
            assert K.attn_tc_error() == 0 and _close(out, ref, tol), f"attn_chunk_tc in {n_splits} key ranges"
    if K.attn_chunk_mma_takes(dq, hd):
        out = fresh()
        K.attn_chunk_mma(dq, dpool, out, items=items64.cuda(), n_items=len(items64), **dev, **kw)
        assert _close(out, ref, tol), "attn_chunk_mma"
        n_o, n_ml = K.attn_chunk_mma_scratch(hd)
        some, lo = items64[-2:], int(meta["seg_q0"][-1])     # (the last request's tiles, its keys cut into ranges)
        out = fresh()
        K.attn_chunk_mma(dq, dpool, out, items=some.cuda(), n_items=len(some), n_splits=4, part_o=scratch(n_o), part_ml=scratch(n_ml), **dev, **kw)
        assert _close(out[lo:], ref[lo:], tol), "attn_chunk_mma in 4 key ranges"
    out = fresh()
    K.attn_chunk(dq, dpool, out, items=items16.cuda(), n_items=len(items16), **dev, **kw)
    assert _close(out, ref, tol), "attn_chunk"
    with pytest.raises(K.KernelError):     # a slope per query head
        K.attn_chunk(dq, dpool, out, items=items16.cuda(), n_items=len(items16), **dev, **{**kw, "slopes": slopes[:-1].cuda()})

    # single tokens
    ctxs = [0, 1, 31, 32, 47, 99, 100, 127, 128, 255, 333, 666, 700, 1023, 1100]
    pool, q, meta, T = _paged_attention_case(dtype, nh, nkv, hd, P, [(c, 1) for c in ctxs], window, keep_first, seed=nh + hd + 1)
    items = torch.arange(len(ctxs), dtype=torch.int32)
    ref = twin(pool, q, meta, T, torch.stack([items, torch.zeros_like(items)], 1))
    dev, dq, dpool = {k: v.cuda() for k, v in meta.items()}, q.cuda(), pool.cuda()
    max_splits = max(ctxs) // K.DECODE_SPLIT + 1
    units = K.decode_units(len(ctxs), nh, hd, dtype, max_splits, "cuda", page_tokens=P, n_kv_heads=nkv, fixed_ranges=keep_first > 0)
    part_o, part_ml = scratch(units * hd), scratch(units * 2)
    counters = torch.zeros(len(ctxs) * nh, dtype=torch.int32, device="cuda")
    use_gqa, ran_gqa = K.USE_GQA_DECODE, False
    try:
        for gqa, deep in [(g, d) for g in (True, False) for d in (None, True, False)]:
            if gqa and not K.attn_decode_gqa_takes(dtype, nh, nkv, hd, P, len(ctxs)):
                continue
            ran_gqa = ran_gqa or gqa
            K.USE_GQA_DECODE = gqa
            K.attn_decode_variant(deep)
            if dtype == torch.bfloat16:
                K.attn_decode_gqa_variant(deep)
            for lo, hi in ((0, len(ctxs)), (8, 9), (len(ctxs) - 1, len(ctxs))):
                out = fresh()
                K.attn_decode(dq, dpool, out, items=items[lo:hi].cuda(), n_items=hi - lo, part_o=part_o, part_ml=part_ml, counters=counters,
                              max_splits=max_splits, **dev, **kw)
                assert K.attn_error() == 0 and (not gqa or K.attn_gqa_error() == 0)
                assert _close(out[lo:hi], ref[lo:hi], tol), f"{'grouped' if gqa else 'per head'}, variant {deep}, requests {lo} to {hi}"
                assert int(counters.abs().sum()) == 0
    finally:
        K.USE_GQA_DECODE = use_gqa
        K.attn_decode_variant(None)
        if dtype == torch.bfloat16:
            K.attn_decode_gqa_variant(None)
    if dtype == torch.bfloat16 and nh != nkv and hd in (64, 128) and len(ctxs) * nkv >= K.GQA_MIN_UNITS:
        assert ran_gqa, "the grouped decode kernel did not take this shape"


@pytest.mark.parametrize("kv_rank,heads", [(96, 6), (160, 3), (192, 16), (224, 1), (320, 5), (384, 4), (448, 20), (512, 16), (64, 4)])
def test_latent_attention_without_a_rotated_part(kv_rank, heads):
    """Every rank the tensor-core kernel has an instance for, over rows without a rotated part: whole and with the keys cut
    into ranges, against the CUDA-core kernel and the twin."""
    import locus_b200.kernels as K

    g = torch.Generator().manual_seed(kv_rank)
    P, segs = 16, [(0, 37), (70, 1), (5, 2), (200, 19)]
    need = [-(-(c + n) // P) for c, n in segs]
    pool = torch.randn(sum(need), 1, 1, P, kv_rank, generator=g).to(torch.bfloat16)
    table = torch.full((len(segs), max(need)), -1, dtype=torch.int32)
    at = 0
    for s, n in enumerate(need):
        table[s, :n] = torch.arange(at, at + n)
        at += n
    T = sum(n for _, n in segs)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32)
    q0 = [sum(n for _, n in segs[:s]) for s in range(len(segs))]
    q_abs, q_rot = torch.randn(heads * T, kv_rank, generator=g).to(torch.bfloat16), torch.zeros(T, 0, dtype=torch.bfloat16)
    ten = dict(seg_q0=i32(q0), seg_qn=i32([n for _, n in segs]), seg_ctx=i32([c for c, _ in segs]), block_table=table)
    kw = dict(n_tokens=T, n_heads=heads, kv_rank=kv_rank, rot_dim=0, page_tokens=P, window=0, scale=0.08)
    tiles = lambda n_q: i32([[s, o] for s, (c, n) in enumerate(segs) for o in range(0, n, n_q)])
    items = tiles(K.LATENT_QUERY_TILE)
    want = torch.zeros(heads * T, kv_rank, dtype=torch.float64)
    EK.PRECISE = True
    try:
        EK.latent_attn(q_abs, q_rot, pool, None, want, items=items, n_items=len(items), **ten, **kw)
    finally:
        EK.PRECISE = False
    dev = {k: v.cuda() for k, v in ten.items()}
    out = torch.zeros(heads * T, kv_rank, dtype=torch.bfloat16, device=DEV)
    K.latent_attn(q_abs.cuda(), q_rot.cuda(), pool.cuda(), None, out, items=items.cuda(), n_items=len(items), **dev, **kw)
    _cmp(out, want, 1e-2)
    assert K.latent_attn_mma_takes(torch.bfloat16, kv_rank, 0)
    shift = K.latent_mma_head_shift(heads)
    items = tiles(64 >> shift)
    units = len(items) * (-(-heads // (1 << shift))) * 5
    part_o, part_ml = torch.full((units * 64 * kv_rank,), float("nan"), device=DEV), torch.full((units * 128,), float("nan"), device=DEV)
    for n_splits in (1, 3, 5):
        out = torch.full((heads * T, kv_rank), float("nan"), dtype=torch.bfloat16, device=DEV)
        K.latent_attn_mma(q_abs.cuda(), q_rot.cuda(), pool.cuda(), None, out, items=items.cuda(), n_items=len(items), head_shift=shift,
                          n_splits=n_splits, part_o=part_o, part_ml=part_ml, **dev, **kw)
        _cmp(out, want, 1.5e-2)


@pytest.mark.parametrize("kv_rank,rot,heads,window,sink", [(512, 0, 16, 0, False), (512, 64, 20, 0, True), (256, 0, 4, 0, False), (256, 64, 16, 90, True),
                                                            (384, 32, 33, 0, False), (128, 0, 1, 64, False), (128, 64, 8, 1, True), (512, 32, 128, 0, False)])
def test_latent_decode_against_its_twin(kv_rank, rot, heads, window, sink):
    """Single tokens on both sides of page, tile and window edges, in one range, the engine's choice and many ranges (more
    than some requests have tiles); rows that are no single tokens stay as they are; unwritten cache is NaN."""
    import locus_b200.kernels as K

    g = torch.Generator().manual_seed(kv_rank + heads)
    P, R = 32, kv_rank + rot
    ctxs = [0, 5, 31, 32, 63, 64, 65, 127, 200, 700, 1023]
    segs = [(3, 4)] + [(c, 1) for c in ctxs]
    need = [-(-(c + n) // P) for c, n in segs]
    pool = (torch.randn(sum(need) + 1, 1, 1, P, R, generator=g) * 0.5).to(torch.bfloat16)
    table, perm, at = torch.full((len(segs), max(need)), -1, dtype=torch.int32), torch.randperm(sum(need), generator=g), 0
    for s, (c, n) in enumerate(segs):
        table[s, :need[s]] = perm[at:at + need[s]].to(torch.int32)
        at += need[s]
        if (c + n) % P:
            pool[int(table[s, need[s] - 1]), 0, 0, (c + n) % P:] = float("nan")
        if window:
            gone = max(0, c - window + 1) // P
            for pg in range(gone):
                pool[int(table[s, pg])] = float("nan")
            table[s, :gone] = -1
    T = sum(n for _, n in segs)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32)
    q_abs, q_rot = torch.randn(heads * T, kv_rank, generator=g).to(torch.bfloat16), torch.randn(T, heads * rot, generator=g).to(torch.bfloat16)
    sk = torch.linspace(-2.0, 8.0, heads) if sink else None
    ten = dict(seg_q0=i32([sum(n for _, n in segs[:s]) for s in range(len(segs))]), seg_ctx=i32([c for c, _ in segs]), block_table=table)
    kw = dict(n_tokens=T, n_heads=heads, kv_rank=kv_rank, rot_dim=rot, page_tokens=P, window=window, scale=0.1)
    items = i32(list(range(1, len(segs))))
    want = torch.zeros(heads * T, kv_rank, dtype=torch.float64)
    EK.PRECISE = True
    try:
        EK.latent_decode(q_abs, q_rot, pool, sk, want, items=items, n_items=len(items), **ten, **kw)
    finally:
        EK.PRECISE = False
    dev = {k: v.cuda() for k, v in ten.items()}
    want = want.view(heads, T, kv_rank)
    for lo, hi in ((0, len(items)), (len(items) - 1, len(items))):
        for n_ranges in (1, K.latent_decode_ranges(hi - lo, heads, 1024), 3, 64):
            units = (hi - lo) * -(-heads // 16) * n_ranges * 16
            out = torch.full((heads * T, kv_rank), 7.0, dtype=torch.bfloat16, device=DEV)
            K.latent_decode(q_abs.cuda(), q_rot.cuda(), pool.cuda(), None if sk is None else sk.cuda(), out, items=items[lo:hi].cuda(), n_items=hi - lo,
                            n_ranges=n_ranges, part_o=torch.full((units * kv_rank,), float("nan"), device=DEV),
                            part_ml=torch.full((2 * units,), float("nan"), device=DEV), **dev, **kw)
            out = out.view(heads, T, kv_rank)
            _cmp(out[:, 4 + lo:4 + hi], want[:, 4 + lo:4 + hi], 1.5e-2)
            assert bool((out[:, :4 + lo] == 7).all())
    n_o, n_ml = K.latent_decode_scratch(kv_rank)
    for b in (1, 3, 8, 40, 148, 1000):
        n = K.latent_decode_ranges(b, heads, 100000)
        assert n == 1 or b * -(-heads // 16) * n * 16 * kv_rank <= n_o


def test_key_ranges_fit_their_scratch_beside_many_other_rows():
    """A short portion behind a long context in a step with many single tokens: the ranges' partial results of all rows fit."""
    import locus_b200.kernels as K

    n_o, n_ml = K.attn_chunk_tc_scratch()
    for heads in (4, 16, 28):
        for rows in (128, 200, 256, 700):
            n = K.attn_chunk_tc_splits(2, heads, 30000, rows)
            assert n >= 1 and (n == 1 or rows * heads * n * K.TC_ATTN_HEAD_DIM <= n_o and rows * heads * n * 2 <= n_ml)
    assert K.attn_chunk_tc_splits(2, 4, 30000, 128) == K.attn_chunk_tc_splits(2, 4, 30000) > 8


@pytest.mark.parametrize("nh,nkv,how", [(4, 4, "plain"), (6, 2, "slopes"), (4, 4, "sink"), (3, 3, "window")])
def test_the_tcgen05_attention_over_plain_rows(nh, nkv, how):
    """The rows form (whole and with the keys cut into ranges) against the twin and against the paged form over the same keys
    and values; the rows come from pages in any order through ``latent_gather``; rows between and behind the segments' own are
    NaN; a page that has gone back leaves zeros."""
    import locus_b200.kernels as K

    g = torch.Generator().manual_seed(nh)
    P, hd, segs = 64, 128, [(0, 5), (100, 130), (3, 1), (331, 257), (64, 64)]
    long = [1, 3, 4]
    need = [-(-(c + n) // P) for c, n in segs]
    W = nkv * hd
    src = torch.randn(sum(need) + 1, 1, 1, P, 2 * W + 8, generator=g).to(torch.bfloat16)
    perm = torch.randperm(sum(need) + 1, generator=g).to(torch.int32)
    table, at = torch.full((len(segs), max(need) + 1), -1, dtype=torch.int32), 0
    for s, n in enumerate(need):
        table[s, :n] = perm[at:at + n]
        at += n
    window = 90 if how == "window" else 0
    row0, rows = torch.full((len(segs),), -1, dtype=torch.int32), 3
    for s in long:
        row0[s] = rows
        rows += sum(segs[s]) + 2
    if window:
        table[3, :3] = -1
    i32 = lambda v: torch.tensor(v, dtype=torch.int32)
    T = sum(n for _, n in segs)
    meta = dict(seg_q0=i32([sum(n for _, n in segs[:s]) for s in range(len(segs))]), seg_qn=i32([n for _, n in segs]), seg_ctx=i32([c for c, _ in segs]))
    dev = {k: v.cuda() for k, v in meta.items()}
    kv = torch.full((rows, 2 * W), float("nan"), dtype=torch.bfloat16, device=DEV)
    kw = dict(segs=i32(long), n_segs=3, row0=row0, seg_qn=meta["seg_qn"], seg_ctx=meta["seg_ctx"], block_table=table)
    K.latent_gather(src.cuda(), kv, page_tokens=P, longest=331 + 257, **{k: v.cuda() if torch.is_tensor(v) else v for k, v in kw.items()})
    want = torch.full((rows, 2 * W), float("nan"), dtype=torch.bfloat16)
    EK.latent_gather(src, want, page_tokens=P, longest=331 + 257, **kw)
    assert torch.equal(kv.cpu().nan_to_num(7e4), want.nan_to_num(7e4))
    items = i32([[s, o] for s in long for o in range(0, segs[s][1], K.MMA_QUERY_TILE)])
    q = torch.randn(T, nh * hd, generator=g).to(torch.bfloat16)
    opts = dict(n_heads=nh, n_kv_heads=nkv, head_dim=hd, scale=0.09)
    slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / nh) for h in range(nh)]) if how == "slopes" else None
    sink = torch.linspace(-1.0, 2.0, nh) if how == "sink" else False
    used = torch.cat([torch.arange(int(dev["seg_q0"][s]), int(dev["seg_q0"][s]) + segs[s][1]) for s in long])
    ref = torch.zeros(T, nh * hd, dtype=torch.float64)
    if not window:
        EK.PRECISE = True
        try:
            EK.attn_chunk_tc_rows(q, want[:, :W], want[:, W:], ref, kv_row0=row0, items=items, n_items=len(items), window=0, slopes=slopes, sink=sink,
                                  **meta, **opts)
        finally:
            EK.PRECISE = False
    else:
        pages = torch.zeros(sum(need) + 1, 2, nkv, P, hd, dtype=torch.bfloat16)
        pages[:, 0] = src[:, 0, 0, :, :W].view(-1, P, nkv, hd).transpose(1, 2)
        pages[:, 1] = src[:, 0, 0, :, W:2 * W].view(-1, P, nkv, hd).transpose(1, 2)
        out = torch.zeros(T, nh * hd, dtype=torch.bfloat16, device=DEV)
        K.attn_chunk_tc(q.cuda(), pages.cuda(), out, items=items.cuda(), n_items=len(items), page_tokens=P, window=window, block_table=table.cuda(), **dev, **opts)
        ref = out.double().cpu()
    for n_splits in (1, 2, 5):
        extra = {}
        if n_splits > 1:
            extra = dict(n_splits=n_splits, part_o=torch.full((T * nh * n_splits * hd,), float("nan"), device=DEV),
                         part_ml=torch.full((T * nh * n_splits * 2,), float("nan"), device=DEV))
        out = torch.full((T, nh * hd), float("nan"), dtype=torch.bfloat16, device=DEV)
        K.attn_chunk_tc_rows(q.cuda(), kv[:, :W], kv[:, W:], out, kv_row0=row0.cuda(), items=items.cuda(), n_items=len(items), window=window,
                             slopes=None if slopes is None else slopes.cuda(), sink=sink.cuda() if torch.is_tensor(sink) else sink,
                             **extra, **dev, **opts)
        assert K.attn_tc_error() == 0
        _cmp(out[used], ref[used], 1.5e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_generation_through_the_engine_and_the_command_line(dtype, cases):
    """Greedy generation with portions and requests side by side: every token is the plain implementation's best one or within
    rounding of it; the command line says the same tokens in float32."""
    from locus_b200.engine.engine import Engine

    case = cases("mix", torch.float32 if dtype == "float32" else torch.bfloat16)
    prompts = [case.tokens[r] for r in ("r2", "r5", "r3")]
    eng = Engine.from_model_dir(case.dir, dtype=dtype, ctx=512, page_tokens=16, max_batch_tokens=32, chunk=16, max_running=2)
    out = eng.generate(prompts, max_new_tokens=8)
    for p, o in zip(prompts, out):
        ref = plain.forward(case.cfg, case.weights, p + o)
        for i, tok in enumerate(o):
            row = ref[len(p) + i - 1]
            assert float(row.max() - row[tok]) <= (1e-4 if dtype == "float32" else 1e-1) * float(ref.abs().max()), (i, tok)
    assert eng.cache.free_pages() == eng.cache.total_pages()
    if dtype != "float32":
        return
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "locus-run"), case.dir, ",".join(map(str, prompts[0])), "8",
                        "--dtype", "float32", "--page-tokens", "16", "--ctx", "512"], capture_output=True, text=True, timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    said = [int(x) for x in r.stdout.replace(",", " ").split() if x.lstrip("-").isdigit()]
    assert said[-8:] == list(out[0]), (said[-8:], out[0])
    archs = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "locus-run"), "--archs"], capture_output=True, text=True)
    assert "Megovik" in archs.stdout


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_as_a_program(dtype, cases, tmp_path):
    import numpy as np

    td = torch.float32 if dtype == "float32" else torch.bfloat16
    case = cases("wide", td)
    out = tmp_path / "out"
    a, b = case.tokens["r1"], case.tokens["r0"][:19]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:20], "want": [0, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[20:22], "want": [1]}, {"id": "b", "tokens": b, "want": [18]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[22:23], "want": [0]}], "end": ["a"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", case.dir, "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True,
                       text=True, timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    ra, rb = case.ref("r1")[0], case.ref("r0")[0]
    want = {0: ra[[0, 19]], 1: torch.stack([ra[21], rb[18]]), 2: ra[[22]]}
    for s, ref in want.items():
        got = torch.from_numpy(np.fromfile(out / f"{s}.f32", dtype="<f4").reshape(ref.shape[0], -1)).double()
        err, _ = errors(got, ref)
        assert float(err.max()) <= TOL[td][0] * 3, (s, float(err.max()))
