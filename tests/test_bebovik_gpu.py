"""The Bebovik design on the GPU against the plain implementation (float64), in float32 and in bfloat16: whole prompts,
decoding token by token, portions down to two tokens, mixed batches with pages that are used again; configurations drawn at
random on pages of 64; a key that stands out just inside and just outside a chunk, in prompts and while decoding; long
decoding through CUDA graphs; heads of 128 in long portions; the new kernels and the new forms of the others alone against
their plain twins; greedy generation through the engine's entry point and the command line; trace replay as a program.
Pages are filled with NaN when they are made and when they go back."""
import functools
import json
import os
import subprocess
import sys

import pytest
import torch

import emulated_kernels as EK
import plain_bebovik as plain
from bebovik_cases import Case, attention, compare, errors, layer, make_runner, model, random_config, run_steps, schedules, sharpen

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEV = "cuda:0"

# max and mean |error| of the logits (their mean over the vocabulary taken off) relative to the largest |logit|
TOL = {torch.float32: (5e-5, 1e-5), torch.bfloat16: (4e-2, 6e-3)}
DTYPES = [torch.float32, torch.bfloat16]
IDS = ["f32", "bf16"]
LENGTHS = {"mix": (1, 2, 37, 70, 45, 19, 130), "odd": (3, 90, 33, 16, 75), "wide": (150, 40, 260), "attention_only": (50, 23),
           "mlp_only": (20, 5)}


def _milder(dtype):
    """The factors on the projections nearer to 1 in bfloat16: with all of them a few positions amplify the rounding of the
    activations beyond what tells a fault from it (the kernels' plain twins with bfloat16 buffers are off there by as much)."""
    return sharpen if dtype == torch.float32 else functools.partial(sharpen, strength=0.4)


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            made[name] = Case(name, tmp_path_factory.mktemp("bebovik"), torch.bfloat16, requests=LENGTHS[name])
        return made[name]

    return get


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("name", list(LENGTHS))
def test_every_schedule_agrees_with_plain(name, dtype, cases):
    case = cases(name)
    runner, cache = make_runner(case, dtype, DEV, page_tokens=16, n_pages=40, max_tokens=320)
    for sched_name, steps in schedules(case).items():
        got, _ = run_steps(runner, cache, case, steps)
        compare(case, got, *TOL[dtype])
        assert cache.free_pages() == cache.total_pages() and cache.state_slots.free == cache.state_slots.total, sched_name


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("seed", list(range(6)))
def test_drawn_configurations_on_pages_of_64(seed, dtype, tmp_path_factory):
    """Configurations drawn at random: portions of changing size and mixed batches of four live requests on pages of 64
    whose pool only holds them when pages are used again."""
    case = Case(f"drawn{seed}", tmp_path_factory.mktemp("drawn"), torch.bfloat16, raw=random_config(500 + seed),
                requests=(230, 1, 150, 40, 97, 180), seed=seed, tweak=_milder(dtype))
    runner, cache = make_runner(case, dtype, DEV, page_tokens=64, n_pages=14, max_tokens=256, max_seq=512)
    sch = schedules(case)
    for name in ("mixed", "chunked"):
        got, _ = run_steps(runner, cache, case, sch[name])
        # (up to six sharpened layers deep)
        compare(case, got, *((2e-4, 4e-5) if dtype == torch.float32 else TOL[dtype]))
        assert cache.free_pages() == cache.total_pages()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("page_tokens", [8, 64])
def test_other_page_sizes_and_the_cuda_core_products(page_tokens, dtype, cases, monkeypatch):
    import locus_b200.kernels as K

    case = cases("mix")
    if page_tokens == 8:
        monkeypatch.setattr(K, "USE_TENSOR_CORES", False)   # bfloat16 on the CUDA-core products and attention
    runner, cache = make_runner(case, dtype, DEV, page_tokens=page_tokens, n_pages=24 if page_tokens == 64 else 90,
                                max_tokens=320, max_seq=1024)
    sch = schedules(case)
    for steps in (sch["mixed"], sch["chunked"]):
        got, _ = run_steps(runner, cache, case, steps)
        compare(case, got, *TOL[dtype])


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_heads_of_128_in_long_portions_on_pages_of_64(dtype, tmp_path_factory):
    """Heads of 128 with values of 96 and four query heads on every key/value head, portions of several hundred tokens that
    span several chunks (the kernels that long portions of that head size take), chunks longer than a portion."""
    raw = model(256, 301, [layer(attention(8, 2, 128, 96, chunk=200, rot=64, base=5e5, scaling=(6.0, 1.0, 5.0, 300), scale=0.1), 192, 1.5),
                           layer(attention(4, 2, 128, 128, chunk=512, rot=128, scale=0.08), 0),
                           layer(attention(4, 4, 64, 64, scale=0.15), 128, 2.0)], emb=6.0, logit_scale=2.0, cap=12.0)
    case = Case("big", tmp_path_factory.mktemp("big"), torch.bfloat16, raw=raw, requests=(700, 90), tweak=_milder(dtype))
    runner, cache = make_runner(case, dtype, DEV, page_tokens=64, n_pages=20, max_tokens=640, max_seq=1024)
    for steps in ([[("r0", 300), ("r1", 40)], [("r0", 399), ("r1", 1)], [("r0", 1), ("r1", 49)]], [[("r0", 600), ("r1", 2)], [("r0", 100), ("r1", 88)]]):
        got, _ = run_steps(runner, cache, case, steps)
        compare(case, got, *TOL[dtype])


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_long_decoding_through_graphs(dtype, tmp_path):
    """Two requests decoded side by side for 200 tokens through CUDA graphs, past several pages and chunks: the replayed
    steps against the same steps launched kernel by kernel and against the plain implementation."""
    from locus_b200.engine.step import StepEntry

    case = Case("mix", tmp_path, torch.bfloat16, requests=(230, 215))
    rows = {}
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
    ref = torch.stack([case.ref("r0")[30:230], case.ref("r1")[15:215]], 1)
    for other in (rows[False], ref):
        err, mean = errors(rows[True].reshape(400, -1), other.reshape(400, -1))
        assert float(err.max()) <= TOL[dtype][0] and mean <= TOL[dtype][1], (float(err.max()), mean)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("chunk,n", [(40, 96), (300, 420)])
def test_keys_just_inside_and_just_outside_a_chunk(chunk, n, dtype, tmp_path_factory):
    """A key that stands out among up to hundreds of others: at the sequence's first position, a chunk's last and first, at
    page borders; seen (or not) by queries in whole prompts, in portions that start at the edges, and decoded one by one."""
    from test_bebovik_host import beacon_case, beacon_reach

    places = (0, chunk - 1, chunk, (chunk // 16 + 1) * 16 - 1, (chunk // 16 + 1) * 16)
    case = beacon_case(tmp_path_factory.mktemp("beacon"), chunk, n, places, torch.bfloat16)
    for i, at in enumerate(places):
        beacon_reach(case, f"r{i}", at, chunk)
    runner, cache = make_runner(case, dtype, DEV, page_tokens=16, n_pages=30, max_tokens=448, slots=1)
    for i in range(len(places)):
        r = f"r{i}"
        tail = n - chunk - 3
        for steps in ([[(r, n)]], [[(r, chunk - 2)]] + [[(r, 1)]] * 5 + [[(r, tail - 20)]] + [[(r, 1)]] * 20,
                      [[(r, 2)], [(r, chunk - 2)], [(r, 2)], [(r, tail - 1)], [(r, 2)]]):
            got, _ = run_steps(runner, cache, case, steps)
            compare(case, got, *TOL[dtype])


# ---------------------------------------------------------------------------
# the kernels alone against their plain twins (float64)


def _cmp(a, b, tol):
    a, b = a.double().cpu(), b.double().cpu()
    assert bool(torch.isfinite(a).all())
    assert float((a - b).abs().max()) <= tol * max(1.0, float(b.abs().max())), float((a - b).abs().max())


@pytest.fixture
def precise(monkeypatch):
    monkeypatch.setattr(EK, "PRECISE", True)


def _norm(H, g, dt):
    return (torch.rand((), generator=g) + 0.5).to(dt), torch.randn(H, generator=g).to(dt), torch.randn(H, generator=g).to(dt)


def _cuda(n):
    return tuple(t.cuda() for t in n)


@pytest.mark.parametrize("wdt", DTYPES, ids=["w32", "w16"])
@pytest.mark.parametrize("odt", DTYPES, ids=IDS)
@pytest.mark.parametrize("H,T", [(256, 1), (50, 7), (2048, 300), (1028, 33), (8, 2)])
def test_dyt_against_its_twin(H, T, odt, wdt, precise):
    """The norm alone (also in place), the addition of a normed and scaled row in front of it, the addition alone, and over
    gathered rows (which leave the stream as it was); inputs from where the tanh is linear to where it is flat."""
    import locus_b200.kernels as K

    g = torch.Generator().manual_seed(H + T)
    tol = 2e-6 if odt == torch.float32 else 5e-3
    x = torch.randn(T, H, generator=g) * torch.logspace(-4, 1.3, H)[torch.randperm(H, generator=g)]
    y = torch.randn(T, H, generator=g) * 0.7
    inner, outer = _norm(H, g, wdt), _norm(H, g, wdt)
    rows = torch.randint(0, T, (5,), generator=g, dtype=torch.int32)
    for scale in (None, torch.randn(H, generator=g).to(wdt)):
        rx, ro = x.clone().double(), torch.zeros(T, H, dtype=torch.float64)
        EK.dyt(rx, outer, ro, add=(y, inner, scale))
        dx, do = x.cuda(), torch.zeros(T, H, dtype=odt, device=DEV)
        dscale = None if scale is None else scale.cuda()
        K.dyt(dx, _cuda(outer), do, add=(y.cuda(), _cuda(inner), dscale))
        _cmp(dx, rx, 2e-6)
        _cmp(do, ro, tol)
        only = x.cuda()
        K.dyt(only, add=(y.cuda(), _cuda(inner), dscale))
        _cmp(only, rx, 2e-6)
        kept, ro = x.cuda(), torch.zeros(5, H, dtype=torch.float64)
        EK.dyt(x.double(), outer, ro, rows, add=(y, inner, scale))
        do = torch.zeros(5, H, dtype=odt, device=DEV)
        K.dyt(kept, _cuda(outer), do, rows.cuda(), add=(y.cuda(), _cuda(inner), dscale))
        _cmp(do, ro, tol)
        assert torch.equal(kept.cpu(), x)
    ro = torch.zeros(T, H, dtype=torch.float64)
    EK.dyt(x.double(), outer, ro)
    do, place = torch.zeros(T, H, dtype=odt, device=DEV), x.cuda()
    K.dyt(x.cuda(), _cuda(outer), do)
    K.dyt(place, _cuda(outer), place)
    _cmp(do, ro, tol)
    _cmp(place, ro, 2e-6)
    with pytest.raises(K.KernelError):
        K.dyt(place, _cuda(outer), place, add=(y.cuda(), _cuda(inner), None))


def test_the_embeddings_norm_against_its_twin(precise):
    import locus_b200.kernels as K

    g = torch.Generator().manual_seed(6)
    for dt in DTYPES:
        for H in (50, 640):
            table, toks, norm = torch.randn(31, H, generator=g).to(dt), torch.randint(0, 31, (19,), generator=g, dtype=torch.int32), _norm(H, g, dt)
            ref, out = torch.zeros(19, H, dtype=torch.float64), torch.zeros(19, H, device=DEV)
            EK.embed_rows(toks, table, ref, scale=3.5, dyt_norm=norm)
            K.embed_rows(toks.cuda(), table.cuda(), out, scale=3.5, dyt_norm=_cuda(norm))
            _cmp(out, ref, 2e-6)


@pytest.mark.parametrize("odt", DTYPES, ids=IDS)
@pytest.mark.parametrize("heads,dims,rot,adjacent,norm", [
    ((6, 2, 2), (64, 64, 64), 24, True, "head"), ((4, 1, 1), (40, 40, 24), 20, True, "head"), ((3, 3, 3), (256, 256, 200), 100, False, "head"),
    ((5, 5, 5), (12, 12, 8), 6, True, "unit"), ((4, 2, 2), (128, 128, 128), 128, False, "rms"), ((2, 2, 2), (24, 24, 32), 24, False, None),
    ((16, 4, 4), (128, 128, 128), 128, True, "head"), ((3, 1, 1), (10, 10, 7), 6, True, "head"), ((2, 1, 1), (200, 200, 16), 0, True, "head")])
def test_head_prep_with_weighted_norms_and_adjacent_pairs(heads, dims, rot, adjacent, norm, odt, precise):
    """Both kernels (a block per token, a warp per head; sizes that are no multiple of 4 have the second only), with and
    without the write of keys and values, at one token and at hundreds; positions in the tens of thousands."""
    import locus_b200.kernels as K

    laid, P = -(-max(dims) // 16) * 16, 16
    g = torch.Generator().manual_seed(sum(dims) + rot)
    widths = [h * d for h, d in zip(heads, dims)]
    offs = (0, widths[0], widths[0] + widths[1])
    nw = (torch.rand(dims[0], generator=g) + 0.5, torch.rand(dims[1], generator=g) + 0.5) if norm == "head" else None
    inv = (1e4 ** (-torch.arange(0, rot, 2) / rot)).float() if rot else None
    i32 = lambda v: torch.tensor(v, dtype=torch.int32)
    for T in (1, 45, 330):
        proj = torch.randn(T, -(-sum(widths) // 8) * 8, generator=g)
        pos, n_pages = torch.arange(40000, 40000 + T, dtype=torch.int32), -(-T // P) + 1
        ten = dict(state_slots=i32([0]), seg_q0=i32([0]), seg_qn=i32([T]), positions=pos,
                   slots=torch.randperm(n_pages * P, generator=g)[:T].to(torch.int32), inv_freq=inv)
        kw = dict(offsets=offs, heads=heads, dims=dims, laid=(laid,) * 3, n_seg=1, longest_new=T, page_tokens=P, rot=rot, norm=norm,
                  eps=1e-5, interleaved=adjacent, q_scale=0.7)
        for write in (True, False):
            rq, rp = torch.zeros(T, heads[0] * laid, dtype=torch.float64), torch.zeros(n_pages, 2, heads[1], P, laid, dtype=torch.float64)
            EK.head_prep(proj, q_out=rq, pool=rp, norm_weights=nw, write_kv=write, **ten, **kw)
            for n_rows in (T, 0):
                dq, dp = torch.full((T, heads[0] * laid), 7.0, dtype=odt, device=DEV), torch.zeros(*rp.shape, dtype=odt, device=DEV)
                K.head_prep(proj.cuda(), q_out=dq, pool=dp, norm_weights=None if nw is None else _cuda(nw), write_kv=write, n_rows=n_rows,
                            **{k: None if v is None else v.cuda() for k, v in ten.items()}, **kw)
                # (float32 angles: position x frequency is rounded once, the twin's float32 angle in the same way)
                _cmp(dq, rq, 3e-6 if odt == torch.float32 else 6e-3)
                _cmp(dp, rp, 3e-6 if odt == torch.float32 else 6e-3)


@pytest.mark.parametrize("odt", DTYPES, ids=IDS)
def test_gate_rows_in_pieces_of_eight_and_in_single_elements(odt, precise):
    import locus_b200.kernels as K

    g = torch.Generator().manual_seed(8)
    for heads, dim, laid, off, T in ((16, 128, 128, 64, 70), (3, 24, 32, 8, 9), (3, 20, 32, 8, 9), (2, 7, 16, 3, 5), (5, 64, 80, 4, 1)):
        o, proj = torch.randn(T, heads * laid, generator=g).to(odt), torch.randn(T, -(-(off + heads * dim) // 4) * 4, generator=g) * 3
        ref, out = o.double(), o.cuda()
        EK.gate_rows(ref, proj, off, n_heads=heads, dim=dim, laid=laid)
        K.gate_rows(out, proj.cuda(), off, n_heads=heads, dim=dim, laid=laid)
        _cmp(out, ref, 1e-6 if odt == torch.float32 else 8e-3)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("M,tc", [(1, True), (5, True), (14, True), (100, True), (300, True), (40, False)])
def test_the_softcap_on_every_product_kernel(M, tc, dtype, precise, monkeypatch):
    """The cap as an epilogue of the row-streaming, the weight-streaming, the tcgen05 and the CUDA-core kernel, from logits
    far below the cap to far above it."""
    import locus_b200.kernels as K

    if not tc:
        monkeypatch.setattr(K, "USE_TENSOR_CORES", False)
    g = torch.Generator().manual_seed(M)
    for Kd, N in ((64, 300), (2048, 128)):     # (few columns and a long sum: a plain product would be cut along K)
        x, w = torch.randn(M, Kd, generator=g).to(dtype), (torch.randn(N, Kd, generator=g) * torch.logspace(-2, 0.5, N)[:, None] * Kd ** -0.5 * 4).to(dtype)
        ref, out = torch.zeros(M, N, dtype=torch.float64), torch.zeros(M, N, device=DEV)
        EK.linear(x, w, ref, act="softcap", act_limit=5.0, act_scale=0.6)
        K.linear(x.cuda(), w.cuda(), out, act="softcap", act_limit=5.0, act_scale=0.6)
        _cmp(out, ref, 1e-5)
        assert float(ref.abs().max()) > 4.7
    with pytest.raises(K.KernelError):
        K.linear(x.cuda(), w.cuda(), out, act="softcap", act_limit=0.0)
    with pytest.raises(K.KernelError):
        K.linear(x.cuda(), w.cuda(), out, w2=w.cuda(), act="softcap", act_limit=5.0)


@pytest.mark.parametrize("chunk", [1, 24, 100, 128, 333, 5000])
@pytest.mark.parametrize("nh,nkv,hd,dtype", [(6, 2, 128, torch.bfloat16), (8, 2, 64, torch.bfloat16), (2, 2, 128, torch.bfloat16),
                                             (3, 1, 96, torch.bfloat16), (4, 2, 64, torch.float32), (2, 1, 16, torch.float32)],
                         ids=["6on2_128", "8on2_64", "2on2_128", "3on1_96", "f32_4on2_64", "f32_2on1_16"])
def test_every_attention_kernel_with_chunks(nh, nkv, hd, dtype, chunk):
    """Portions (tcgen05 whole and with its keys cut into ranges, mma.sync in both forms, CUDA cores) and single tokens
    (streaming per head and per group of query heads in both variants, fixed ranges) against the twin in float64; requests
    on both sides of every kind of edge; pages in front of the chunk have gone back, so a key of another chunk is NaN."""
    import locus_b200.kernels as K
    from test_mekizen_gpu import _close, _paged_attention_case

    P = 64
    tol = 1.5e-2 if dtype == torch.bfloat16 else 2e-5
    kw = dict(n_heads=nh, n_kv_heads=nkv, head_dim=hd, page_tokens=P, window=0, scale=0.11, chunk=chunk)

    def twin(pool, q, meta, T, items):
        ref = torch.zeros(T, nh * hd, dtype=torch.float64)
        EK.PRECISE = True
        try:
            EK.attn_chunk(q, pool, ref, items=items, n_items=len(items), **meta, **kw)
        finally:
            EK.PRECISE = False
        return ref

    segs = [(0, 5), (33, 17), (100, 2), (64, 64), (190, 130), (331, 4), (600, 70)]
    pool, q, meta, T = _paged_attention_case(dtype, nh, nkv, hd, P, segs, 0, 0, seed=nh + hd, chunk=chunk)
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
    with pytest.raises(K.KernelError):     # a window beside chunks
        K.attn_chunk(dq, dpool, out, items=items16.cuda(), n_items=len(items16), **dev, **{**kw, "window": 9})

    # single tokens
    ctxs = [0, 1, 23, 24, 31, 32, 47, 99, 100, 127, 128, 255, 332, 333, 666, 700, 1023, 1100]
    pool, q, meta, T = _paged_attention_case(dtype, nh, nkv, hd, P, [(c, 1) for c in ctxs], 0, 0, seed=nh + hd + 1, chunk=chunk)
    items = torch.arange(len(ctxs), dtype=torch.int32)
    ref = twin(pool, q, meta, T, torch.stack([items, torch.zeros_like(items)], 1))
    dev, dq, dpool = {k: v.cuda() for k, v in meta.items()}, q.cuda(), pool.cuda()
    max_splits = max(ctxs) // K.DECODE_SPLIT + 1
    units = K.decode_units(len(ctxs), nh, hd, dtype, max_splits, "cuda", page_tokens=P, n_kv_heads=nkv)
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
    if dtype == torch.bfloat16 and nh != nkv and hd in (64, 128):
        assert ran_gqa, "the grouped decode kernel did not take this shape"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_generation_through_the_engine_and_the_command_line(dtype, cases):
    """Greedy generation with portions, requests side by side and a pool that chunks give pages back to: every token is the
    plain implementation's best one or within rounding of it; the command line says the same tokens in float32."""
    from locus_b200.engine.engine import Engine

    case = cases("mix")
    prompts = [case.tokens[r] for r in ("r2", "r5", "r3")]
    eng = Engine.from_model_dir(case.dir, dtype=dtype, ctx=512, page_tokens=16, max_batch_tokens=32, chunk=16, max_running=2)
    out = eng.generate(prompts, max_new_tokens=8)
    for p, o in zip(prompts, out):
        ref = plain.forward(case.cfg, case.weights, p + o)
        for i, tok in enumerate(o):
            row = ref[len(p) + i - 1]
            assert float(row.max() - row[tok]) <= (1e-4 if dtype == "float32" else 8e-2) * float(ref.abs().max()), (i, tok)
    assert eng.cache.free_pages() == eng.cache.total_pages()
    if dtype != "float32":
        return
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "locus-run"), case.dir, ",".join(map(str, prompts[0])), "8",
                        "--dtype", "float32", "--page-tokens", "16", "--ctx", "512"], capture_output=True, text=True, timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    said = [int(x) for x in r.stdout.replace(",", " ").split() if x.lstrip("-").isdigit()]
    assert said[-8:] == list(out[0]), (said[-8:], out[0])
    archs = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "locus-run"), "--archs"], capture_output=True, text=True)
    assert "Bebovik" in archs.stdout


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_as_a_program(dtype, cases, tmp_path):
    import numpy as np

    case = cases("mix")
    out = tmp_path / "out"
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": case.tokens["r2"][:20], "want": [0, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": case.tokens["r2"][20:22], "want": [1]},
                                     {"id": "b", "tokens": case.tokens["r5"], "want": [18]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": case.tokens["r2"][22:23], "want": [0]}], "end": ["a"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", case.dir, "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True,
                       text=True, timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    ref2, ref5 = case.ref("r2"), case.ref("r5")
    want = {0: ref2[[0, 19]], 1: torch.stack([ref2[21], ref5[18]]), 2: ref2[[22]]}
    tol = TOL[torch.float32 if dtype == "float32" else torch.bfloat16][0]
    for s, ref in want.items():
        got = torch.from_numpy(np.fromfile(out / f"{s}.f32", dtype="<f4").reshape(ref.shape[0], -1)).double()
        err, _ = errors(got, ref)
        assert float(err.max()) <= tol * 3, (s, float(err.max()))
