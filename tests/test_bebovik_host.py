"""The Bebovik design through the engine's host logic on the CPU (the kernels replaced by their plain torch twins):
configuration and plan, weights by name (scalars among them), rotation frequencies, pages that go back at a chunk's end,
whole prompts, decoding token by token, portions down to two tokens, mixed batches, chunk edges, and greedy generation
through the scheduler -- all against the plain implementation, which shares no code with any of it.  The kernels
themselves are covered by the gpu tests."""
import copy
import math

import pytest
import torch

import emulated_kernels as EK
import plain_bebovik as plain
from bebovik_cases import BEACON, CONFIGS, Case, attention, beacon, compare, errors, layer, make_runner, model, random_config, run_steps, schedules
import locus_b200.models  # noqa: F401  (registers the architectures)
from locus_b200.config import ConfigError, find_arch
from locus_b200.config.bebovik import BebovikConfig

TOL = (2e-5, 4e-6)   # max and mean |error| of the logits relative to the largest |logit|; float32 twins
F64 = torch.float64
SHOWS = 40 * TOL[0]   # what a fault must move the logits by to count as shown: far beyond the tolerance


@pytest.fixture(autouse=True)
def _emulate(monkeypatch):
    EK.install(monkeypatch)


def _set(raw, path, value):
    node = raw
    for k in path[:-1]:
        node = node[k]
    node[path[-1]] = value
    return raw


def test_config_reads_every_size_and_refuses_what_is_wrong():
    cfg = BebovikConfig.from_dict(copy.deepcopy(CONFIGS["mix"]))
    a, b, c = (cfg.layers[i].mixer for i in (0, 1, 2))
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.chunk) == (4, 2, 24, 24, 0.31, 20)
    s = a.rot.scaling
    assert (a.rot.base, a.rot.dims, s.factor, s.low, s.high, s.original) == (3000.0, 12, 4.0, 1.0, 3.0, 60.0)
    assert b.rot.scaling is None and (b.vdim, b.chunk) == (32, 33)
    assert c.rot is None and c.chunk == 0 and cfg.layers[2].mlp is None
    assert (cfg.layers[1].mlp.ff, cfg.layers[1].mlp.limit) == (40, 0.75)
    assert (cfg.vocab, cfg.width, cfg.eps, cfg.embedding_scale, cfg.logit_scale, cfg.logit_softcap) == (89, 72, 1e-5, 5.0, 0.75, 6.0)
    for path, value, word in ((("layers", 0, "type"), "conv", "type"), (("layers", 0, "mixer", "kv_heads"), 3, "kv_heads"),
                              (("layers", 0, "mixer", "rot", "dims"), 7, "rot.dims"), (("layers", 0, "mixer", "rot", "dims"), 26, "rot.dims"),
                              (("layers", 0, "mixer", "rot", "scaling", "factor"), 0, "factor"),
                              (("layers", 0, "mixer", "rot", "scaling", "high"), 0.5, "high"),
                              (("layers", 0, "mixer", "mask", "size"), 0, "mask.size"), (("layers", 0, "mlp", "kind"), "moe", "kind"),
                              (("layers", 0, "mlp", "limit"), 0, "limit"), (("layers", 0, "mlp"), 3, "mlp"), (("norm",), None, "norm"),
                              (("logit_softcap",), 0, "logit_softcap"), (("logit_scale",), None, "logit_scale"),
                              (("embedding",), None, "embedding"), (("layers",), [], "layers"), (("width",), -1, "width")):
        with pytest.raises(ConfigError, match=word):
            BebovikConfig.from_dict(_set(copy.deepcopy(CONFIGS["mix"]), path, value))


def test_plan_names_tensors_and_groups_layers_by_chunk(tmp_path):
    from locus_b200.cache import CacheManager
    from locus_b200.models.model import Model

    e = find_arch("Bebovik")
    m = Model(e.build_plan(e.parse_config(copy.deepcopy(CONFIGS["mix"]))), torch.float32, "cpu")
    needs = m.cache_needs()
    assert [(p.chunk, p.window, p.n_kv_heads, p.head_dim) for p, _, _ in needs] == [(20, 0, 2, 32), (33, 0, 3, 32), (0, 0, 2, 48), (7, 0, 1, 32)]
    assert all(s is None and c is None for _, s, c in needs)
    names = {s.name: s.shape for _, s in m.tensor_sources()}
    assert names["embed.norm.alpha"] == names["final.norm.alpha"] == names["l1.norm2b.alpha"] == ()
    assert names["l0.mix.q.norm"] == (24,) and names["l1.mix.g"] == (6 * 32, 72) and names["l2.mix.o"] == (72, 16)
    assert {"embed", "head", "embed.norm", "embed.norm.b", "final.norm.b", "l0.norm1b.b", "l0.ls1", "l0.ls2", "l3.mix.k.norm",
            "l0.mlp.gate", "l3.mlp.down", "l2.ls1", "l2.norm1b"} <= set(names)
    assert not {"l2.norm2", "l2.norm2b", "l2.ls2", "l2.mlp.up"} & set(names)
    # pools: a group with chunks holds what its requests can hold at once, the group without one everything
    c = CacheManager(needs, page_tokens=8, n_pages=100, n_state_slots=2, max_seq_tokens=400, max_step_tokens=16)
    assert [g.n_pages for g in c.groups] == [2 * (5 + 1), 2 * (7 + 1), 100, 2 * (3 + 1)]
    assert c.pages_needed(0, 400, 16) == 6 and c.pages_needed(2, 400, 16) == 50 and c.pages_needed(0, 10, 16) == 2
    with pytest.raises(ValueError, match="chunks"):
        from locus_b200.parts.attention import Attention
        Attention("a", hidden=8, n_heads=1, n_kv_heads=1, head_dim=16, qkv_bias=False, window=4, chunk=4)


def test_pages_go_back_at_the_end_of_a_chunk():
    """Pages wholly below the start of the chunk that the next token lies in are free, whatever the portions; the others
    are held; a request that ends gives everything back."""
    from locus_b200.cache import CacheManager
    from locus_b200.parts.base import PagedKvSpec

    for chunk, P in ((20, 8), (8, 8), (1, 4), (6, 16), (64, 8)):
        c = CacheManager([(PagedKvSpec(1, 16, chunk=chunk), None, None)], page_tokens=P, n_pages=64, n_state_slots=1,
                         max_seq_tokens=256, dtype=torch.float32, device="cpu")
        seq, n = c.open("a"), 0
        for k in (1, 5, 14, 1, 19, 2, 40, 8, 7, 1, 64):
            assert c.ensure_capacity(seq, k)
            c.commit(seq, k)
            n += k
            row = c.table_row(seq, 0)
            dead = (n // chunk * chunk) // P
            assert all(p < 0 for p in row[:dead]) and all(p >= 0 for p in row[dead:]), (chunk, P, n)
            c.check_invariants()
        c.release(seq)
        assert c.free_pages() == c.total_pages()


def test_rotation_frequencies_scaled_by_wavelength():
    from locus_b200.parts.position import Rotary

    for base, dims, sc in ((10000.0, 64, (8.0, 1.0, 4.0, 1000)), (500.0, 10, (3.0, 0.5, 2.5, 77)), (2.0, 6, (5.0, 1.0, 1.0, 13))):
        rot = {"base": base, "dims": dims, "scaling": dict(zip(("factor", "low", "high", "original"), sc))}
        part = Rotary("p", head_dim=dims, theta=base, interleaved=True, scaling=rot["scaling"])
        assert part.magnitude() == 1.0
        assert torch.allclose(part.frequencies(), torch.tensor(plain.frequencies(rot), dtype=F64), rtol=1e-13, atol=0)
        f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
        got = plain.frequencies(rot)
        wave = [2 * math.pi / v for v in f]
        assert all(g == v for g, v, l in zip(got, f, wave) if l < sc[3] / sc[2])
        assert all(math.isclose(g, v / sc[0]) for g, v, l in zip(got, f, wave) if l > sc[3] / sc[1])
        assert all(v / sc[0] <= g * (1 + 1e-12) and g <= v for g, v in zip(got, f))
    with pytest.raises(ValueError, match="low"):
        Rotary("p", head_dim=8, theta=10.0, scaling={"factor": 2.0, "original": 8, "high": 2.0, "low": 0.0})


def test_plain_mechanisms_against_their_closed_forms():
    g = torch.Generator().manual_seed(5)
    # the norm: elementwise, a scalar inside, weight and bias outside
    w = {"n": torch.tensor([2.0, -1.0]), "n.b": torch.tensor([0.5, 0.25]), "n.alpha": torch.tensor(0.7)}
    y = plain.dyt(w, "n", torch.tensor([[1.0, -2.0]], dtype=F64))
    a = float(torch.tensor(0.7))
    assert math.isclose(float(y[0, 0]), 2.0 * math.tanh(a) + 0.5) and math.isclose(float(y[0, 1]), -math.tanh(-2 * a) + 0.25)
    # the rotation: adjacent pairs, the tail untouched, position 0 unchanged
    x = torch.randn(4, 1, 6, generator=g, dtype=F64)
    r = plain.rotate_adjacent(x, torch.arange(4), {"base": 100.0, "dims": 4})
    assert torch.equal(r[0], x[0]) and torch.equal(r[..., 4:], x[..., 4:])
    ang = 3.0 * 100.0 ** (-2.0 / 4)
    assert math.isclose(float(r[3, 0, 2]), float(x[3, 0, 2]) * math.cos(ang) - float(x[3, 0, 3]) * math.sin(ang))
    assert math.isclose(float(r[3, 0, 3]), float(x[3, 0, 3]) * math.cos(ang) + float(x[3, 0, 2]) * math.sin(ang))
    # the chunks
    assert [plain.first_visible(p, {"size": 3}) for p in range(7)] == [0, 0, 0, 3, 3, 3, 6] and plain.first_visible(9, None) == 0
    # the feed-forward's clamps: gate bounded above only, the linear part on both sides
    w = {n: torch.ones(1, 1) for n in ("e.gate", "e.up", "e.down")}
    y = plain.clamped_ff({"limit": 1.5}, w, "e.", torch.tensor([[5.0], [-5.0], [0.5]], dtype=F64))
    for v, z in zip(y[:, 0].tolist(), (5.0, -5.0, 0.5)):
        gt, u = min(z, 1.5), max(-1.5, min(z, 1.5))
        assert math.isclose(v, gt / (1 + math.exp(-1.702 * gt)) * (u + 1.0))
    assert math.isclose(float(plain.softcap(torch.tensor(7.0, dtype=F64), 5.0)), 5.0 * math.tanh(1.4))


def test_norms_around_a_sublayer_go_with_other_norms_and_scales():
    """The pending addition behind a sublayer: folded by a Dynamic Tanh, applied first by another norm, with and without a
    scale; an RMS norm behind the sublayer takes the scale into its weight; the head's factor without a cap."""
    from locus_b200.engine.batch import Runtime
    from locus_b200.parts.base import PartSpec, PendingNorm, make_part
    from locus_b200.parts.block import LmHead

    g = torch.Generator().manual_seed(2)
    W = 12
    rand = lambda *s: torch.randn(*s, generator=g)
    dyt = make_part("norm", PartSpec("dynamic_tanh", {"width": W}), "d")
    dyt.params = {"alpha": torch.tensor(0.8), "weight": rand(W), "bias": rand(W)}
    rms = make_part("norm", PartSpec("rmsnorm", {"width": W, "eps": 1e-6}), "r")
    rms.params = {"weight": rand(W)}
    f = {"d": lambda z: torch.tanh(0.8 * z) * dyt.params["weight"] + dyt.params["bias"],
         "r": lambda z: z / torch.sqrt((z * z).mean(-1, keepdim=True) + 1e-6) * rms.params["weight"]}
    parts = {"d": dyt, "r": rms}
    for inner in "dr":
        for outer in "dr":
            for scale in (None, rand(W)):
                for rows in (None, torch.tensor([3, 0], dtype=torch.int32)):
                    x, y = rand(5, W), rand(5, W)
                    want = x + f[inner](y) * (1.0 if scale is None else scale)
                    out = torch.zeros(5 if rows is None else 2, W)
                    parts[outer].forward(x, out, rows, add=PendingNorm(y, parts[inner], scale))
                    assert torch.allclose(out, f[outer](want if rows is None else want[rows.long()]), atol=1e-5)
                    if rows is None:
                        assert torch.allclose(x, want, atol=1e-5)
    head = LmHead("h", vocab=9, hidden=W, scale=0.5)
    head.params = {"weight": rand(9, W)}
    head.bind(Runtime(torch.device("cpu"), torch.float32, 4, 1, 4))
    h, lg = rand(3, W), torch.zeros(3, 9)
    head.forward(h, lg)
    assert torch.allclose(lg, 0.5 * h @ head.params["weight"].T, atol=1e-5)


@pytest.mark.parametrize("name", ["mix", "odd", "wide", "mlp_only"])
def test_every_schedule_against_the_plain_implementation(tmp_path, name):
    lens = (41, 1, 23, 37, 2, 30) if name != "wide" else (75, 33, 5)
    case = Case(name, tmp_path, torch.float32, requests=lens)
    for sched, steps in schedules(case).items():
        runner, cache = make_runner(case, torch.float32, "cpu", page_tokens=8, n_pages=40, max_tokens=160, slots=4)
        got, _ = run_steps(runner, cache, case, steps)
        compare(case, got, *TOL)
        assert cache.free_pages() == cache.total_pages() and cache.state_slots.free == cache.state_slots.total, sched


def test_a_drawn_configuration_in_mixed_batches(tmp_path):
    for seed in (3, 11):
        case = Case(f"drawn{seed}", tmp_path, torch.float32, raw=random_config(seed), requests=(60, 9, 34, 21), seed=seed)
        runner, cache = make_runner(case, torch.float32, "cpu", page_tokens=16, n_pages=24, max_tokens=160, slots=4)
        got, _ = run_steps(runner, cache, case, schedules(case)["mixed"])
        compare(case, got, 1e-4, 2e-5)


def test_the_sharpened_weights_show_each_fault(tmp_path, monkeypatch):
    """What the comparisons rest on: with these weights another chunk, another rotated part or base, unscaled frequencies,
    half-split pairs, a head norm behind the rotation, a lost gate, bias, scalar, layer scale, clamp, cap or factor each
    move the logits by far more than the tolerance."""
    case = Case("mix", tmp_path, torch.float32, requests=(50,))
    ref = case.ref("r0")
    scale = float((ref - ref.mean(-1, keepdim=True)).abs().max())

    def moved(cfg=None, weights=None):
        lg = plain.forward(cfg or case.cfg, weights or case.weights, case.tokens["r0"])
        return float((lg - ref).abs().max()) / scale

    mx = ("layers", 0, "mixer")
    for key, value in ((mx + ("mask", "size"), 21), (mx + ("mask", "size"), 19), (("layers", 1, "mixer", "mask", "size"), 34),
                       (("layers", 3, "mixer", "mask", "size"), 8), (mx + ("rot", "dims"), 10), (mx + ("rot", "base"), 2500.0),
                       (mx + ("rot", "scaling"), None), (mx + ("rot", "scaling", "factor"), 5.0), (mx + ("rot", "scaling", "low"), 1.3),
                       (mx + ("rot", "scaling", "high"), 4.0), (mx + ("rot", "scaling", "original"), 80), (mx + ("scale",), 0.25),
                       (("layers", 0, "mlp", "limit"), 9.0), (("layers", 3, "mlp", "limit"), 2.0), (("embedding", "scale"), 4.5),
                       (("logit_scale",), 0.7), (("logit_softcap",), 7.0), (("norm", "eps"), 1e-1)):
        assert moved(_set(copy.deepcopy(case.cfg), key, value)) > SHOWS, key
    for name in case.weights:
        if name.endswith((".alpha", ".b", ".ls1", ".ls2", ".q.norm", ".k.norm", ".mix.g")):
            w = dict(case.weights)
            w[name] = torch.zeros_like(w[name]) if name.endswith((".b", ".mix.g")) else torch.ones_like(w[name])
            assert moved(weights=w) > SHOWS, name
    half = lambda v, p, rot: plain_half_split(v, p, rot)
    monkeypatch.setattr(plain, "rotate_adjacent", half)
    assert moved() > SHOWS
    monkeypatch.undo()
    monkeypatch.setattr(plain, "head_rms", lambda x, w, eps: x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps))
    assert moved() > SHOWS
    monkeypatch.undo()
    EK.install(monkeypatch)


def plain_half_split(v, positions, rot):
    n = rot["dims"]
    ang = positions.to(F64)[:, None] * torch.tensor(plain.frequencies(rot), dtype=F64)[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    a, b = v[..., : n // 2], v[..., n // 2:n]
    return torch.cat([a * c - b * s, b * c + a * s, v[..., n:]], -1)


def beacon_case(tmp_path, chunk, length, places, dtype=torch.float32):
    """A one-layer model whose token ``BEACON`` stands out, once at each of ``places`` (r<i>: at places[i])."""
    raw = model(48, 50, [layer(attention(4, 2, 16, 16, chunk=chunk, rot=8, scale=0.5), 0)])
    case = Case(f"beacon{chunk}", tmp_path, dtype, raw=raw, requests=(length,) * len(places), tweak=beacon)
    for i, at in enumerate(places):
        case.tokens[f"r{i}"] = [BEACON if p == at else (t if t != BEACON else BEACON + 1) for p, t in enumerate(case.tokens[f"r{i}"])]
    return case


def beacon_reach(case, rid, at, chunk):
    """The plain implementation sees the beacon from every later position of its chunk and from no other."""
    other = list(case.tokens[rid])
    other[at] = BEACON + 1
    moved, _ = errors(plain.forward(case.cfg, case.weights, other), case.ref(rid))
    end = min(len(other), (at // chunk + 1) * chunk) if chunk else len(other)
    assert float(moved[at:end].min()) > SHOWS, (at, float(moved[at:end].min()))
    outside = torch.cat([moved[:at], moved[end:]])
    assert outside.numel() == 0 or float(outside.max()) < 1e-12


def test_keys_just_inside_and_just_outside_a_chunk(tmp_path):
    """A key that stands out at a chunk's first position, its last, at page borders and in the sequence's first tokens, seen
    (or not) by queries in prompts, in portions that start at the edges, and decoded one by one."""
    chunk, n = 40, 96
    places = (0, 39, 40, 47, 48, 79, 80)
    case = beacon_case(tmp_path, chunk, n, places)
    for i, at in enumerate(places):
        beacon_reach(case, f"r{i}", at, chunk)
    steps = []
    for i in range(len(places)):
        r = f"r{i}"
        steps += [[[(r, n)]], [[(r, 38)]] + [[(r, 1)]] * 5 + [[(r, 35)]] + [[(r, 1)]] * 18, [[(r, 2)], [(r, 38)], [(r, 2)], [(r, 37)], [(r, 2)], [(r, 15)]]][i % 3]
    runner, cache = make_runner(case, torch.float32, "cpu", page_tokens=8, n_pages=12, max_tokens=96, slots=1)
    got, _ = run_steps(runner, cache, case, steps)
    compare(case, got, *TOL)


def test_pages_and_slots_are_used_again_under_a_small_pool(tmp_path):
    case = Case("wide", tmp_path, torch.float32, requests=(70, 70, 40, 40, 40))
    runner, cache = make_runner(case, torch.float32, "cpu", page_tokens=8, n_pages=17, max_tokens=72, slots=2)
    steps = [[("r0", 30)], [("r0", 30)], [("r0", 10)], [("r1", 24), ("r2", 8)], [("r1", 23), ("r2", 32)],
             [("r1", 23), ("r3", 2)], [("r3", 38), ("r4", 1)], [("r4", 39)]]
    got, _ = run_steps(runner, cache, case, steps)
    compare(case, got, *TOL)
    assert cache.free_pages() == cache.total_pages()


def test_long_decoding_token_by_token_on_pages_that_chunks_give_back(tmp_path):
    """150 tokens of a model whose layers all have chunks, through a pool that holds one chunk and a page."""
    case = Case("attention_only", tmp_path, torch.float32, requests=(150,))
    runner, cache = make_runner(case, torch.float32, "cpu", page_tokens=4, n_pages=6, max_tokens=32, slots=2)
    got, _ = run_steps(runner, cache, case, [[("r0", 3)]] + [[("r0", 1)]] * 147)
    compare(case, got, *TOL)
    assert cache.free_pages() == cache.total_pages()


def test_greedy_generation_through_the_scheduler(tmp_path):
    from locus_b200.engine.engine import Engine
    from locus_b200.models import load_model

    case = Case("mix", tmp_path, torch.float32, requests=(9, 21, 3))
    m = load_model(case.dir, torch.float32, "cpu")
    eng = Engine.from_model(m, ctx=256, page_tokens=8, max_batch_tokens=16, chunk=8, max_running=2, use_graphs=False)
    prompts = [case.tokens[r] for r in ("r0", "r1", "r2")]
    outs = eng.generate(prompts, max_new_tokens=6)
    for p, o in zip(prompts, outs):
        seq = list(p)
        for tok in o:
            lg = plain.forward(case.cfg, case.weights, seq)
            top2 = torch.topk(lg[-1], 2).values
            if float(top2[0] - top2[1]) > 1e-4 * float(lg[-1].abs().max()):
                assert int(torch.argmax(lg[-1])) == tok
            seq.append(tok)
    assert eng.cache.free_pages() == eng.cache.total_pages()
