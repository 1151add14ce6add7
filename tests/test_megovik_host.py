"""The Megovik design through the engine's host logic on the CPU (the kernels replaced by their plain torch twins):
configuration and plan, weights by name, the run order with the embedding added again, pending additions, whole prompts,
decoding token by token, portions down to two tokens, mixed batches, far keys, pages and slots used again, and greedy
generation through the scheduler -- all against the plain implementation, which shares no code with any of it.  The kernels
themselves are covered by the gpu tests."""
import copy
import math

import pytest
import torch

import emulated_kernels as EK
import plain_megovik as plain
from megovik_cases import (BEACON, BEACON_HEADS, CONFIGS, Case, attention, beacon, compare, dense, errors, latent, make_runner, model,
                           moe, random_config, run_steps, schedules, with_mlp)
import locus_b200.models  # noqa: F401  (registers the architectures)
from locus_b200.config import ConfigError, find_arch
from locus_b200.config.megovik import MegovikConfig

TOL = (5e-5, 8e-6)    # max and mean |error| of the logits relative to the largest |logit|; float32 twins
TIE = 1e-4            # margin of a router's choice, of the spread of its scores, below which either pick is right
F64 = torch.float64
SHOWS = 20 * TOL[0]   # what a fault must move the logits by to count as shown: far beyond the tolerance


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
    cfg = MegovikConfig.from_dict(copy.deepcopy(CONFIGS["mix"]))
    a, b, c = (cfg.layers[i].mixer for i in (0, 1, 2))
    assert (a.heads, a.dim, a.vdim, a.q_rank, a.kv_rank, a.scale) == (3, 24, 16, 0, 40, 0.21)
    assert (b.heads, b.kv_heads, b.dim, b.scale, b.q_temp.coef, b.q_temp.every) == (6, 2, 24, 0.3, 0.4, 9)
    assert (c.q_rank, c.kv_rank, c.vdim, c.scale) == (32, 24, 40, 0.25)
    m = cfg.layers[0].mlp
    assert (m.experts, m.top, m.group_count, m.group_keep, m.scale, m.expert_ff) == (8, 3, 4, 2, 2.5, 24)
    assert cfg.layers[1].mlp.ff == 56 and cfg.layers[3].mlp is None and cfg.loop == (1, 4, 3)
    assert (cfg.vocab, cfg.width, cfg.max_positions, cfg.eps, cfg.embedding_scale, cfg.logit_scale) == (89, 72, 1024, 1e-5, 3.0, 0.8)
    plainer = MegovikConfig.from_dict(copy.deepcopy(CONFIGS["attention_only"]))
    assert plainer.loop is None and MegovikConfig.from_dict(copy.deepcopy(CONFIGS["odd"])).layers[2].mlp.group_count == 1
    mx, ff = ("layers", 1, "mixer"), ("layers", 0, "mlp")
    for path, value, word in ((("layers", 0, "type"), "conv", "type"), (mx + ("kv_heads",), 4, "kv_heads"), (mx + ("vdim",), 16, "vdim"),
                              (mx + ("q_temp", "every"), 0, "every"), (mx + ("q_temp", "coef"), None, "coef"), (mx + ("scale",), None, "scale"),
                              (("layers", 2, "mixer", "q_rank"), None, "q_rank"), (("layers", 0, "mixer", "kv_rank"), 0, "kv_rank"),
                              (ff + ("kind",), "glu", "kind"), (ff, 3, "mlp"), (ff + ("router", "top"), 9, "top"),
                              (ff + ("router", "groups", "count"), 3, "groups"), (ff + ("router", "groups", "keep"), 1, "groups"),
                              (("layers", 1, "mlp", "ff"), -2, "ff"), (("loop", "stop"), 6, "loop"), (("loop", "times"), 0, "times"),
                              (("norm",), None, "norm"), (("logit_scale",), None, "logit_scale"), (("embedding",), None, "embedding"),
                              (("max_positions",), None, "max_positions"), (("layers",), [], "layers"), (("width",), -1, "width")):
        with pytest.raises(ConfigError, match=word):
            MegovikConfig.from_dict(_set(copy.deepcopy(CONFIGS["mix"]), path, value))


def test_plan_names_tensors_and_gives_every_pass_its_own_cache():
    from locus_b200.models.model import Model

    e = find_arch("Megovik")
    m = Model(e.build_plan(e.parse_config(copy.deepcopy(CONFIGS["mix"]))), torch.float32, "cpu")
    assert [(c.layer, c.add_embedding) for c in m.plan.order] == plain.run_order(CONFIGS["mix"])
    assert [c.layer for c in m.plan.order] == [0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4]
    assert [i for i, c in enumerate(m.plan.order) if c.add_embedding] == [4, 7]
    needs = m.cache_needs()
    one, keys = lambda r: (1, r, False), lambda g, d: (g, d, True)
    assert [(p.n_kv_heads, p.head_dim, p.has_v) for p, _, _ in needs] == [one(40)] + [keys(2, 32), one(24), keys(4, 16)] * 3 + [keys(1, 32)]
    assert all(s is None and c is None and p.window == 0 and p.chunk == 0 for p, s, c in needs)
    assert m.plan.max_positions == 1024
    names = {s.name: s.shape for _, s in m.tensor_sources()}
    assert names["pos"] == (1024, 72) and names["l1.mlp.gate.b"] == (56,) and names["l1.mlp.down.b"] == (72,)
    assert names["l1.mix.k.norm"] == (24,) and names["l1.mix.o"] == (72, 144) and names["l2.mix.uq"] == (32, 32)
    assert names["l0.mix.q"] == (72, 72) and names["l0.mlp.router"] == (8, 72) and names["l0.mlp.e7.down"] == (72, 24)
    assert {"embed", "head", "final.norm", "l3.norm1", "l2.mix.dq.norm", "l0.mix.dkv.norm", "l0.mix.uv"} <= set(names)
    assert not {"l1.mix.v", "l0.mix.dq", "l3.mlp.up", "l0.norm2", "l2.mix.q", "l0.mix.sink", "l1.mix.g"} & set(names)
    # a loop that runs once, or over no layer, adds nothing
    for loop in ((1, 4, 1), (2, 2, 5)):
        raw = copy.deepcopy(CONFIGS["mix"])
        raw["loop"] = dict(zip(("start", "stop", "times"), loop))
        assert [(c.layer, c.add_embedding) for c in e.build_plan(e.parse_config(raw)).order] == [(i, False) for i in range(5)]


def test_a_context_ends_where_the_position_vectors_end(tmp_path):
    from locus_b200.engine.step import StepEntry, StepError

    raw = model(32, 40, [with_mlp(attention(2, 1, 16), None)], positions=20)
    case = Case("short", tmp_path, torch.float32, raw=raw, requests=(20,))
    runner, cache = make_runner(case, torch.float32, "cpu", page_tokens=8, n_pages=8, max_tokens=32, slots=1)
    got, routed = run_steps(runner, cache, case, [[("r0", 19)], [("r0", 1)]])
    compare(case, got, routed, *TOL, TIE)
    seq = cache.open("x")
    assert cache.ensure_capacity(seq, 21)
    with pytest.raises(StepError, match="context overflow"):
        runner.step([StepEntry(seq, [1] * 21, [20])])


def test_plain_mechanisms_against_their_closed_forms():
    assert plain.slopes(4) == [0.25, 0.0625, 0.015625, 0.00390625] and math.isclose(plain.slopes(6)[0], 2.0 ** (-4.0 / 3.0))
    t = {"coef": 0.5, "every": 10}
    assert plain.temperature(8, t) == 1.0 and math.isclose(plain.temperature(9, t), 1 + 0.5 * math.log(2))
    assert math.isclose(plain.temperature(29, t), 1 + 0.5 * math.log(4)) and plain.temperature(50, None) == 1.0
    # one query over three keys: scores 2, 0, 1 less slope times the distance
    q, k = torch.tensor([[0.0], [0.0], [1.0]], dtype=F64), torch.tensor([[2.0], [0.0], [1.0]], dtype=F64)
    v = torch.tensor([[1.0], [10.0], [100.0]], dtype=F64)
    e = [math.exp(2.0 - 0.6), math.exp(0.0 - 0.3), math.exp(1.0)]
    assert math.isclose(float(plain.causal_softmax(q, k, v, 1.0, 0.3)[2, 0]), (e[0] + 10 * e[1] + 100 * e[2]) / sum(e))
    # the router: groups of two by the sum of their scores, the best expert's group may be closed
    r = {"top": 2, "scale": 3.0, "groups": {"count": 3, "keep": 2}}
    s = [0.9, 0.05, 0.6, 0.5, 0.7, 0.45]
    picked, groups, _ = plain.choose(r, s)
    assert picked == [4, 2] and all(math.isclose(a, b) for a, b in zip(groups, (0.95, 1.1, 1.15)))
    assert all(math.isclose(a, b) for a, b in zip(plain.shares(r, s, picked), (3 * 0.7 / 1.3, 3 * 0.6 / 1.3)))
    assert plain.choose({"top": 1, "scale": 1.0}, s)[0] == [0] and plain.shares(r, [0.0] * 6, [1, 2]) == [0.0, 0.0]
    # the dense unit: the rectified gate, biases on all three projections
    w = {f"e.{n}": torch.full((1, 1), m) for n, m in (("gate", 2.0), ("up", 3.0), ("down", 0.5))}
    w.update({f"e.{n}.b": torch.full((1,), m) for n, m in (("gate", -1.0), ("up", 0.25), ("down", 7.0))})
    for z in (1.5, 0.3):
        assert math.isclose(float(plain.dense_ff(w, "e.", torch.tensor([[z]], dtype=F64))), max(2 * z - 1, 0) * (3 * z + 0.25) * 0.5 + 7.0)


def test_rows_added_between_two_layer_calls_go_with_every_norm_and_pending_sum():
    """x += y behind what the block in front left, folded into an RMS norm's pass or applied in front of another norm; over
    all rows (which come back changed) and over gathered rows; widths with and without the folded form."""
    from locus_b200.parts.base import PartSpec, PendingAdd, PendingRows, make_part

    g = torch.Generator().manual_seed(2)
    for W in (12, 10):
        rand = lambda *s: torch.randn(*s, generator=g)
        rms = make_part("norm", PartSpec("rmsnorm", {"width": W, "eps": 1e-6}), "r")
        ln = make_part("norm", PartSpec("layernorm", {"width": W, "eps": 1e-6}), "l")
        rms.params, ln.params = {"weight": rand(W)}, {"weight": rand(W), "bias": rand(W)}
        pairs, pos = rand(10, W), torch.randperm(10, generator=g).to(torch.int32)
        summed = torch.stack([pairs[pos[2 * t]] + pairs[pos[2 * t + 1]] for t in range(5)])
        for norm in (rms, ln):
            for before in (False, True):
                for rows in (None, torch.tensor([3, 0], dtype=torch.int32)):
                    x, y = rand(5, W), rand(5, W)
                    want = x + y + (summed if before else 0.0)
                    out, ref = torch.zeros(5 if rows is None else 2, W), torch.zeros(5 if rows is None else 2, W)
                    norm.forward(x, out, rows, add=PendingRows(y, PendingAdd(pairs, pos, 2) if before else None))
                    norm.forward(want, ref, rows)
                    assert torch.allclose(out, ref, atol=1e-5)
                    if rows is None:
                        assert torch.allclose(x, want, atol=1e-5)


def test_parts_refuse_what_does_not_go_together():
    from locus_b200.parts.attention import Attention
    from locus_b200.parts.base import LayerCall
    from locus_b200.parts.block import Embedding
    from locus_b200.parts.feed_forward import DenseMlp, SparseMoe
    from locus_b200.models.model import Model

    a = dict(hidden=8, n_heads=2, n_kv_heads=1, head_dim=16, qkv_bias=False)
    for bad in (dict(values="queries"), dict(values="keys", v_dim=32), dict(values="keys", conv_taps=3), dict(q_temp=(0.5, 0)),
                dict(slopes=(0.5,)), dict(values="keys", qkv_bias=True)):
        with pytest.raises(ValueError):
            Attention("a", **{**a, **bad})
    with pytest.raises(ValueError, match="bias"):
        DenseMlp("m", hidden=8, intermediate=8, bias=True)
    with pytest.raises(ValueError, match="activation"):
        SparseMoe("m", hidden=8, n_experts=2, top_k=1, norm_topk=True, expert_intermediate=8, activation="reglu")
    with pytest.raises(ValueError, match="position"):
        Embedding("e", vocab=4, hidden=8, positions={"tensor": "p", "count": 4}, pair={"tensor": "b", "buckets": 3, "mul_prev": 1, "mul_cur": 1})
    e = find_arch("Pozozen")
    from pozozen_cases import CONFIGS as POZ
    raw = next(c for c in POZ.values() if c.get("streams", 0) > 1)
    plan = e.build_plan(e.parse_config(copy.deepcopy(raw)))
    plan.order[-1] = LayerCall(plan.order[-1].layer, add_embedding=True)
    with pytest.raises(ValueError, match="one residual stream"):
        Model(plan, torch.float32, "cpu")


@pytest.mark.parametrize("name", ["mix", "odd", "wide", "moe_only", "latents_only", "dense_only"])
def test_every_schedule_against_the_plain_implementation(tmp_path, name):
    lens = {"mix": (33, 1, 20, 29, 2), "wide": (60, 21, 5)}.get(name, (41, 1, 23, 2, 30))
    case = Case(name, tmp_path, torch.float32, requests=lens)
    for sched, steps in schedules(case).items():
        runner, cache = make_runner(case, torch.float32, "cpu", page_tokens=8, n_pages=30, max_tokens=160, slots=4)
        got, routed = run_steps(runner, cache, case, steps)
        compare(case, got, routed, *TOL, TIE)
        assert cache.free_pages() == cache.total_pages() and cache.state_slots.free == cache.state_slots.total, sched


def test_drawn_configurations_in_mixed_batches(tmp_path):
    for seed in (3, 11, 12):
        case = Case(f"drawn{seed}", tmp_path, torch.float32, raw=random_config(seed), requests=(50, 9, 34, 21), seed=seed)
        runner, cache = make_runner(case, torch.float32, "cpu", page_tokens=16, n_pages=24, max_tokens=160, slots=4)
        got, routed = run_steps(runner, cache, case, schedules(case)["mixed"])
        compare(case, got, routed, 2e-4, 4e-5, TIE)


def test_the_sharpened_weights_show_each_fault(tmp_path, monkeypatch):
    """What the comparisons rest on: with these weights another loop, a lost position vector, temperature, slope, norm weight,
    bias, group or factor, values behind the keys' norm, and an embedding that is not added again each move the logits by
    far more than the tolerance."""
    case = Case("mix", tmp_path, torch.float32, requests=(40,))
    ref = case.ref("r0")[0]
    scale = float((ref - ref.mean(-1, keepdim=True)).abs().max())

    def moved(cfg=None, weights=None):
        lg = plain.forward(cfg or case.cfg, weights or case.weights, case.tokens["r0"])
        return float((lg - ref).abs().max()) / scale

    mx, router = ("layers", 1, "mixer"), ("layers", 0, "mlp", "router")
    for key, value in ((mx + ("q_temp",), None), (mx + ("q_temp", "coef"), 0.35), (mx + ("q_temp", "every"), 10), (mx + ("scale",), 0.28),
                       (("layers", 3, "mixer", "q_temp", "every"), 24), (("layers", 0, "mixer", "scale"), 0.2), (("layers", 2, "mixer", "scale"), 0.2),
                       (router + ("scale",), 2.3), (router + ("top",), 2), (router + ("groups", "keep"), 3), (router + ("groups",), None),
                       (("layers", 4, "mlp", "router", "groups"), None), (("embedding", "scale"), 2.8), (("logit_scale",), 0.75),
                       (("loop", "times"), 2), (("loop", "stop"), 3), (("loop", "start"), 2), (("loop",), None), (("norm", "eps"), 1e-1),
                       (("layers", 1, "mlp"), None), (("layers", 2, "mlp"), None)):
        assert moved(_set(copy.deepcopy(case.cfg), key, value)) > SHOWS, key
    for name in case.weights:
        if name.endswith((".b", ".norm", ".norm1")) or name == "pos":
            w = dict(case.weights)
            w[name] = torch.zeros_like(w[name]) if name.endswith(".b") or name == "pos" else torch.ones_like(w[name])
            assert moved(weights=w) > SHOWS, name
    # each equation changed in the plain implementation
    keep = {n: getattr(plain, n) for n in ("slopes", "causal_softmax", "run_order", "temperature")}

    def shows(name, other):
        monkeypatch.setattr(plain, name, other)
        assert moved() > SHOWS, name
        monkeypatch.setattr(plain, name, keep[name])

    shows("slopes", lambda heads: [0.0] * heads)
    shows("slopes", lambda heads: [2.0 ** (-8.0 * h / heads) for h in range(heads)])
    shows("run_order", lambda cfg: [(i, False) for i, _ in keep["run_order"](cfg)])
    shows("run_order", lambda cfg: [(i, k > 0 and i in (1, 2, 3) and k > 3) for k, (i, _) in enumerate(keep["run_order"](cfg))])
    shows("temperature", lambda p, t: keep["temperature"](p - 1, t))
    shows("causal_softmax", lambda q, k, v, s, slope=0.0: keep["causal_softmax"](q, k, k if slope and k.shape == v.shape else v, s, slope))


def beacon_case(tmp_path, kind, length, places, dtype=torch.float32):
    """A one-layer model whose token ``BEACON`` stands out, once at each of ``places`` (r<i>: at places[i])."""
    mixer = {"attention": attention(4, 2, 16, scale=2.0), "latent": latent(BEACON_HEADS, 16, 16, 32, scale=0.5),
             "latent2": latent(BEACON_HEADS, 16, 24, 32, q_rank=16, scale=0.5)}[kind]
    raw = model(48, 50, [with_mlp(mixer, None)], emb=1.0)
    case = Case(f"beacon_{kind}", tmp_path, dtype, raw=raw, requests=(length,) * len(places), tweak=beacon)
    for i, at in enumerate(places):
        case.tokens[f"r{i}"] = [BEACON if p == at else (t if t != BEACON else BEACON + 1) for p, t in enumerate(case.tokens[f"r{i}"])]
    return case


def beacon_reach(case, rid, at):
    """The plain implementation sees the beacon from every later position and from none before it."""
    other = list(case.tokens[rid])
    other[at] = BEACON + 1
    moved, _ = errors(plain.forward(case.cfg, case.weights, other), case.ref(rid)[0])
    assert float(moved[at:].min()) > SHOWS, (at, float(moved[at:].min()))
    assert at == 0 or float(moved[:at].max()) < 1e-12


@pytest.mark.parametrize("kind", ["attention", "latent", "latent2"])
def test_keys_far_away(tmp_path, kind):
    """A key that stands out at the first position, at page borders and late, seen by queries in prompts, in portions that
    start around it, and decoded one by one."""
    n, places = 90, (0, 7, 8, 47, 48, 70)
    case = beacon_case(tmp_path, kind, n, places)
    steps = []
    for i, at in enumerate(places):
        r = f"r{i}"
        beacon_reach(case, r, at)
        steps += [[[(r, n)]], [[(r, 60)]] + [[(r, 1)]] * 30, [[(r, 2)], [(r, 45)], [(r, 2)], [(r, 2)], [(r, 30)]] + [[(r, 1)]] * 9][i % 3]
    runner, cache = make_runner(case, torch.float32, "cpu", page_tokens=8, n_pages=12, max_tokens=96, slots=1)
    got, routed = run_steps(runner, cache, case, steps)
    compare(case, got, routed, *TOL, TIE)


def test_long_portions_with_expanded_keys_and_values(tmp_path, monkeypatch):
    """Portions of at least eight tokens take the rows form, as long as their contexts' rows fit together: beside single tokens
    and short portions in one step, with cached tokens in front, more of them than fit, and behind pages in any order."""
    import locus_b200.kernels as K

    monkeypatch.setattr(K, "LATENT_EXPAND_FROM", 8)
    monkeypatch.setattr(K, "latent_decode_takes", lambda dtype, rank, rot: rank == 32)   # (single tokens apart in the first layer)
    monkeypatch.setattr(K, "latent_expand_rows", lambda dtype, H, dn, dr, dv, rank: 90 if dn == dv else 0)
    raw = model(48, 50, [with_mlp(latent(4, 16, 16, 32), dense(24)), with_mlp(latent(2, 24, 24, 24, q_rank=16), None)])
    case = Case("expanded", tmp_path, torch.float32, raw=raw, requests=(60, 40, 30, 70))
    runner, cache = make_runner(case, torch.float32, "cpu", page_tokens=8, n_pages=30, max_tokens=160, slots=4)
    calls, rows = [], K.attn_chunk_tc_rows
    singles, decode = [], K.latent_decode
    monkeypatch.setattr(K, "latent_decode", lambda *a, **kw: (singles.append(kw["items"].tolist()), decode(*a, **kw)))
    monkeypatch.setattr(K, "attn_chunk_tc_rows", lambda *a, **kw: (calls.append(sorted({int(s) for s, _ in kw["items"].tolist()})), rows(*a, **kw)))
    steps = [[("r0", 20), ("r1", 2)], [("r0", 10), ("r1", 20), ("r2", 1)], [("r0", 30), ("r1", 18), ("r2", 28), ("r3", 50)], [("r2", 1), ("r3", 18)], [("r3", 1)], [("r3", 1)]]
    got, routed = run_steps(runner, cache, case, steps)
    compare(case, got, routed, *TOL, TIE)
    # (third step: 60 rows, 40 that do not fit, 29, 50 that do not)
    assert calls == [[0]] * 2 + [[0, 1]] * 2 + [[0, 2]] * 2 + [[1]] * 2
    assert singles == [[2], [0], [0], [0]]


def test_pages_and_slots_are_used_again_under_a_small_pool(tmp_path):
    case = Case("wide", tmp_path, torch.float32, requests=(60, 60, 30, 30, 30))
    runner, cache = make_runner(case, torch.float32, "cpu", page_tokens=8, n_pages=13, max_tokens=72, slots=2)
    steps = [[("r0", 30)], [("r0", 30)], [("r1", 24), ("r2", 8)], [("r1", 13), ("r2", 22)],
             [("r1", 23), ("r3", 2)], [("r3", 28), ("r4", 1)], [("r4", 29)]]
    got, routed = run_steps(runner, cache, case, steps)
    compare(case, got, routed, *TOL, TIE)
    assert cache.free_pages() == cache.total_pages()


def test_long_decoding_token_by_token(tmp_path):
    case = Case("attention_only", tmp_path, torch.float32, requests=(130,))
    runner, cache = make_runner(case, torch.float32, "cpu", page_tokens=4, n_pages=40, max_tokens=32, slots=2)
    got, routed = run_steps(runner, cache, case, [[("r0", 3)]] + [[("r0", 1)]] * 127)
    compare(case, got, routed, *TOL, TIE)


def test_greedy_generation_through_the_scheduler(tmp_path):
    from locus_b200.engine.engine import Engine
    from locus_b200.models import load_model

    case = Case("mix", tmp_path, torch.float32, requests=(9, 21, 3))
    m = load_model(case.dir, torch.float32, "cpu")
    eng = Engine.from_model(m, ctx=256, page_tokens=8, max_batch_tokens=16, chunk=8, max_running=2, use_graphs=False)
    prompts = [case.tokens[r] for r in ("r0", "r1", "r2")]
    outs = eng.generate(prompts, max_new_tokens=6)
    for p, o in zip(prompts, outs):
        lg = plain.forward(case.cfg, case.weights, list(p) + list(o))
        for i, tok in enumerate(o):
            row = lg[len(p) + i - 1]
            assert float(row.max() - row[tok]) <= 1e-4 * float(lg.abs().max())
    assert eng.cache.free_pages() == eng.cache.total_pages()
