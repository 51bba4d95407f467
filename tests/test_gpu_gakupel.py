"""The Gakupel design through the engine: the step function, the cache and state manager, trace replay, the scheduler
and the Python entry point, in 32-bit and in bfloat16, against the plain implementation of tests/plain_gakupel.py, on
four small configurations of the tests' own (tests/gakupel_models.py)."""
import math

import pytest
import torch

import tiny
import gakupel_models as tm

pytestmark = pytest.mark.gpu

LENGTHS = {"a": [1, 2, 5, 40, 90, 130, 33, 64], "b": [3, 1, 70, 16, 17, 100, 48, 2], "c": [600, 7, 129, 64, 200, 65, 1, 150],
           "d": [120, 31, 57, 2, 64, 90, 16, 100]}
TOL = {"float32": 5e-5, "bfloat16": 2.5e-2}


def _close(got, ref, dtype, what, sens=None):
    """A position's bound is the general one or, where that is larger, six times the sensitivity to rounding of the position
    and its two neighbours on either side (tests/gakupel_models.py: a norm that divides by nearly nothing, sums that cancel;
    the estimate is one draw of rounding noise, and what makes a position sensitive also holds a token earlier or later
    through the recurrent state). 32-bit: every position within its bound; bfloat16: up to 3 % of a request's positions (at
    least one) may lie over it, none over four times."""
    scale = float(ref.abs().max())
    assert got.shape == ref.shape and torch.isfinite(got).all(), what
    bad = (got.double() - ref.double()).abs().amax(-1) / scale
    bound = torch.full_like(bad, TOL[dtype])
    if sens is not None:
        near = torch.nn.functional.max_pool1d(sens[:bad.shape[0]].double()[None, None], 5, 1, 2)[0, 0]
        bound = torch.maximum(bound, 6.0 * near)
    over = int((bad > bound).sum())
    allowed = 0 if dtype == "float32" else max(1, (3 * got.shape[0]) // 100)
    if over > allowed or bool((bad > 4 * bound).any()):
        worst = int((bad / bound).argmax())
        raise AssertionError(f"{what}: {over} of {got.shape[0]} positions over their bound (allowed {allowed}), the worst "
                             f"{float(bad[worst]):.3e} at {worst} (bound {float(bound[worst]):.1e}); first wrong position "
                             f"{int((bad > bound).nonzero()[0])}")


def _plain(cfg, w, reqs, dtype):
    """({id: plain logits}, {id: sensitivity per position})"""
    exact = {rid: tm.plain.forward(cfg, w, toks) for rid, toks in reqs.items()}
    ref = {rid: t.float() for rid, t in exact.items()}
    sens = {rid: tm.sensitivity(cfg, w, toks, exact[rid], dtype) for rid, toks in reqs.items()}
    return ref, sens


@pytest.fixture(scope="module", params=[(m, d) for m in ("a", "b", "c", "d") for d in ("float32", "bfloat16")], ids=lambda p: f"{p[0]}-{p[1]}")
def setup(request, tmp_path_factory):
    from hipinfer_b200.engine.runner import ModelRunner

    which, dtype = request.param
    folder, cfg, w = tm.make_folder(tmp_path_factory.mktemp(f"gakupel_{which}_{dtype}"), which, seed=7,
                                    dtype=torch.float32 if dtype == "float32" else torch.bfloat16)
    requests = {f"r{i}": tiny.random_tokens(n, cfg["vocab"], 300 + i) for i, n in enumerate(LENGTHS[which])}
    ref, sens = _plain(cfg, w, requests, dtype)
    longest = -(-max(LENGTHS[which]) // 64) * 64
    # pages for four live requests of the longest kind and four state slots: both are used again
    runner = ModelRunner.from_folder(folder, dtype=dtype, page_size=16, num_pages=4 * longest // 16, max_num_seqs=4)
    yield dict(which=which, dtype=dtype, folder=folder, cfg=cfg, weights=w, requests=requests, ref=ref, sens=sens, runner=runner,
               stepper=tiny.RunnerStepper(runner))
    assert not runner.live_requests()
    runner.cache.check()
    assert runner.cache.free_pages() == [p.num_pages for p in runner.cache.pools]


def _check(setup, plan, what):
    got = tiny.run_plan(setup["stepper"], setup["requests"], plan)
    for rid, ref in setup["ref"].items():
        _close(got[rid], ref, setup["dtype"], f"{what} {setup['which']} {setup['dtype']} {rid}", setup["sens"][rid])
    return got


def test_whole_prompts(setup):
    _check(setup, tiny.plan_whole(setup["requests"]), "whole")


def test_whole_prompts_with_the_recurrence_in_short_pieces(setup, monkeypatch):
    """Prompts of a few dozen tokens already run the matrix memory in pieces (of 8 tokens), in a batch of unequal
    requests too; the states the pieces leave are the ones that the single tokens after them start from."""
    from hipinfer_b200.kernels import ops

    monkeypatch.setattr(ops, "MS_PIECE_TOKENS", 8)
    _check(setup, tiny.plan_whole(setup["requests"]), "whole in pieces")
    _check(setup, tiny.plan_tail_decode(setup["requests"], 5), "pieces then single tokens")
    _check(setup, tiny.plan_mixed(setup["requests"], 11), "mixed in pieces")


def test_last_tokens_one_by_one(setup):
    _check(setup, tiny.plan_tail_decode(setup["requests"], 48), "tail")


def test_every_token_alone(setup):
    short = {r: t for r, t in setup["requests"].items() if len(t) <= 70}
    got = tiny.run_plan(setup["stepper"], short, [[(r, 1)] for r, t in short.items() for _ in t])
    for rid in short:
        _close(got[rid], setup["ref"][rid], setup["dtype"], f"token by token {rid}", setup["sens"][rid])


@pytest.mark.parametrize("sizes", [(7, 2, 16, 3, 2, 33, 5, 2, 64, 1, 9), (2,), (15, 17, 1, 31), (64, 2, 63, 66)])
def test_portions(setup, sizes):
    _check(setup, tiny.plan_portions(setup["requests"], sizes), f"portions {sizes}")


@pytest.mark.parametrize("seed", [0, 1, 2])
def test_mixed_batches(setup, seed):
    _check(setup, tiny.plan_mixed(setup["requests"], seed), f"mixed{seed}")


def test_mixed_batches_with_long_portions(setup):
    _check(setup, tiny.plan_mixed_long(setup["requests"], 1, long=(65, 140)), "mixed long")


def test_a_request_in_a_batch_equals_the_request_alone(setup):
    """Beyond rounding nothing of a row depends on the batch (a routed layer runs single rows and sorted portions on
    different kernels, so the sums' order may differ)."""
    reqs = setup["requests"]
    alone = tiny.run_plan(setup["stepper"], reqs, tiny.plan_whole(reqs))
    ids = list(reqs)
    together = tiny.run_plan(setup["stepper"], reqs, [[(r, len(reqs[r])) for r in ids[:4]], [(r, len(reqs[r])) for r in ids[4:]]])
    tol = 1e-5 if setup["dtype"] == "float32" else 2e-2
    for rid in ids:
        scale = float(alone[rid].abs().max())
        assert float((alone[rid] - together[rid]).abs().max()) <= tol * scale, rid


def test_a_state_slot_and_pages_used_again_start_clean(setup):
    """The same request after others have used and returned every slot and page gives the same bits as on a fresh engine
    state (the recurrent state is zeroed at admission; pages hold what the request itself wrote)."""
    reqs, st = setup["requests"], setup["stepper"]
    first = tiny.run_plan(st, {"r3": reqs["r3"]}, [[("r3", len(reqs["r3"]))]])["r3"]
    others = {r: reqs[r] for r in ("r4", "r5", "r0", "r2", "r7")}
    tiny.run_plan(st, others, tiny.plan_mixed(others, 5))
    again = tiny.run_plan(st, {"r3": reqs["r3"]}, [[("r3", len(reqs["r3"]))]])["r3"]
    assert torch.equal(first, again)


def test_long_decoding(setup):
    """A short prompt, then hundreds of single tokens: decode-only steps replay from CUDA graphs."""
    cfg = setup["cfg"]
    n = min(cfg["max_positions"], 330 if setup["which"] != "c" else 560)
    toks = tiny.random_tokens(n, cfg["vocab"], 77)
    ref, sens = _plain(cfg, setup["weights"], {"long": toks}, setup["dtype"])
    got = tiny.run_plan(setup["stepper"], {"long": toks}, [[("long", 6)]] + [[("long", 1)]] * (n - 6))["long"]
    _close(got, ref["long"], setup["dtype"], "long decoding", sens["long"])
    r = setup["runner"]
    assert r.steps_run > 0


def test_two_requests_decode_together_through_graph_replays(setup):
    reqs = setup["requests"]
    a, b = "r4", "r5"
    ha, hb = len(reqs[a]) // 2, len(reqs[b]) // 3 + 1
    plan = [[(a, ha), (b, hb)]] + [[(a, 1), (b, 1)]] * min(len(reqs[a]) - ha, len(reqs[b]) - hb)
    fed_a, fed_b = ha + len(plan) - 1, hb + len(plan) - 1
    sub = {a: reqs[a][:fed_a], b: reqs[b][:fed_b]}
    got = tiny.run_plan(setup["stepper"], sub, plan)
    _close(got[a], setup["ref"][a][:fed_a], setup["dtype"], "pair a", setup["sens"][a])
    _close(got[b], setup["ref"][b][:fed_b], setup["dtype"], "pair b", setup["sens"][b])


def test_trace_replay_program(setup, tmp_path):
    """bin/trace_run as a child process on the same folder: portions, single tokens, a batch, few pages."""
    reqs = {r: setup["requests"][r] for r in ("r2", "r3", "r6", "r7")}
    tr = tiny.TraceRun(setup["folder"], setup["dtype"], tmp_path / "out", 2 * 64 * -(-max(len(t) for t in reqs.values()) // 64))
    try:
        got = tiny.run_plan(tr, reqs, tiny.plan_mixed(reqs, 3, max_live=2))
    finally:
        tr.close()
    for rid in reqs:
        _close(got[rid], setup["ref"][rid], setup["dtype"], f"trace_run {rid}", setup["sens"][rid])


def test_greedy_generation_through_the_entry_point_and_scheduler(setup):
    """Engine.generate and three requests through the scheduler at once, against greedy decoding with the plain model; a
    different token is accepted only where the plain logits nearly tie."""
    from hipinfer_b200 import Engine

    cfg, n_new = setup["cfg"], 12
    model = tm.PlainGakupel(cfg, setup["weights"])

    def plain_greedy(prompt):
        model.reset()
        logits = model.forward(prompt)[-1]
        out, steps = [], []
        for _ in range(n_new):
            steps.append(logits)
            out.append(int(logits.argmax()))
            logits = model.forward([out[-1]])[-1]
        return out, steps

    def same(got, want, steps, what):
        for i, (g, w) in enumerate(zip(got, want)):
            if g != w:
                top = torch.topk(steps[i], 2).values
                gap = float(top[0] - top[1]) / float(steps[i].abs().max())
                assert gap < (0.02 if setup["dtype"] == "bfloat16" else 1e-3), f"{what}: token {i} is {g}, plain {w} (gap {gap:.5f})"
                return
        assert len(got) == len(want)

    eng = Engine(setup["folder"], dtype=setup["dtype"], max_batch=3, max_seq=min(256, cfg["max_positions"]), max_prefill=32)
    try:
        prompts = [tiny.random_tokens(n, cfg["vocab"], 900 + n) for n in (9, 70, 33)]
        want = [plain_greedy(p) for p in prompts]
        same(eng.generate(prompts[0], n_new), want[0][0], want[0][1], "generate")
        ids = [eng.add_request(p, n_new) for p in prompts]        # portions of 32 tokens beside decoding requests
        done = eng.run()
        for i, rid in enumerate(ids):
            same(done[rid], want[i][0], want[i][1], f"scheduler request {i}")
    finally:
        eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("layers", ["parallel only", "attention only", "delta only", "one layer", "no feed-forward", "ten layers"])
def test_models_of_one_kind_of_layer(layers, dtype, tmp_path):
    """Models of one kind of layer (one without any state, one without any cache), a single layer, layers without
    feed-forward, and a deeper one (the average over eleven states): whole, in portions, token by token and mixed."""
    from hipinfer_b200.engine.runner import ModelRunner

    cfg = tm.model(90, 64, {
        "parallel only": [tm.parallel((2, 2, 32, 16, 0.3, 20), (3, 32, 16, 15.0), mlp=tm.moe(48, 2, 1)),
                          tm.parallel((4, 1, 16, 16), (4, 16, 32, 5.0), mlp=tm.moe(32, 4, 2, (2, 1), 1.0, 16))],
        "attention only": [tm.attention(4, 2, 32, rot_dims=16, mlp=tm.moe(32, 2, 1)), tm.attention(2, 1, 16, rot_dims=16, mlp=tm.dense(64))],
        "delta only": [tm.delta(2, 2, 32, 32, 4, mlp=tm.dense(96)), tm.delta(4, 1, 16, 64, 2, mlp=tm.moe(32, 3, 2))],
        "one layer": [tm.parallel((4, 2, 16, 16), (2, 16, 16, 15.0), mlp=tm.moe(32, 2, 2))],
        "no feed-forward": [tm.parallel((2, 1, 16, 32, 0.2, 5), (2, 32, 16, 9.0)), tm.delta(2, 1, 16, 16, 3), tm.attention(1, 1, 32, rot_dims=8)],
        "ten layers": [tm.parallel((2, 1, 16, 16), (2, 16, 16, 15.0)), tm.delta(2, 1, 16, 16, 4), tm.attention(2, 1, 16, rot_dims=16),
                       tm.delta(2, 2, 16, 16, 2), tm.attention(2, 2, 16)] * 2}[layers], max_positions=200)
    folder, cfg, w = tm.make_folder(tmp_path / "m", cfg, seed=3, dtype=torch.float32 if dtype == "float32" else torch.bfloat16)
    reqs = {"a": tiny.random_tokens(150, 90, 1), "b": tiny.random_tokens(37, 90, 2)}
    ref, sens = _plain(cfg, w, reqs, dtype)
    runner = ModelRunner.from_folder(folder, dtype=dtype, page_size=16, num_pages=24, max_num_seqs=2)
    st = tiny.RunnerStepper(runner)
    for plan in (tiny.plan_whole(reqs), tiny.plan_portions(reqs, (5, 2, 40, 1, 17)), tiny.plan_tail_decode(reqs, 20),
                 tiny.plan_mixed(reqs, 4, max_live=2)):
        got = tiny.run_plan(st, reqs, plan)
        for rid in reqs:
            _close(got[rid], ref[rid], dtype, f"{layers} {rid}", sens[rid])
    assert not runner.live_requests()


def _random_config(seed):
    """A configuration drawn from sizes that resemble real layers in the small: all kinds of layer and feed-forward in a
    random order, sizes on either side of every kernel's size steps."""
    import random

    rng = random.Random(seed)
    pick = rng.choice
    width = pick([64, 96, 128, 160, 192, 256])
    kinds = ["parallel", "attention", "delta"] + [pick(["parallel", "attention", "delta"]) for _ in range(rng.randint(0, 2))]
    rng.shuffle(kinds)
    layers = []
    for kind in kinds:
        what = pick(["none", "dense", "moe", "moe"])
        mlp = None
        if what == "dense":
            mlp = tm.dense(pick([32, 72, 96, 256]))
        elif what == "moe":
            n, span = pick([(1, 4), (2, 2), (4, 2), (4, 4), (3, 3), (8, 1)])
            keep = rng.randint(1, n)
            mlp = tm.moe(pick([32, 64, 96]), n * span, rng.randint(1, min(4, keep * span)), (n, keep) if n > 1 else None,
                         pick([0.5, 1.0, 2.5]), pick([None, 32, 64]))
        kv = pick([1, 2, 4])
        dim = pick([16, 32, 48, 64, 80, 96, 128])
        if kind == "attention":
            layers.append(tm.attention(kv * pick([1, 2, 3, 5]), kv, dim, rot_dims=pick([dim, dim // 2, 0]), base=pick([100.0, 10000.0, 500000.0]), mlp=mlp))
        elif kind == "delta":
            layers.append(tm.delta(kv * pick([1, 2, 3]), kv, pick([16, 32, 48, 64, 128]), pick([16, 32, 48, 64, 128]), pick([2, 3, 4, 9]), mlp=mlp))
        else:
            left = (kv * pick([1, 2, 3, 5]), kv, dim, pick([16, 32, 48, 64, 96, 128])) + pick([(), (0.3, 50), (1.0, 7)])
            layers.append(tm.parallel(left, (pick([1, 2, 4, 6]), pick([16, 32, 48, 64, 128]), pick([16, 32, 48, 64, 128]), pick([2.0, 15.0, 30.0])),
                                      pick([0.3, 0.7, 1.0]), pick([0.8, 1.0, -0.4]), mlp=mlp))
    return tm.model(pick([64, 97, 300, 576]), width, layers, eps=pick([1e-5, 1e-6]), max_positions=512)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", list(range(12)))
def test_random_configurations(seed, dtype, tmp_path):
    """A dozen configurations drawn at random: whole prompts, the last tokens one by one, portions, and a mixed batch,
    against the plain model."""
    from hipinfer_b200.engine.runner import ModelRunner

    cfg = _random_config(seed)
    folder, cfg, w = tm.make_folder(tmp_path / "m", cfg, seed=seed, dtype=torch.float32 if dtype == "float32" else torch.bfloat16)
    reqs = {"a": tiny.random_tokens(210, cfg["vocab"], 1), "b": tiny.random_tokens(41, cfg["vocab"], 2), "c": tiny.random_tokens(1, cfg["vocab"], 3)}
    ref, sens = _plain(cfg, w, reqs, dtype)
    runner = ModelRunner.from_folder(folder, dtype=dtype, page_size=16, num_pages=36, max_num_seqs=3)
    st = tiny.RunnerStepper(runner)
    for plan in (tiny.plan_whole(reqs), tiny.plan_tail_decode(reqs, 24), tiny.plan_portions(reqs, (17, 2, 40, 1, 33)),
                 tiny.plan_mixed(reqs, seed, max_live=3)):
        got = tiny.run_plan(st, reqs, plan)
        for rid in reqs:
            _close(got[rid], ref[rid], dtype, f"random configuration {seed} {rid}", sens[rid])
    assert not runner.live_requests()
