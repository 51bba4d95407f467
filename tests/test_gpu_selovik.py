"""The Selovik design through the engine: the step function, the cache and state manager, trace replay, the scheduler
and the Python entry point, in 32-bit and in bfloat16, against the plain implementation of tests/plain_selovik.py, on
five small configurations of the tests' own (tests/selovik_models.py)."""
import pytest
import torch

import tiny
import selovik_models as tm

pytestmark = pytest.mark.gpu

LENGTHS = {"a": [1, 2, 5, 40, 90, 130, 33, 64], "b": [3, 1, 70, 16, 17, 100, 48, 2], "c": [330, 7, 129, 64, 200, 65, 1, 150],
           "d": [120, 31, 57, 2, 64, 90, 16, 100], "e": [90, 3, 41, 2, 130, 17, 1, 64]}
TOL = {"float32": 2e-5, "bfloat16": 2.5e-2}
MARGIN = {"float32": 1e-3, "bfloat16": 0.012}      # of the routers' calls, in softmax units


def _close(got, ref, dtype, what, sens=None):
    """A position's bound is the general one or, where that is larger, six times the sensitivity to rounding of the position
    (tests/selovik_models.py). 32-bit: every position within its bound; bfloat16: up to 2 % of a request's positions (at least
    one) may lie over it, none over four times."""
    scale = float(ref.abs().max())
    assert got.shape == ref.shape and torch.isfinite(got).all(), what
    bad = (got.double() - ref.double()).abs().amax(-1) / scale
    bound = torch.full_like(bad, TOL[dtype])
    if sens is not None and dtype == "bfloat16":
        bound = torch.maximum(bound, 6.0 * sens[:bad.shape[0]].double())
    over = int((bad > bound).sum())
    allowed = 0 if dtype == "float32" else max(1, got.shape[0] // 50)
    if over > allowed or bool((bad > 4 * bound).any()):
        worst = int((bad / bound).argmax())
        raise AssertionError(f"{what}: {over} of {got.shape[0]} positions over their bound (allowed {allowed}), the worst "
                             f"{float(bad[worst]):.3e} at {worst} (bound {float(bound[worst]):.1e}); first wrong position "
                             f"{int((bad > bound).nonzero()[0])}")


def _plain(cfg, w, reqs, dtype):
    """({id: plain logits}, {id: sensitivity per position})"""
    exact = {rid: tm.plain.forward(cfg, w, toks) for rid, toks in reqs.items()}
    sens = {rid: tm.sensitivity(cfg, w, toks, exact[rid]) if dtype == "bfloat16" else None for rid, toks in reqs.items()}
    return {rid: t.float() for rid, t in exact.items()}, sens


def _torch_dtype(dtype):
    return torch.float32 if dtype == "float32" else torch.bfloat16


@pytest.fixture(scope="module", params=[(m, d) for m in ("a", "b", "c", "d", "e") for d in ("float32", "bfloat16")], ids=lambda p: f"{p[0]}-{p[1]}")
def setup(request, tmp_path_factory):
    from hipinfer_b200.engine.runner import ModelRunner

    which, dtype = request.param
    folder, cfg, w = tm.make_folder(tmp_path_factory.mktemp(f"selovik_{which}_{dtype}"), which, seed=7, dtype=_torch_dtype(dtype))
    requests = {f"r{i}": tm.safe_tokens(cfg, w, n, 300 + i, MARGIN[dtype]) for i, n in enumerate(LENGTHS[which])}
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
    state (the previous token of a slot's last owner is not the new one's; pages hold what the request itself wrote)."""
    reqs, st = setup["requests"], setup["stepper"]
    first = tiny.run_plan(st, {"r3": reqs["r3"]}, [[("r3", len(reqs["r3"]))]])["r3"]
    others = {r: reqs[r] for r in ("r4", "r5", "r0", "r2", "r7")}
    tiny.run_plan(st, others, tiny.plan_mixed(others, 5))
    again = tiny.run_plan(st, {"r3": reqs["r3"]}, [[("r3", len(reqs["r3"]))]])["r3"]
    assert torch.equal(first, again)


def test_long_decoding(setup):
    """A short prompt, then hundreds of single tokens: decode-only steps replay from CUDA graphs, and the windows' pages are
    given back and used again on the way (the pool is smaller than the sequence)."""
    from hipinfer_b200.engine.runner import ModelRunner

    cfg = setup["cfg"]
    n = min(cfg["max_positions"], 280 if setup["which"] != "c" else 400)
    toks = tm.safe_tokens(cfg, setup["weights"], n, 77, MARGIN[setup["dtype"]])
    ref, sens = _plain(cfg, setup["weights"], {"long": toks}, setup["dtype"])
    got = tiny.run_plan(setup["stepper"], {"long": toks}, [[("long", 6)]] + [[("long", 1)]] * (n - 6))["long"]
    _close(got, ref["long"], setup["dtype"], "long decoding", sens["long"])
    widest = [(L["mixer"].get("mask") or {}).get("size") for L in cfg["layers"]]
    if None in widest:
        return
    few = -(-max(widest) // 16) + 2
    runner = ModelRunner.from_folder(setup["folder"], dtype=setup["dtype"], page_size=16, num_pages=few, max_num_seqs=1)
    assert few * 16 < n
    got = tiny.run_plan(tiny.RunnerStepper(runner), {"long": toks}, [[("long", 6)]] + [[("long", 1)]] * (n - 6))["long"]
    _close(got, ref["long"], setup["dtype"], "long decoding on few pages", sens["long"])


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


def test_every_plane_of_a_prompt_and_of_single_tokens(setup):
    """The residual stream after every layer run of a whole prompt and of decoded tokens, against the plain layers."""
    runner, toks = setup["runner"], setup["requests"]["r3"]
    from hipinfer_b200.engine import StepEntry

    layers = []
    tm.plain.forward(setup["cfg"], setup["weights"], toks, layers)
    cut = max(1, len(toks) - 3)
    steps = [toks[:cut]] + [[t] for t in toks[cut:]]
    at = 0
    for part in steps:
        planes = {}
        runner.step([StepEntry("p", part, [0])], dump=planes)
        for i, want in enumerate(layers):
            got, want = planes[(i, "after_feed_forward")].double().cpu(), want[at:at + len(part)]
            tol = 1e-5 if setup["dtype"] == "float32" else 4e-2
            assert float((got - want).abs().max()) <= tol * float(want.abs().max()), (i, at)
        at += len(part)
    runner.end("p")


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
    """Engine.generate and three requests through the scheduler at once: every token is the plain model's first choice after
    the tokens before it, or nearly ties with it (and no router's call was close on the way)."""
    from hipinfer_b200 import Engine

    cfg, w, n_new = setup["cfg"], setup["weights"], 12

    def check(prompt, got, what):
        calls = []
        logits = tm.plain.forward(cfg, w, prompt + got[:-1], calls=calls)
        assert len(got) == n_new
        for i, t in enumerate(got):
            row = logits[len(prompt) - 1 + i]
            gap = float(row.max() - row[t]) / float(row.abs().max())
            close_call = bool(calls) and float(torch.stack(calls)[:, :len(prompt) + i].min()) < MARGIN[setup["dtype"]]
            assert gap < (0.03 if setup["dtype"] == "bfloat16" else 1e-3) or close_call, f"{what}: token {i} is {t} (gap {gap:.5f})"
            if close_call:
                return

    eng = Engine(setup["folder"], dtype=setup["dtype"], max_batch=3, max_seq=min(256, cfg["max_positions"]), max_prefill=32)
    try:
        prompts = [tm.safe_tokens(cfg, w, n, 900 + n, MARGIN[setup["dtype"]]) for n in (9, 70, 33)]
        check(prompts[0], eng.generate(prompts[0], n_new), "generate")
        ids = [eng.add_request(p, n_new) for p in prompts]        # portions of 32 tokens beside decoding requests
        done = eng.run()
        for i, rid in enumerate(ids):
            check(prompts[i], done[rid], f"scheduler request {i}")
    finally:
        eng.close()


def test_preempted_requests_go_on_where_they_were(tmp_path):
    """A pool too small for three requests: the scheduler takes one back and runs it again from its first token; what it and the
    others produce is what they produce alone (the previous token of a slot belongs to its present owner)."""
    from hipinfer_b200 import Engine

    cfg = tm.model(80, 64, [tm.layer(2, 1, 16, 32, None, 16, mlp=tm.dense(64)), tm.layer(2, 2, 16, 16, None, 8)], loop=(0, 2, 2), max_positions=200)
    folder, cfg, w = tm.make_folder(tmp_path / "m", cfg, seed=2, dtype=torch.float32)
    prompts = [tiny.random_tokens(n, 80, n) for n in (40, 50, 30)]
    alone = []
    eng = Engine(folder, dtype="float32", max_batch=3, max_seq=192, max_prefill=32)
    for p in prompts:
        alone.append(eng.generate(p, 60))
    eng.close()
    eng = Engine(folder, dtype="float32", max_batch=3, max_seq=192, max_prefill=32, num_pages=15)
    ids = [eng.add_request(p, 60) for p in prompts]
    done = eng.run()
    assert [done[i] for i in ids] == alone and eng.scheduler.n_preemptions > 0
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("what", ["no loop", "no bigram table", "nothing but attention", "one layer four times", "an expert alone", "all choices"])
def test_models_without_some_of_the_parts(what, dtype, tmp_path):
    from hipinfer_b200.engine.runner import ModelRunner

    two = [tm.layer(4, 2, 16, 32, 20, 16, mlp=tm.moe(32, 4, 2, 2, (3, 2), 16)), tm.layer(2, 1, 32, 64, None, 16, scaling=tm.yarn(4.0, 64), mlp=tm.dense(64))]
    cfg = {"no loop": tm.model(90, 64, two),
           "no bigram table": tm.model(90, 64, two, loop=(1, 2, 2), bigram=None),
           "nothing but attention": tm.model(90, 64, [tm.layer(3, 1, 8, 16, 31, 4), tm.layer(2, 2, 16, 8, 90)], loop=(0, 1, 2)),
           "one layer four times": tm.model(90, 64, two[:1], loop=(0, 1, 4), scale=3.0),
           "an expert alone": tm.model(90, 64, [tm.layer(2, 1, 16, 16, 16, 8, mlp=tm.moe(32, 1, 1))]),
           "all choices": tm.model(90, 64, [tm.layer(2, 1, 16, 16, 16, 8, mlp=tm.moe(32, 3, 5, 2, None, 24))], loop=(0, 1, 2))}[what]
    cfg["max_positions"] = 200
    folder, cfg, w = tm.make_folder(tmp_path / "m", cfg, seed=3, dtype=_torch_dtype(dtype))
    reqs = {"a": tm.safe_tokens(cfg, w, 150, 1, MARGIN[dtype]), "b": tm.safe_tokens(cfg, w, 37, 2, MARGIN[dtype])}
    ref, sens = _plain(cfg, w, reqs, dtype)
    runner = ModelRunner.from_folder(folder, dtype=dtype, page_size=16, num_pages=24, max_num_seqs=2)
    st = tiny.RunnerStepper(runner)
    for plan in (tiny.plan_whole(reqs), tiny.plan_portions(reqs, (5, 2, 40, 1, 17)), tiny.plan_tail_decode(reqs, 20),
                 tiny.plan_mixed(reqs, 4, max_live=2)):
        got = tiny.run_plan(st, reqs, plan)
        for rid in reqs:
            _close(got[rid], ref[rid], dtype, f"{what} {rid}", sens[rid])
    assert not runner.live_requests()


def _random_config(seed):
    """A configuration drawn from sizes that resemble real layers in the small, on either side of every kernel's size steps."""
    import random

    rng = random.Random(seed)
    pick = rng.choice
    layers = []
    for _ in range(rng.randint(2, 4)):
        what = pick(["none", "dense", "moe", "moe"])
        mlp = None
        if what == "dense":
            mlp = tm.dense(pick([32, 72, 96, 256]))
        elif what == "moe":
            n, span = pick([(1, 6), (2, 3), (3, 2), (4, 3), (3, 4), (7, 1)])
            keep = rng.randint(1, n)
            identity = rng.randint(0, n * span - 2)
            mlp = tm.moe(pick([32, 64, 96, 50]), n * span - identity, rng.randint(1, min(4, keep * span)), identity,
                         (n, keep) if n > 1 else None, pick([None, 32, 64, 50]))
        kv, dim = pick([1, 2, 4]), pick([8, 16, 32, 48, 64, 128])
        layers.append(tm.layer(kv * pick([1, 2, 3, 5]), kv, dim, pick([16, 32, 48, 64, 128]), pick([None, 1, 7, 31, 64, 65, 150]),
                               pick([0, 2, dim // 2, dim]), base=pick([100.0, 10000.0, 500000.0]),
                               scaling=pick([None, tm.yarn(4.0, 64), tm.yarn(32.0, 200, 16.0, 2.0)]), diff=pick([0.1, 0.5, 0.8]), mlp=mlp))
    start = rng.randint(0, len(layers) - 1)
    loop = pick([None, (start, rng.randint(start + 1, len(layers)), rng.randint(1, 3))])
    return tm.model(pick([64, 97, 300]), pick([64, 96, 128, 160]), layers, loop=loop, bigram=pick([None, (31, 5, 3), (997, 131, 77)]),
                    scale=pick([1.0, 5.0]), logit_scale=pick([1.0, 0.3]), eps=pick([1e-5, 1e-6]), max_positions=512)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", list(range(12)))
def test_random_configurations(seed, dtype, tmp_path):
    """A dozen configurations drawn at random: whole prompts, the last tokens one by one, portions, and a mixed batch,
    against the plain model."""
    from hipinfer_b200.engine.runner import ModelRunner

    cfg = _random_config(seed)
    folder, cfg, w = tm.make_folder(tmp_path / "m", cfg, seed=seed, dtype=_torch_dtype(dtype))
    reqs = {"a": tm.safe_tokens(cfg, w, 210, 1, MARGIN[dtype]), "b": tm.safe_tokens(cfg, w, 41, 2, MARGIN[dtype]), "c": tm.safe_tokens(cfg, w, 1, 3, MARGIN[dtype])}
    ref, sens = _plain(cfg, w, reqs, dtype)
    runner = ModelRunner.from_folder(folder, dtype=dtype, page_size=16, num_pages=36, max_num_seqs=3)
    st = tiny.RunnerStepper(runner)
    for plan in (tiny.plan_whole(reqs), tiny.plan_tail_decode(reqs, 24), tiny.plan_portions(reqs, (17, 2, 40, 1, 33)),
                 tiny.plan_mixed(reqs, seed, max_live=3)):
        got = tiny.run_plan(st, reqs, plan)
        for rid in reqs:
            _close(got[rid], ref[rid], dtype, f"random configuration {seed} {rid}", sens[rid])
    assert not runner.live_requests()
