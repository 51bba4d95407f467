"""Each mechanism of the Selovik design alone: the kernel against the plain function of tests/plain_selovik.py, in 32-bit and
in bfloat16, at sizes the vectorised paths take and at sizes they do not, with inputs made so that a fault shows (one key at a
window's edge whose score stands out, a slot that holds another request's token, choices of both signs)."""
import math
from types import SimpleNamespace

import pytest
import torch

import plain_selovik as plain

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
TOL = {torch.float32: 2e-5, torch.bfloat16: 1.2e-2}
F = torch.float64
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])


def rnd(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


def close(got, want, dtype, what="", tol=None):
    got, want = got.double().cpu(), want.double()
    err, ref = float((got - want).abs().max()), float(want.abs().max())
    assert got.shape == want.shape and torch.isfinite(got).all(), what
    assert err <= (tol or TOL[dtype]) * ref, f"{what}: {err:.3e} > {tol or TOL[dtype]:.0e} * {ref:.3e}"


def i32(values):
    return torch.tensor(list(values), dtype=torch.int32, device=DEV)


def batch_of(lengths, ctx=None, slots=None, tokens=None):
    """What the kernels read of a step: requests of `lengths` rows each, after `ctx` cached tokens."""
    ctx = ctx or [0] * len(lengths)
    starts = [sum(lengths[:r]) for r in range(len(lengths))]
    return SimpleNamespace(n_requests=len(lengths), max_q_len=max(lengths), req_q_start=i32(starts), req_q_len=i32(lengths),
                           req_ctx_len=i32(ctx), req_state_slot=i32(slots or range(len(lengths))), h_q_len=list(lengths),
                           h_ctx_len=list(ctx), h_q_start=starts, extra={}, n_rows=sum(lengths), dump=None,
                           row_request=i32(r for r, n in enumerate(lengths) for _ in range(n)),
                           positions=i32(c + i for c, n in zip(ctx, lengths) for i in range(n)),
                           max_pos=max(c + n for c, n in zip(ctx, lengths)) - 1, tokens=None if tokens is None else i32(tokens))


def part(role, kind, params, dtype, tensors, **ctx):
    from hipinfer_b200.parts.registry import BuildContext, build_part
    from hipinfer_b200.parts.spec import PartSpec

    p = build_part(role, PartSpec(kind, params), BuildContext(dtype, DEV, **ctx))
    assert sorted(s.name for s in p.param_specs()) == sorted(tensors)
    for s in p.param_specs():
        assert tuple(s.shape) == tuple(tensors[s.name].shape), s.name
    p.load({n: t.to(DEV) for n, t in tensors.items()})
    return p


# ------------------------------------------------------------------------------------------ embedding
@BOTH
@pytest.mark.parametrize("W", [50, 64, 1000, 2048, 3072, 8196])
@pytest.mark.parametrize("bigram", [(37, 5, 3), (1, 2, 9), (1009, 4000000007, 2500000001), None])
def test_bigram_embedding_over_portions_and_slots(dtype, W, bigram):
    """Two requests in portions beside each other (a portion's first row finds the token before it in the request's slot), then
    another request in a slot that holds an old token; the copy is the same bits."""
    from hipinfer_b200.parts.spec import PartSpec

    V, eps, scale = 60, 1e-5, 3.25
    t = {"embed": rnd(V, W, seed=1), "embed.norm": rnd(W, seed=2, scale=0.3)}
    if bigram:
        t["bigram"] = rnd(bigram[0] + 1, W, seed=3, scale=3.0)
    t = {n: v.to(dtype) for n, v in t.items()}
    p = part("embedding", "token_bigram", dict(name="embed", vocab_size=V, hidden_size=W, scale=scale, bigram=bigram,
                                               norm=PartSpec("rmsnorm", dict(name="embed.norm", size=W, eps=eps, one_plus=True))), dtype, t)
    assert list(p.state_need()) == (["previous"] if bigram else [])
    cfg = dict(norm=dict(eps=eps), embedding=dict(scale=scale))
    if bigram:
        cfg["embedding"]["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    g = torch.Generator().manual_seed(4)
    reqs = [torch.randint(0, V, (n,), generator=g).tolist() for n in (23, 9, 5)]
    want = [plain.embedding(r, t, cfg) for r in reqs]
    state = {"previous": torch.full((5,), 41, dtype=torch.int32, device=DEV)}
    fed, got, slots = [0, 0, 0], [[], [], []], [3, 0, 3]
    # (request, rows): portions of both, single tokens, and at last request 2 in the slot of request 0
    for step in ([(0, 1), (1, 4)], [(1, 1), (0, 9)], [(0, 1)], [(0, 2), (1, 2)], [(1, 2), (0, 10)], [(2, 3)], [(2, 1)], [(2, 1)]):
        toks = [reqs[r][fed[r]:fed[r] + n] for r, n in step]
        b = batch_of([n for _, n in step], [fed[r] for r, _ in step], [slots[r] for r, _ in step], [x for ts in toks for x in ts])
        copy = torch.empty(b.n_rows, W, device=DEV)
        x = p.forward(b, state, copy=copy)
        assert torch.equal(x, copy) and x.dtype == torch.float32
        at = 0
        for r, n in step:
            got[r].append(x[at:at + n].cpu())
            fed[r] += n
            at += n
    for r in range(3):
        close(torch.cat(got[r]), want[r], torch.float32, f"request {r}")
    if bigram:
        assert state["previous"].tolist() == [reqs[1][-1], 41, 41, reqs[2][-1], 41]


# ------------------------------------------------------------------------------------------ norms, the block, the loop
@BOTH
@pytest.mark.parametrize("W", [50, 64, 1000, 2048, 4096, 8192, 8196])
def test_two_norms_of_one_row_with_what_a_pass_adds(dtype, W):
    from hipinfer_b200.kernels import ops

    T, eps = 5, 1e-5
    x, add, vec = rnd(T, W, seed=1) * 3, rnd(T, W, seed=2), rnd(W, seed=3)
    w1, w2 = 1 + 0.3 * rnd(W, seed=4), 1 + 0.3 * rnd(W, seed=5)
    d = lambda t: t.to(DEV).clone()
    for a, v in ((None, None), (add, vec), (None, vec), (add, None)):
        s = x.double() + (0 if a is None else a.double()) + (0 if v is None else v.double())
        for u1, u2 in ((w1, w2), (w1, None), (None, None)):
            xd = d(x)
            y1, y2 = ops.two_norms(xd, None if u1 is None else d(u1), None if u2 is None else d(u2), eps, dtype,
                                   None if a is None else d(a), None if v is None else d(v))
            close(xd, s, torch.float32, "sum")
            assert (y1 is None) == (u1 is None) and (y2 is None) == (u2 is None)
            if u1 is not None:
                close(y1, plain.norm(s, u1.double() - 1, eps), dtype, "first")
            if u2 is not None:
                close(y2, plain.norm(s, u2.double() - 1, eps), dtype, "second")


def test_norm_weight_around_zero_with_a_gain():
    x, w = rnd(6, 96, seed=1) * 4, rnd(96, seed=2, scale=0.4)
    p = part("norm", "rmsnorm", dict(name="n", size=96, eps=1e-4, one_plus=True, gain=0.3), torch.float32, {"n": w})
    close(p.forward(x.to(DEV), rows=i32([4, 1])), 0.3 * plain.norm(x.double()[[4, 1]], w.double(), 1e-4), torch.float32)


@pytest.mark.parametrize("second", ["rmsnorm", "layernorm", "other eps"])
def test_block_adds_both_results_of_the_same_rows(second):
    """Mixer and feed-forward read norms of the same x (the feed-forward does not see the mixer's result), also where the norms
    are not of one kind."""
    from hipinfer_b200.cache.storage import LayerCache
    from hipinfer_b200.parts.registry import BuildContext, build_part
    from hipinfer_b200.parts.spec import LayerSpec, PartSpec

    W, T, eps = 32, 9, 1e-5
    m = dict(heads=2, kv_heads=1, dim=8, vdim=16, scale=0.4, diff=0.4, mask=dict(size=4))
    shapes = {"q": (32, W), "k": (16, W), "v": (16, W), "g": (32, W), "o": (W, 32), "lq1": (8,), "lk1": (8,), "lq2": (8,), "lk2": (8,)}
    t = {"l.mix." + n: rnd(*s, seed=i, scale=0.3) for i, (n, s) in enumerate(shapes.items())}
    t.update({"l.mlp.up": rnd(40, W, seed=20, scale=0.3), "l.mlp.down": rnd(W, 40, seed=21, scale=0.3),
              "l.norm1": rnd(W, seed=22, scale=0.3), "l.norm2": rnd(W, seed=23, scale=0.3)})
    n2 = {"rmsnorm": PartSpec("rmsnorm", dict(name="norm2", size=W, eps=eps, one_plus=True)), "layernorm": PartSpec("layernorm", dict(name="norm2", size=W, eps=eps)),
          "other eps": PartSpec("rmsnorm", dict(name="norm2", size=W, eps=0.5, one_plus=True))}[second]
    layer = LayerSpec("l.", "parallel_two_norms", dict(
        mixer_norm=PartSpec("rmsnorm", dict(name="norm1", size=W, eps=eps, one_plus=True)), feed_forward_norm=n2,
        mixer=PartSpec("differential_attention", dict(hidden_size=W, eps=eps, biases=False, window=4, **{k: v for k, v in m.items() if k != "mask"})),
        feed_forward=PartSpec("activated", dict(hidden_size=W, intermediate_size=40, activation="relu2"))))
    b = build_part("block", PartSpec("parallel_two_norms", dict(layer=layer)), BuildContext(torch.float32, DEV, max_model_len=16), "l.")
    b.load({n: v.to(DEV) for n, v in t.items()})
    x, first, step = rnd(T, W, seed=30), rnd(T, W, seed=31), rnd(W, seed=32)
    planes = {n: torch.zeros(1, heads, 16, width, device=DEV) for n, heads, width in b.mixer.cache_need().planes}
    batch = batch_of([T])
    batch.block_tables, batch.slot_maps = [i32([0])[None]], [i32(range(T))]
    xd = x.to(DEV).clone()
    b.forward(xd, batch, LayerCache(planes, 0, True), {}, entry=(first.to(DEV), step.to(DEV)))
    s = x.double() + first.double() + step.double()
    w = {n.split("l.", 1)[1]: v.double() for n, v in t.items()}
    h2 = {"rmsnorm": lambda: plain.norm(s, w["norm2"], eps), "other eps": lambda: plain.norm(s, w["norm2"], 0.5),
          "layernorm": lambda: torch.nn.functional.layer_norm(s, (W,), w["norm2"], None, eps)}[second]()
    want = s + plain.attention(plain.norm(s, w["norm1"], eps), plain.sub(w, "mix."), m, eps) + plain.dense(h2, plain.sub(w, "mlp."))
    close(xd, want, torch.float32, tol=4e-5)


def test_a_pass_of_layers_whose_block_knows_nothing_of_it(tmp_path):
    """The loop over blocks that do not add a pass's vector themselves (the decoder then does), and over an embedding that keeps
    no copy of its rows: a pre-norm model run three times against the sum of its steps."""
    import dataclasses

    import selovik_models as tm
    import tiny
    from hipinfer_b200.config import config_from_dict, get_architecture
    from hipinfer_b200.config.base import register_architecture
    from hipinfer_b200.engine.batch import StepEntry
    from hipinfer_b200.engine.runner import ModelRunner
    from hipinfer_b200.parts.spec import LayerSpec, PartSpec

    cfg = tm.model(64, 32, [tm.layer(2, 1, 16, 16, 20, 16, mlp=tm.dense(48)), tm.layer(2, 2, 8, 16, None, 4, mlp=tm.dense(32))],
                   loop=(0, 2, 3), bigram=None, max_positions=100)
    w = tm.draw_weights(cfg, 3, torch.float32)

    def spec(c):
        s = get_architecture("Selovik").build_spec(c)
        layers = tuple(LayerSpec(L.prefix, "pre_norm", L.parts, L.params) for L in s.layers)
        return dataclasses.replace(s, layers=layers, embedding=PartSpec("token", dict(name="embed", vocab_size=64, hidden_size=32)))

    register_architecture("SelovikPreNorm", type(config_from_dict(cfg)), spec)
    c = dataclasses.replace(config_from_dict(cfg), architecture="SelovikPreNorm")
    toks = tiny.random_tokens(40, 64, 2)
    for dtype, tol in (("float32", 5e-5), ("bfloat16", 3e-2)):
        runner = ModelRunner(c, {n: t.to(DEV) for n, t in w.items() if n != "embed.norm"}, dtype=dtype, num_pages=8, max_num_seqs=1)
        got = [runner.step([StepEntry("a", toks[:25], list(range(25)))]).cpu()]
        got += [runner.step([StepEntry("a", [t], [0])]).cpu() for t in toks[25:]]
        x = x0 = w["embed"].double()[toks]
        for t in range(3):
            x = x + (x0 if t else 0) + w["loop.step"].double()[t]
            for i in range(2):
                p = plain.sub(w, f"l{i}.")
                x = x + plain.attention(plain.norm(x, p["norm1"], 1e-5), plain.sub(p, "mix."), cfg["layers"][i]["mixer"], 1e-5)
                x = x + plain.dense(plain.norm(x, p["norm2"], 1e-5), plain.sub(p, "mlp."))
        close(torch.cat(got), plain.norm(x, w["final.norm"].double(), 1e-5) @ w["embed"].double().T, torch.float32, dtype, tol=tol)


# ------------------------------------------------------------------------------------------ rotation and cache write
@BOTH
@pytest.mark.parametrize("H,G,M,D,E,rot", [(6, 2, 2, 64, 32, 64), (3, 1, 2, 10, 6, 6), (4, 4, 1, 32, 64, 16), (2, 1, 2, 128, 128, 8), (4, 2, 3, 16, 24, 0),
                                           (2, 2, 2, 24, 40, 12), (5, 1, 2, 32, 32, 24)])
@pytest.mark.parametrize("scaling", [None, dict(factor=8.0, original=100, fast=32.0, slow=1.0)])
@pytest.mark.parametrize("T", [1, 11, 700])
def test_rotation_with_scaling_and_maps_side_by_side(dtype, H, G, M, D, E, rot, scaling, T):
    """Every map of every q and k head is rotated by itself; a kv head's maps lie side by side in its key row; values pass."""
    from hipinfer_b200.kernels import ops

    ps, base, off = 8, 5000.0, 4
    proj = rnd(T, off + H * M * D + G * M * D + G * E, seed=1)
    pos = torch.randint(0, 3000, (T,), generator=torch.Generator().manual_seed(2))
    pages = -(-T // ps) + 2
    slots = torch.randperm(pages * ps, generator=torch.Generator().manual_seed(4))[:T].to(torch.int32)
    table = ops.shared_rope_table(rot, base, 3000, DEV, dict(scaling, kind="yarn") if scaling else None)
    q = torch.empty(T, H * M * D, dtype=dtype, device=DEV)
    kc, vc = torch.zeros(pages, G, ps, M * D, dtype=dtype, device=DEV), torch.zeros(pages, G, ps, E, dtype=dtype, device=DEV)
    offs = (off, off + H * M * D, off + H * M * D + G * M * D)
    ops.rope_norm_store(proj.to(DEV), offs, pos.to(torch.int32).to(DEV), slots.to(DEV), table, rot, "half", False, 0.0, q, kc, vc, H * M,
                        G * M, D, E, ps, maps=M)
    p64, r = proj.double(), dict(dims=rot, base=base, scaling=scaling)
    tol = None if dtype == torch.bfloat16 else 3e-4                      # float32(position) * frequency is a 32-bit angle
    close(q.view(T, H, M, D), plain.rotate(p64[:, offs[0]:offs[1]].reshape(T, H, M, D), pos, r), dtype, "q", tol)
    k = plain.rotate(p64[:, offs[1]:offs[2]].reshape(T, G, M, D), pos, r).reshape(T, G, M * D)
    page, o = (slots // ps).long(), (slots % ps).long()
    close(kc.cpu()[page, :, o], k, dtype, "k", tol)
    close(vc.cpu()[page, :, o], p64[:, offs[2]:].reshape(T, G, E), dtype, "v")
    assert int((kc != 0).any(-1).any(1).sum()) == T
    q2 = torch.empty_like(q)                                              # without a slot map: q alone, the same bits
    ops.rope_norm_store(proj.to(DEV), offs, pos.to(torch.int32).to(DEV), None, table, rot, "half", False, 0.0, q2, None, None, H * M, G * M, D,
                        E, ps, maps=M)
    assert torch.equal(q, q2)


# ------------------------------------------------------------------------------------------ attention
def _attention(dtype, m, h, w, cuts, eps=1e-5, W=48, page=16):
    """A differential_attention part over one sequence cut into `cuts`: its result."""
    from hipinfer_b200.cache.storage import LayerCache

    T = sum(cuts)
    rot = m.get("rot") or dict(dims=0, base=1.0)
    sc = dict(rot["scaling"], kind="yarn") if rot.get("scaling") else None
    p = part("mixer", "differential_attention", dict(
        hidden_size=W, heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=m["scale"], diff=m["diff"], eps=eps,
        window=(m.get("mask") or {}).get("size"), biases=False, rot_dims=rot["dims"], rot_base=rot["base"], rot_scaling=sc), dtype,
        {"mix." + n: t for n, t in w.items()}, page_size=page, max_model_len=T)
    need = p.cache_need()
    pages = -(-T // page)
    planes = {n: torch.full((pages, heads, page, width), float("nan"), dtype=dtype, device=DEV) for n, heads, width in need.planes}
    perm = torch.randperm(pages, generator=torch.Generator().manual_seed(9)).to(torch.int32)
    got, at = [], 0
    for n in cuts:
        b = batch_of([n], [at])
        table = perm.clone()
        if p.window:                                     # pages behind the window of every row of the step are gone
            table[:max(0, at - p.window + 1) // page] = -1
        b.block_tables = [table[None].to(DEV)]
        for plane in planes.values():                    # (the pools start zeroed; what is behind a window may hold anything)
            for lp in range(at // page if at % page else at // page, -(-(at + n) // page)):
                fresh = plane[int(perm[lp])]
                fresh[torch.isnan(fresh)] = 0
        b.slot_maps = [i32(int(perm[j // page]) * page + j % page for j in range(at, at + n))]
        x = torch.zeros(n, W, dtype=torch.float32, device=DEV)
        p.forward(h[at:at + n].to(dtype).to(DEV), x, b, LayerCache(planes, 0, True), {})
        got.append(x.cpu())
        at += n
    return torch.cat(got)


def _weights(m, dtype, W=48, gain=0.2):
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    w = dict(q=rnd(H * 2 * D, W, seed=1, scale=gain), k=rnd(G * 2 * D, W, seed=2, scale=gain), v=rnd(G * E, W, seed=3, scale=0.2),
             g=rnd(H * E, W, seed=4, scale=0.2), o=rnd(W, H * E, seed=5, scale=0.1),
             **{n: rnd(D, seed=6 + i, scale=0.4 / D ** 0.25) for i, n in enumerate(("lq1", "lk1", "lq2", "lk2"))})
    return {n: t.to(dtype) for n, t in w.items()}


ATTN = [dict(heads=9, kv_heads=3, dim=32, vdim=64, scale=0.2, diff=0.45, mask=dict(size=37), rot=dict(dims=16, base=1000.0, scaling=dict(factor=6.0, original=64, fast=32.0, slow=1.0))),
        dict(heads=6, kv_heads=2, dim=64, vdim=128, scale=0.125, diff=0.2, mask=dict(size=64), rot=dict(dims=64, base=500.0)),
        dict(heads=3, kv_heads=3, dim=10, vdim=6, scale=0.3, diff=0.8, mask=dict(size=17), rot=dict(dims=6, base=100.0)),
        dict(heads=4, kv_heads=1, dim=128, vdim=64, scale=0.1, diff=0.4, mask=dict(size=65)),
        dict(heads=2, kv_heads=1, dim=16, vdim=32, scale=0.25, diff=0.3, rot=dict(dims=16, base=10000.0)),
        dict(heads=20, kv_heads=1, dim=8, vdim=24, scale=0.35, diff=0.6, mask=dict(size=1), rot=dict(dims=2, base=10.0)),
        dict(heads=8, kv_heads=4, dim=64, vdim=64, scale=0.125, diff=0.5, mask=dict(size=130), rot=dict(dims=32, base=2000.0)),
        dict(heads=2, kv_heads=2, dim=32, vdim=128, scale=0.15, diff=0.5, rot=dict(dims=32, base=2000.0))]


@BOTH
@pytest.mark.parametrize("m", ATTN, ids=lambda m: f"{m['heads']}-{m['kv_heads']}-{m['dim']}-{m['vdim']}-w{(m.get('mask') or {}).get('size', 0)}")
@pytest.mark.parametrize("cuts", [(300,), (1,) * 20, (33, 2, 1, 64, 17, 63, 1, 1, 2, 129), (200,) + (1,) * 12, (129, 128, 43)])
def test_attention_part_in_portions(dtype, m, cuts):
    """Pages behind the window hold NaN and are gone from the block table: a key that is not visible is never read."""
    w, h = _weights(m, dtype), rnd(sum(cuts), 48, seed=20).to(dtype).float()
    want = plain.attention(h.double(), {n: t.double() for n, t in w.items()}, m, 1e-5)
    close(_attention(dtype, m, h, w, cuts), want, dtype, tol=4e-5 if dtype == torch.float32 else 2e-2)


@pytest.mark.parametrize("page", [8, 32, 64])
@pytest.mark.parametrize("H,G,D,window", [(1, 1, 32, 50), (8, 4, 32, 700), (6, 2, 32, 513), (4, 1, 32, None), (3, 1, 64, 300), (8, 2, 64, None), (2, 2, 64, 257)])
def test_attention_over_pages_of_other_sizes_and_several_chunks(page, H, G, D, window):
    """One to four heads a kv head, windows of several key chunks of the decode kernel, pages of 8 to 64 tokens: a long portion, then
    single tokens far into the sequence (whose window starts inside a page, on its edge and on a chunk's edge)."""
    m = dict(heads=H, kv_heads=G, dim=D, vdim=2 * D, scale=D ** -0.5, diff=0.4, rot=dict(dims=D, base=3000.0))
    if window:
        m["mask"] = dict(size=window)
    dtype, T = torch.bfloat16, 1160
    w, h = _weights(m, dtype), rnd(T, 48, seed=20).to(dtype).float()
    want = plain.attention(h.double(), {n: t.double() for n, t in w.items()}, m, 1e-5)
    close(_attention(dtype, m, h, w, (1020, 3, 1, 70) + (1,) * 66, page=page), want, dtype, tol=2e-2)


@BOTH
@pytest.mark.parametrize("window", [1, 2, 16, 63, 64, 65, 128, 150])
@pytest.mark.parametrize("dim,vdim", [(32, 64), (64, 128), (24, 16)])
@pytest.mark.parametrize("split", [0, 12, 200])
def test_a_key_just_inside_and_just_outside_the_window(dtype, window, dim, vdim, split):
    """One key of one map stands out for every later query (both maps by turns); its value is large. A query sees it up to the
    window's last place and not one further, in a prompt, in its later portions and in single tokens."""
    T, W, at = 240, 48, 40
    for map_ in (0, 1):
        m = dict(heads=2, kv_heads=1, dim=dim, vdim=vdim, scale=1.0, diff=0.5, mask=dict(size=window))
        w = _weights(m, dtype, gain=0.02)
        q, k = w["q"].view(2, 2, dim, W), w["k"].view(1, 2, dim, W)
        q[:, :, 0], k[:, :, 0] = 0.0, 0.0
        q[:, map_, 0, 0] = 6.0                             # channel 0 is one in every row, channel 1 marks the key
        k[:, map_, 0, 1] = 4.0
        w["v"][:, 1] = 3.0
        h = rnd(T, W, seed=21, scale=0.3)
        h[:, 0], h[:, 1] = 1.0, 0.0
        h[at, 1] = 1.0
        h = h.to(dtype).float()
        want = plain.attention(h.double(), {n: t.double() for n, t in w.items()}, m, 1e-5)
        cuts = (T,) if not split else (split, 1, 1, T - split - 2) if split == 12 else (split,) + (1,) * (T - split)
        if split == 200 and at + window > T:
            continue
        got = _attention(dtype, m, h, w, cuts)
        close(got, want, dtype, tol=4e-5 if dtype == torch.float32 else 2.5e-2)
        # and the key matters: with a window one longer or one shorter the rows at the edge differ plainly
        for other, row in ((window + 1, at + window), (window - 1, at + window - 1)):
            if row < T and other > 0:
                alt = plain.attention(h.double(), {n: t.double() for n, t in w.items()}, dict(m, mask=dict(size=other)), 1e-5)
                assert float((alt[row] - want[row]).abs().max()) > 0.1 * float(want[row].abs().max()), (other, row)


@pytest.mark.parametrize("m", [ATTN[0], ATTN[1], ATTN[6], ATTN[7]], ids=["32-64", "64-128", "64-64", "32-128"])
def test_unequal_requests_in_one_batch(m):
    """Long portions, short ones and single rows of several requests at once, over caches of several lengths, on pages that lie
    in any order."""
    from hipinfer_b200.kernels import ops

    H, G, D, E, ps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], 16
    window, dtype, eps, lam = (m.get("mask") or {}).get("size") or 0, torch.bfloat16, 1e-5, 0.61
    lengths, ctx = [150, 1, 16, 15, 129, 1, 2], [0, 299, 37, 5, 200, 0, 63]
    total = [c + n for c, n in zip(ctx, lengths)]
    R, wide = len(lengths), -(-max(total) // ps)
    n_pages = sum(-(-t // ps) for t in total)
    perm = torch.randperm(n_pages, generator=torch.Generator().manual_seed(1))
    kc, vc = torch.zeros(n_pages, G, ps, 2 * D, dtype=dtype), torch.zeros(n_pages, G, ps, E, dtype=dtype)
    tables, at = torch.full((R, wide), -1, dtype=torch.int32), 0
    k, v, q = [], [], []
    for r in range(R):
        n = -(-total[r] // ps)
        tables[r, :n] = perm[at:at + n].to(torch.int32)
        at += n
        k.append(rnd(total[r], G, 2 * D, seed=10 + r).to(dtype))
        v.append(rnd(total[r], G, E, seed=30 + r).to(dtype))
        q.append(rnd(lengths[r], H, 2 * D, seed=50 + r).to(dtype))
        for j in range(total[r]):
            kc[tables[r, j // ps], :, j % ps], vc[tables[r, j // ps], :, j % ps] = k[r][j], v[r][j]
    b = batch_of(lengths, ctx)
    b.block_tables = [tables.to(DEV)]
    gate = rnd(b.n_rows, H * E + 6, seed=70)
    out = torch.empty(b.n_rows, H * E, dtype=dtype, device=DEV)
    ops.attention_window(torch.cat(q).reshape(b.n_rows, -1).to(DEV), kc.to(DEV), vc.to(DEV), b, 0, out, H, G, D, E, 2, ps, window, 0,
                         m["scale"], lam, 0.7, eps, True, gate=gate.to(DEV), gate_offset=6)
    at = 0
    for r in range(R):
        pos, kp = torch.arange(ctx[r], total[r])[:, None], torch.arange(total[r])[None]
        hide = (kp > pos) | ((pos - kp >= window) if window else torch.zeros(1, dtype=torch.bool))
        want = torch.zeros(lengths[r], H, E, dtype=F)
        for hd in range(H):
            g = hd // (H // G)
            a = [torch.softmax(((q[r][:, hd, j * D:(j + 1) * D].double() @ k[r][:, g, j * D:(j + 1) * D].double().T) * m["scale"])
                               .masked_fill(hide, float("-inf")), -1) @ v[r][:, g].double() for j in (0, 1)]
            want[:, hd] = plain.head_norm(a[0] - lam * a[1], eps) * 0.7
        want = want.reshape(lengths[r], -1) * torch.sigmoid(gate[at:at + lengths[r], 6:].double())
        close(out[at:at + lengths[r]], want, dtype, f"request {r}", tol=2e-2)
        at += lengths[r]


# ------------------------------------------------------------------------------------------ feed-forwards
@BOTH
@pytest.mark.parametrize("W,ff", [(64, 96), (50, 30), (128, 320), (256, 1024)])
@pytest.mark.parametrize("T", [1, 7, 40, 64, 65, 300])
def test_dense_feed_forward_with_the_square_of_relu(dtype, W, ff, T):
    up, down, h = rnd(ff, W, seed=1, scale=2.0 / math.sqrt(W)).to(dtype), rnd(W, ff, seed=2, scale=1 / math.sqrt(ff)).to(dtype), rnd(T, W, seed=3).to(dtype)
    p = part("feed_forward", "activated", dict(hidden_size=W, intermediate_size=ff, activation="relu2"), dtype, {"mlp.up": up, "mlp.down": down})
    x = torch.zeros(T, W, device=DEV)
    p.forward(h.to(DEV), x, None)
    close(x, plain.dense(h.double(), {"up": up.double(), "down": down.double()}), dtype)


ROUTERS = [dict(experts=9, identity=6, top=4, groups=dict(count=5, keep=3)), dict(experts=14, identity=2, top=2, groups=dict(count=8, keep=1)),
           dict(experts=5, top=2), dict(experts=1, top=1), dict(experts=1, identity=3, top=2), dict(experts=4, identity=4, top=3, groups=dict(count=8, keep=4)),
           dict(experts=6, top=6, groups=dict(count=2, keep=2)), dict(experts=40, identity=8, top=5, groups=dict(count=6, keep=2))]


@BOTH
@pytest.mark.parametrize("r", ROUTERS, ids=lambda r: f"{r['experts']}-{r.get('identity', 0)}-{r['top']}-{(r.get('groups') or {}).get('count', 1)}")
@pytest.mark.parametrize("W", [64, 50, 2048])
@pytest.mark.parametrize("T", [3, 400, 701])
def test_router(dtype, r, W, T):
    """Corrections of both signs move the choice but not the weights; a group is as good as its best; choice scores below zero are
    still chosen; the identity experts' weights are summed. Rows whose call is close are left out."""
    from hipinfer_b200.kernels import ops

    top, n_id = r["top"], r.get("identity", 0)
    E = r["experts"] + n_id
    h, router = rnd(T, W, seed=1).to(dtype), rnd(E, W, seed=2, scale=1.5 / math.sqrt(W)).to(dtype)
    corr = (rnd(E, seed=3) * 0.2 - 0.15).to(dtype)
    g = r.get("groups") or dict(count=1, keep=1)
    idw = torch.full((T,), 7.0, device=DEV)
    expert, weight = ops.moe_route(h.to(DEV), router.to(DEV), top, None, "softmax", corr.to(DEV), g["count"], g["keep"], identity=n_id,
                                   identity_weight=idw)
    h64, r64, c64 = h.double(), router.double(), corr.double()
    chosen, want = plain.route(h64, r64, c64, r)
    sure = plain.closest_call(h64, r64, c64, r) > 1e-4
    ordered = torch.sort(torch.gather(torch.softmax(h64 @ r64.T, -1) + c64, 1, chosen), -1, descending=True).values
    if top > 1:
        sure &= (ordered[:, :-1] - ordered[:, 1:]).amin(-1) > 1e-4      # (the order among the chosen is compared too)
    assert int(sure.sum()) > T // 2
    assert torch.equal(expert.cpu().long()[sure], chosen[sure])
    close(weight.cpu()[sure], want[sure], torch.float32)
    if n_id:
        close(idw.cpu()[sure], torch.where(chosen >= r["experts"], want, torch.zeros_like(want)).sum(-1)[sure] + 0.0, torch.float32, tol=1e-4)
    if g["keep"] < g["count"] and E > g["count"] and T > 100:
        ungrouped = plain.route(h64, r64, c64, dict(top=top))[0]
        assert float((ungrouped.sort(-1).values != chosen.sort(-1).values).any(-1).double().mean()) > 0.03, "the groups decide nothing: not tested"
        by_two = torch.softmax(h64 @ r64.T, -1) + c64
        by_two = torch.sort(by_two.reshape(T, g["count"], -1), -1, descending=True).values[..., :2].sum(-1)
        by_max = (torch.softmax(h64 @ r64.T, -1) + c64).reshape(T, g["count"], -1).amax(-1)
        assert bool((by_two.argmax(-1) != by_max.argmax(-1)).any()), "ranked by two or by one: not told apart"


def test_router_ties_go_to_the_lower_index():
    from hipinfer_b200.kernels import ops

    h, router, corr = torch.ones(1, 16, device=DEV), torch.zeros(8, 16, device=DEV), torch.zeros(8, device=DEV)
    expert, weight = ops.moe_route(h, router, 3, None, "softmax", corr, 4, 2)
    assert expert.tolist() == [[0, 1, 2]] and float((weight - 1 / 8).abs().max()) < 1e-6


@BOTH
@pytest.mark.parametrize("W,Fe,Fs,r", [(64, 32, 48, ROUTERS[0]), (50, 10, 6, ROUTERS[2]), (128, 96, None, ROUTERS[5]), (96, 40, 200, ROUTERS[4]),
                                       (64, 64, 64, ROUTERS[1])])
@pytest.mark.parametrize("T,prompt", [(1, False), (3, False), (8, False), (9, False), (40, False), (70, True), (200, True)])
def test_experts_with_identity_and_shared_ones(dtype, W, Fe, Fs, r, T, prompt):
    """The three ways a step runs the experts, beside a shared one; identity experts among the choices. Every token's code sits
    in the first channels, so that no call is close."""
    top, n_id = r["top"], r.get("identity", 0)
    E = r["experts"] + n_id
    t = {"mlp.router": torch.cat([3.0 * torch.eye(E), torch.zeros(E, W - E)], 1), "mlp.correction": 0.15 * rnd(E, seed=2) - 0.3}
    for e in range(r["experts"]):
        t.update({f"mlp.e{e}.gate": rnd(Fe, W, seed=10 + e, scale=0.3), f"mlp.e{e}.up": rnd(Fe, W, seed=40 + e, scale=0.3),
                  f"mlp.e{e}.down": rnd(W, Fe, seed=70 + e, scale=0.2)})
    if Fs:
        t.update({"mlp.shared.gate": rnd(Fs, W, seed=3, scale=0.3), "mlp.shared.up": rnd(Fs, W, seed=4, scale=0.3),
                  "mlp.shared.down": rnd(W, Fs, seed=5, scale=0.2)})
    t = {n: v.to(dtype) for n, v in t.items()}
    g, gen = r.get("groups"), torch.Generator().manual_seed(8)
    h = rnd(T, W, seed=7).to(dtype)
    todo = torch.ones(T, dtype=torch.bool)
    for _ in range(300):
        h[todo, :E] = torch.randn(int(todo.sum()), E, generator=gen).to(dtype)
        todo = plain.closest_call(h.double(), t["mlp.router"].double(), t["mlp.correction"].double(), r) < 0.01
        if not bool(todo.any()):
            break
    assert not bool(todo.any())
    p = part("feed_forward", "routed", dict(hidden_size=W, experts=r["experts"], identity=n_id, top=top, expert_size=Fe, score="softmax",
                                            weight_at="output", groups=(g["count"], g["keep"]) if g else None, shared_size=Fs), dtype, t)
    x = torch.full((T, W), 0.5, device=DEV)
    p.forward(h.to(DEV), x, SimpleNamespace(max_q_len=T if prompt else 1, dump=None))
    want = 0.5 + plain.experts(h.double(), {n.split("mlp.")[1]: v.double() for n, v in t.items()}, r)
    close(x, want, dtype)
    if n_id and T > 8:
        chosen = plain.route(h.double(), t["mlp.router"].double(), t["mlp.correction"].double(), r)[0]
        assert bool((chosen >= r["experts"]).any()) and bool((chosen < r["experts"]).any())


@pytest.mark.parametrize("E,W,F,T,top,n_id", [(3, 64, 32, 40, 2, 1), (9, 128, 80, 300, 2, 5), (5, 96, 160, 515, 3, 0), (70, 64, 64, 900, 4, 10),
                                              (200, 64, 32, 600, 3, 0), (1, 64, 128, 129, 1, 0), (4, 256, 48, 1, 1, 3)])
@pytest.mark.parametrize("at_output", [True, False])
def test_all_experts_products_in_one_kernel(E, W, F, T, top, n_id, at_output):
    """Blocks of sorted rows that end inside a tile of 128, experts without rows, more than 64 experts, both tile widths; rows of
    identity experts are left alone. The weight multiplies the result, or both halves of the gate/up product."""
    from hipinfer_b200.kernels import fast, ops

    g = torch.Generator().manual_seed(E)
    wgu, wd = (torch.randn(*s, generator=g) * s[2] ** -0.5 for s in ((E, 2 * F, W), (E, W, F)))
    wgu, wd, x = wgu.bfloat16(), wd.bfloat16(), torch.randn(T, W, generator=g).bfloat16()
    expert = torch.stack([torch.randperm(E + n_id, generator=g)[:top] for _ in range(T)]).to(torch.int32)
    if E > 2:
        expert[expert == 1] = 0                                  # an expert without rows, another with many
    score = torch.rand(T, top, generator=g)
    offsets, pos, src = ops.moe_sort(expert.to(DEV), E + n_id)
    xs, sc = ops.moe_gather(x.to(DEV), src, top, offsets[E:]), score.to(DEV)
    b, order = offsets.tolist(), src.cpu().long()
    for tile in (128, 256, 0):
        act = torch.full((T * top, F), 7.0, dtype=torch.bfloat16, device=DEV)
        ys = torch.full((T * top, W), 7.0, device=DEV)
        assert fast.grouped_linear(xs, wgu.to(DEV), offsets, act, src, sc, at_output, tile)
        assert fast.grouped_linear(act, wd.to(DEV), offsets, ys, None, None, False, tile)
        for e in range(E):
            rows = order[b[e]:b[e + 1]]
            if not rows.numel():
                continue
            gu = (x[rows // top].double() @ wgu[e].double().T).view(-1, F // 16, 2, 16)
            gate, up, s = gu[:, :, 0].reshape(-1, F), gu[:, :, 1].reshape(-1, F), score.flatten()[rows][:, None].double()
            close(act[b[e]:b[e + 1]], plain.silu(gate) * up * s if at_output else plain.silu(gate * s) * (up * s), torch.bfloat16)
            close(ys[b[e]:b[e + 1]], act[b[e]:b[e + 1]].cpu().double() @ wd[e].double().T, torch.float32, tol=1e-4)
        assert bool((act[b[E]:] == 7).all()) and bool((ys[b[E]:] == 7).all())
    # the same by the kernels for few rows
    few = torch.full((T * top, F), 7.0, dtype=torch.bfloat16, device=DEV)
    for parts in (1, 2, 4):
        assert ops.moe_grouped_act(x.to(DEV), src, top, wgu.to(DEV), offsets, sc, few, at_output, parts, 16)
        close(few[:b[E]], act[:b[E]].cpu(), torch.bfloat16)
        assert bool((few[b[E]:] == 7).all())


def test_a_step_all_of_whose_choices_are_identity_experts():
    """No expert with weights has a row: nothing is read of them, in any of the three ways."""
    W = 64
    t = {"mlp.router": torch.cat([torch.zeros(2, W), torch.ones(2, W)]), "mlp.correction": torch.zeros(4)}
    for e in range(2):
        t.update({f"mlp.e{e}.{k}": torch.full(s, float("nan")) for k, s in (("gate", (32, W)), ("up", (32, W)), ("down", (W, 32)))})
    for dtype in (torch.float32, torch.bfloat16):
        p = part("feed_forward", "routed", dict(hidden_size=W, experts=2, identity=2, top=2, expert_size=32, score="softmax", weight_at="output"), dtype,
                 {n: v.to(dtype) for n, v in t.items()})
        for T, prompt in ((2, False), (30, False), (100, True)):
            h = rnd(T, W, seed=3).abs().to(dtype)
            x = torch.zeros(T, W, device=DEV)
            p.forward(h.to(DEV), x, SimpleNamespace(max_q_len=T if prompt else 1, dump=None))
            s = torch.softmax(h.double() @ t["mlp.router"].double().T, -1)
            close(x, s[:, 2:].sum(-1, keepdim=True) * h.double(), dtype)
