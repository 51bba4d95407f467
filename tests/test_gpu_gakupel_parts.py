"""Each mechanism of the Gakupel design alone: the kernel against the plain function of tests/plain_gakupel.py, in 32-bit and
in bfloat16, at sizes the vectorised paths take and at sizes they do not, with inputs made so that a fault shows (one key far
back whose score stands out, a bias that changes within a page, a state a closed gate must forget, choices of both signs)."""
import math
from types import SimpleNamespace

import pytest
import torch

import plain_gakupel as plain

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
TOL = {torch.float32: 2e-5, torch.bfloat16: 1.2e-2}
F = torch.float64


def rnd(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


def close(got, want, dtype, what="", tol=None):
    got, want = got.double().cpu(), want.double()
    err, ref = float((got - want).abs().max()), float(want.abs().max())
    assert got.shape == want.shape and torch.isfinite(got).all(), what
    assert err <= (tol or TOL[dtype]) * ref, f"{what}: {err:.3e} > {tol or TOL[dtype]:.0e} * {ref:.3e}"


def i32(values):
    return torch.tensor(list(values), dtype=torch.int32, device=DEV)


def batch_of(lengths, ctx=None, slots=None):
    """What the kernels read of a step: requests of `lengths` rows each, after `ctx` cached tokens."""
    ctx = ctx or [0] * len(lengths)
    starts = [sum(lengths[:r]) for r in range(len(lengths))]
    return SimpleNamespace(n_requests=len(lengths), max_q_len=max(lengths), req_q_start=i32(starts), req_q_len=i32(lengths),
                           req_ctx_len=i32(ctx), req_state_slot=i32(slots or range(len(lengths))), h_q_len=list(lengths),
                           h_ctx_len=list(ctx), h_q_start=starts, extra={}, n_rows=sum(lengths),
                           row_request=i32(r for r, n in enumerate(lengths) for _ in range(n)),
                           positions=i32(c + i for c, n in zip(ctx, lengths) for i in range(n)),
                           max_pos=max(c + n for c, n in zip(ctx, lengths)) - 1)


def part(role, kind, params, dtype, tensors, **ctx):
    from hipinfer_b200.parts.registry import BuildContext, build_part
    from hipinfer_b200.parts.spec import PartSpec

    p = build_part(role, PartSpec(kind, params), BuildContext(dtype, DEV, **ctx))
    assert sorted(s.name for s in p.param_specs()) == sorted(tensors)
    for s in p.param_specs():
        assert tuple(s.shape) == tuple(tensors[s.name].shape), s.name
    p.load({n: t.to(DEV) for n, t in tensors.items()})
    return p


# ------------------------------------------------------------------------------------------ the norm on the result, the depth
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W", [50, 64, 176, 1000, 2048, 4096, 8192, 8196])
def test_norm_on_the_result_and_depth_average(dtype, W):
    """x + LN(y) (one result; two with constant scales; an RMS norm; without a bias), with the row as it came and the new row
    kept, and the average over the kept states; the rounded copy is the new x rounded once."""
    from hipinfer_b200.kernels import ops

    T, eps = 7, 1e-5
    x, y, z = rnd(T, W, seed=1) * 3, rnd(T, W, seed=2) * 0.3 + 2.0, rnd(T, W, seed=3) * 5
    w, b = (1 + 0.3 * rnd(W, seed=4)).to(dtype), (0.3 * rnd(W, seed=5)).to(dtype)
    x64, y64, w64, b64 = x.double(), y.double(), w.double(), b.double()
    pair64 = 0.65 * y64 - 1.4 * z.double()
    d = lambda t: None if t is None else t.to(DEV).clone()
    for what, res, want_res, bias, center in (("one", d(y), plain.layer_norm(y64, w64, b64, eps), b, True),
                                              ("two", ops.ScaledPair(d(y), d(z), 0.65, -1.4), plain.layer_norm(pair64, w64, b64, eps), b, True),
                                              ("rms", d(y), plain.rms(y64, eps) * w64, None, False)):
        xd, rounded = d(x), torch.empty(T, W, dtype=dtype, device=DEV)
        ops.output_norm(xd, res, d(w), d(bias), eps, rounded, center=center)
        close(xd, x64 + want_res, torch.float32, what)
        assert torch.equal(rounded, xd.to(dtype))
        for n in (1, 2, 7):
            states = rnd(n + 1, T, W, seed=6 + n)
            coef = rnd(n + 1, seed=20 + n)
            # the kept states are planes of one tensor; the new row becomes the next plane
            sd, xd = d(states), d(x)
            ops.output_norm(xd, res, d(w), d(bias), eps, rounded, None, sd[n], sd[:n], d(coef), center=center)
            want = plain.depth_average(list(states[:n].double()) + [x64 + want_res], coef.double())
            close(xd, want, torch.float32, f"{what}, average over {n + 1}")
            close(sd[n], x64 + want_res, torch.float32, "kept")
            assert torch.equal(sd[:n].cpu(), states[:n]) and torch.equal(rounded, xd.to(dtype))
            # the row as it came is the first state (a layer of one sublayer at the start)
            sd, xd = d(states), d(x)
            ops.output_norm(xd, res, d(w), d(bias), eps, None, sd[0], sd[n], sd[:n], d(coef), center=center)
            want = plain.depth_average([x64] + list(states[1:n].double()) + [x64 + want_res], coef.double())
            close(xd, want, torch.float32, f"{what}, first state")
            assert torch.equal(sd[0].cpu(), x)


# ------------------------------------------------------------------------------------------ norms, rotation, temperature
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,rot", [(6, 2, 64, 32), (3, 1, 10, 6), (4, 4, 32, 32), (2, 1, 128, 0), (9, 3, 80, 48)])
def test_head_norm_rotation_and_raw_keys_as_values(dtype, H, G, D, rot):
    """q and k: each head by its own root mean square, times a weight the heads share, then rotated (pairs (i, i + rot/2)); the
    values are the k columns as they are."""
    from hipinfer_b200.kernels import ops

    T, ps, eps, base = 11, 8, 1e-5, 5000.0
    proj = rnd(T, 3 + H * D + G * D, seed=1)
    proj[:, 3:3 + D] *= 6.0
    wq, wk = 1 + 0.3 * rnd(D, seed=2), 1 + 0.3 * rnd(D, seed=3)
    pos = torch.tensor([0, 1, 2, 3, 40, 41, 42, 500, 501, 7, 8])
    slots = torch.randperm(4 * ps, generator=torch.Generator().manual_seed(4))[:T].to(torch.int32)
    table = ops.shared_rope_table(rot, base, 600, DEV)
    q = torch.empty(T, H * D, dtype=dtype, device=DEV)
    kc, vc = (torch.zeros(4, G, ps, D, dtype=dtype, device=DEV) for _ in range(2))
    ops.rope_norm_store(proj.to(DEV), (3, 3 + H * D, 3 + H * D), pos.to(torch.int32).to(DEV), slots.to(DEV), table, rot, "half", False, 0.0,
                        q, kc, vc, H, G, D, D, ps, row_norm_eps=eps, head_norm=(wq.to(DEV), wk.to(DEV)))
    p64 = proj.double()
    raw = p64[:, 3 + H * D:].reshape(T, G, D)
    want_q = plain.rotate_half(plain.rms(p64[:, 3:3 + H * D].reshape(T, H, D), eps) * wq.double(), pos, rot, base)
    want_k = plain.rotate_half(plain.rms(raw, eps) * wk.double(), pos, rot, base)
    tol = None if dtype == torch.bfloat16 else 1e-4
    close(q.view(T, H, D), want_q, dtype, "q", tol)
    for t in range(T):
        page, off = int(slots[t]) // ps, int(slots[t]) % ps
        close(kc[page, :, off], want_k[t], dtype, "k", tol)
        close(vc[page, :, off], raw[t], dtype, "v")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("coef,every", [(0.35, 48), (1.0, 1), (-0.2, 7), (0.5, 2.5)])
def test_query_temperature_steps_with_the_position(dtype, coef, every):
    """The factor changes exactly where (p + 1) is a multiple of `every`; keys and values are not touched."""
    from hipinfer_b200.kernels import ops

    H, G, D, E, ps, eps = 2, 1, 16, 8, 16, 1e-6
    pos = [0, 1, 5, 6, 7, 13, 62, 63, 64, 126, 127, 128, 1000, 4095]
    T = len(pos)
    proj = rnd(T, H * D + G * D + G * E, seed=1)
    wq, wk = 1 + 0.3 * rnd(H * D, seed=2), 1 + 0.3 * rnd(G * D, seed=3)
    q = torch.empty(T, H * D, dtype=dtype, device=DEV)
    kc, vc = torch.zeros(1, G, ps, D, dtype=dtype, device=DEV), torch.zeros(1, G, ps, E, dtype=dtype, device=DEV)
    table = ops.shared_rope_table(0, 1.0, 5000, DEV)
    ops.rope_norm_store(proj.to(DEV), (0, H * D, H * D + G * D), i32(pos), i32(range(T)), table, 0, "half", False, 0.0, q, kc, vc, H, G, D,
                        E, ps, row_norm=(wq.to(DEV), wk.to(DEV)), row_norm_eps=eps, q_temp=(coef, every))
    temp = torch.tensor([1 + coef * math.log(math.floor((p + 1) / every) + 1) for p in pos], dtype=F)
    close(q, plain.rms(proj[:, :H * D].double(), eps) * wq.double() * temp[:, None], dtype, "q")
    close(kc[0, 0, :T], plain.rms(proj[:, H * D:H * D + D].double(), eps) * wk.double(), dtype, "k")
    close(vc[0, 0, :T], proj[:, H * D + D:].double(), dtype, "v")


# ------------------------------------------------------------------------------------------ attention
def _paged(k, v, ps, dtype, seed):
    """Keys and values [n, G, D] in pages in a random order; (k cache, v cache, table)."""
    n, G, D = k.shape
    pages = -(-n // ps)
    order = torch.randperm(pages + 3, generator=torch.Generator().manual_seed(seed))[:pages]
    kc, vc = torch.zeros(pages + 3, G, ps, D), torch.zeros(pages + 3, G, ps, v.shape[-1])
    for j in range(n):
        kc[order[j // ps], :, j % ps], vc[order[j // ps], :, j % ps] = k[j], v[j]
    return kc.to(dtype).to(DEV), vc.to(dtype).to(DEV), order.to(torch.int32)


def _attention_case(dtype, H, G, D, E, ps, bias, one, lengths, ctx, r1, r2):
    """(q, caches, batch, wanted): requests of `lengths` rows after `ctx` cached tokens. One key far back in each request has a
    score that stands out for its last row, so that a lost or shifted key shows."""
    scale = D ** -0.5
    qs, caches, tables, want = [], [], [], []
    for i, (n, c) in enumerate(zip(lengths, ctx)):
        tot = n + c
        q, k, v = rnd(n, H, D, seed=10 + i), rnd(tot, G, D, seed=30 + i), rnd(tot, G, E, seed=50 + i)
        far = max(0, tot // 3 - 1)
        k[far] = 3.0 * k[far]
        q[-1] = 2.5 * k[far].repeat_interleave(H // G, 0)
        q, k, v = (t.to(dtype).float() for t in (q, k, v))
        out = torch.zeros(n, H, E, dtype=F)
        for h in range(H):
            g = h // (H // G)
            s = q[:, h].double() @ k[:, g].double().T * scale
            dist = (torch.arange(c, tot)[:, None] - torch.arange(tot)[None, :])
            if bias:
                s = s - r1[h].double() * torch.log(1 + r2[h].double() * dist.clamp(min=0))
            s = s.masked_fill(dist < 0, float("-inf"))
            m = s.amax(-1, keepdim=True).clamp(min=0) if one else s.amax(-1, keepdim=True)
            e = torch.exp(s - m)
            out[:, h] = e @ v[:, g].double() / (e.sum(-1, keepdim=True) + (torch.exp(-m) if one else 0.0))
        want.append(out.reshape(n, H * E))
        qs.append(q.reshape(n, H * D))
        caches.append((k, v))
    base, kcs, vcs = 0, [], []
    width = max(-(-(n + c) // ps) for n, c in zip(lengths, ctx))
    for i, (k, v) in enumerate(caches):
        kc, vc, order = _paged(k, v, ps, dtype, i)
        row = torch.full((width,), -1, dtype=torch.int32)
        row[:order.numel()] = order + base
        tables.append(row)
        kcs.append(kc)
        vcs.append(vc)
        base += kc.shape[0]
    batch = batch_of(lengths, ctx)
    batch.block_tables = [torch.stack(tables).to(DEV)]
    return torch.cat(qs).to(dtype).to(DEV), torch.cat(kcs), torch.cat(vcs), batch, torch.cat(want)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,E,ps", [(4, 2, 64, 64, 16), (8, 2, 96, 32, 16), (3, 1, 10, 6, 8), (20, 1, 32, 32, 16), (4, 4, 128, 64, 32),
                                        (6, 2, 96, 96, 16), (2, 2, 48, 80, 16), (8, 2, 128, 128, 16), (1, 1, 64, 64, 64)])
@pytest.mark.parametrize("bias,one", [(True, True), (False, False), (True, False), (False, True)])
def test_attention_with_distance_bias_and_constant_sink(dtype, H, G, D, E, ps, bias, one):
    """Unequal portions (single rows, a few rows, more than a flash tile, after cached tokens that end at and around page
    borders); the bias falls steeply over the first keys, so that a distance that is off by one shows. The tensor-core
    kernels, the warp-MMA kernels and the plain one."""
    from hipinfer_b200.kernels import ops

    r1, r2 = 0.4 + rnd(H, seed=1).abs(), 0.2 + rnd(H, seed=2).abs()
    q, kc, vc, batch, want = _attention_case(dtype, H, G, D, E, ps, bias, one, [1, 1, 5, 150, 70, 1, 16], [0, 333, 64, 0, 129, 64, 15], r1, r2)
    kw = dict(sink=torch.zeros(H, device=DEV) if one else None, distance=ops.DistanceBias(r1.to(DEV), r2.to(DEV)) if bias else None)
    plains = (False, True) if dtype == torch.bfloat16 else (False,)
    for force_rows, force_plain in [(False, p) for p in plains] + ([(True, False)] if dtype == torch.bfloat16 else []):
        att = torch.full(want.shape, float("nan"), dtype=dtype, device=DEV)
        ops.attention_masked(q, kc, vc, batch, 0, att, H, G, D, E, ps, D ** -0.5, force_rows=force_rows, force_plain=force_plain, **kw)
        close(att, want, dtype, f"rows {force_rows} plain {force_plain}", 5e-5 if dtype == torch.float32 else None)


@pytest.mark.parametrize("D,G,H", [(64, 2, 8), (64, 1, 3), (128, 2, 8), (128, 1, 1)])
@pytest.mark.parametrize("rows", [2, 12, 40])
@pytest.mark.parametrize("steep", [False, True])
def test_single_rows_far_into_their_sequences(D, G, H, rows, steep):
    """Decode steps of few and of many rows at unequal positions up to 1,300, at and around the key splits' edges, and portions
    beside them. steep: a bias that falls by hundreds within a tile (the kernels that bound a tile's maximum by its nearest
    key leave such a one to the others)."""
    from hipinfer_b200.kernels import ops

    ctx = ([0, 1299, 255, 256, 511, 512, 513, 767, 1023, 1024, 63, 64] + list(range(100, 1300, 43)))[:rows]
    r1, r2 = (30.0 if steep else 0.3) + rnd(H, seed=1).abs(), 0.2 + rnd(H, seed=2).abs()
    dist = ops.DistanceBias(r1.to(DEV), r2.to(DEV))
    assert (dist.spread > 60) == steep
    sink = torch.zeros(H, device=DEV)
    for lengths, c in (([1] * rows, ctx), ([1] * (rows - 1) + [300], ctx[:-1] + [777])):
        q, kc, vc, batch, want = _attention_case(torch.bfloat16, H, G, D, D, 16, True, True, lengths, c, r1, r2)
        att = torch.full(want.shape, float("nan"), dtype=torch.bfloat16, device=DEV)
        ops.attention_masked(q, kc, vc, batch, 0, att, H, G, D, D, 16, D ** -0.5, sink=sink, distance=dist)
        close(att, want, torch.bfloat16, f"{lengths[-1]}")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_sink_takes_the_weight_where_scores_are_low(dtype):
    """Scores far below zero: with one in the denominator the result is nearly nothing; a softmax without it is not."""
    from hipinfer_b200.kernels import ops

    H = G = 1
    D = E = 64
    n = 40
    k, v = rnd(n, 1, D, seed=1), 1 + rnd(n, 1, E, seed=2)
    k[..., 0] = 8.0
    q = torch.zeros(n, 1, D)
    q[..., 0] = -1.0
    q, k, v = (t.to(dtype).float() for t in (q, k, v))
    batch = batch_of([n])
    kc, vc, order = _paged(k, v, 16, dtype, 3)
    batch.block_tables = [order[None].to(DEV)]
    s = plain.causal_softmax(q[:, 0].double() @ k[:, 0].double().T, True) @ v[:, 0].double()
    att = torch.empty(n, E, dtype=dtype, device=DEV)
    ops.attention_masked(q.reshape(n, D).to(dtype).to(DEV), kc, vc, batch, 0, att, 1, 1, D, E, 16, 1.0, sink=torch.zeros(1, device=DEV))
    close(att, s, dtype)
    ops.attention_masked(q.reshape(n, D).to(dtype).to(DEV), kc, vc, batch, 0, att, 1, 1, D, E, 16, 1.0)
    assert float(att.float().abs().min(-1).values.max()) > 5 * float(s.abs().max())


def _attention_part(params, tensors, m, cfg_fn, h, cuts, dtype, sub=""):
    """A masked_attention part over one sequence cut into `cuts`, against the plain function on the whole."""
    from hipinfer_b200.cache.storage import LayerCache

    T, W = h.shape
    p = part("mixer", "masked_attention", params, dtype, tensors, page_size=16, max_model_len=T)
    need = p.cache_need()
    pages = -(-T // 16)
    planes = {n: torch.zeros(pages, heads, 16, width, dtype=dtype, device=DEV) for n, heads, width in need.planes}
    perm = torch.randperm(pages, generator=torch.Generator().manual_seed(9)).to(torch.int32)
    got, at = [], 0
    for n in cuts:
        b = batch_of([n], [at])
        b.block_tables = [perm[None].to(DEV)]
        b.slot_maps = [i32(int(perm[j // 16]) * 16 + j % 16 for j in range(at, at + n))]
        x = torch.zeros(n, W, dtype=torch.float32, device=DEV)
        p.forward(h[at:at + n].to(dtype).to(DEV), x, b, LayerCache(planes, 0, True), {})
        got.append(x.cpu())
        at += n
    close(torch.cat(got), cfg_fn({k.split("mix.", 1)[1]: v.double() for k, v in tensors.items()}, h.double()), dtype,
          tol=4e-5 if dtype == torch.float32 else 2e-2)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,rot", [(4, 2, 64, 32), (6, 2, 16, 16), (3, 3, 10, 0), (4, 1, 128, 64)])
@pytest.mark.parametrize("cuts", [(180,), (1,) * 20, (33, 2, 1, 64, 17, 63)])
def test_attention_part_with_keys_as_values(dtype, H, G, D, rot, cuts):
    W, T = 48, sum(cuts)
    m = dict(heads=H, kv_heads=G, dim=D, vdim=D, scale=D ** -0.5, rot=dict(base=1000.0, dims=rot))
    t = {"mix.q": rnd(H * D, W, seed=1, scale=0.2), "mix.k": rnd(G * D, W, seed=2, scale=0.2), "mix.q.norm": 1 + 0.3 * rnd(D, seed=3),
         "mix.k.norm": 1 + 0.3 * rnd(D, seed=4), "mix.o": rnd(W, H * D, seed=5, scale=0.1)}
    t = {n: v.to(dtype).float() if dtype == torch.bfloat16 else v for n, v in t.items()}
    h = rnd(T, W, seed=6).to(dtype).float()
    params = dict(hidden_size=W, heads=H, kv_heads=G, dim=D, vdim=D, scale=m["scale"], eps=1e-5, rot_dims=rot, rot_base=1000.0,
                  pairing="half", head_norm=True, values="keys")
    _attention_part(params, {n: v.to(dtype) for n, v in t.items()}, m, lambda w, h64: plain.shared_key_attention(h64, w, m, 1e-5), h, cuts, dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,E,temp", [(4, 2, 64, 64, (0.5, 16)), (6, 2, 16, 24, None), (3, 1, 10, 6, (1.0, 3)), (4, 4, 80, 48, (0.35, 48))])
@pytest.mark.parametrize("cuts", [(180,), (1,) * 20, (33, 2, 1, 64, 17, 63)])
def test_attention_part_with_distance_bias_and_temperature(dtype, H, G, D, E, temp, cuts):
    W, T = 48, sum(cuts)
    m = dict(heads=H, kv_heads=G, dim=D, vdim=E, scale=D ** -0.5)
    if temp:
        m["q_temp"] = dict(coef=temp[0], every=temp[1])
    t = {"mix.q": rnd(H * D, W, seed=1, scale=0.2), "mix.k": rnd(G * D, W, seed=2, scale=0.2), "mix.v": rnd(G * E, W, seed=7, scale=0.2),
         "mix.q.norm": 1 + 0.3 * rnd(H * D, seed=3), "mix.k.norm": 1 + 0.3 * rnd(G * D, seed=4), "mix.r1": 0.3 + rnd(H, seed=8).abs(),
         "mix.r2": 0.1 + rnd(H, seed=9).abs(), "mix.o": rnd(W, H * E, seed=5, scale=0.1)}
    t = {n: v.to(dtype) for n, v in t.items()}
    h = rnd(T, W, seed=6).to(dtype).float()
    params = dict(hidden_size=W, heads=H, kv_heads=G, dim=D, vdim=E, scale=m["scale"], eps=1e-5, rot_dims=0, row_norm=True, q_temp=temp,
                  distance_bias=True, sink="one")
    _attention_part(params, t, m, lambda w, h64: plain.distance_attention(h64, w, m, 1e-5), h, cuts, dtype)


# ------------------------------------------------------------------------------------------ recurrences
@pytest.mark.parametrize("H,G,N,P", [(4, 2, 64, 64), (2, 2, 32, 128), (3, 1, 7, 10), (2, 1, 128, 96), (2, 2, 48, 48), (1, 1, 256, 40), (2, 2, 70, 6),
                                     (1, 1, 500, 12), (1, 1, 600, 12)])
@pytest.mark.parametrize("kind", ["linear", "linear in pieces", "delta"])
def test_walk_over_unequal_requests_and_portions(H, G, N, P, kind, monkeypatch):
    """Requests of 1 to 90 tokens in one launch, each continued by a second portion and then by single tokens, from slots in
    another order than the requests; decays from 1 (nothing forgotten) to 0 (everything)."""
    from hipinfer_b200.kernels import ops

    monkeypatch.setattr(ops, "MS_PIECE_TOKENS", 8 if kind == "linear in pieces" else 0)
    delta = kind == "delta"
    portions = [[1, 37, 90, 16], [5, 40, 33, 17], [1, 1, 1, 1], [1, 1, 1, 1], [2, 3, 7, 6]]
    slots = [2, 0, 4, 1]
    lens = [sum(p[r] for p in portions) for r in range(4)]
    state = torch.full((5, H, N, P), 7.0, device=DEV)
    nstate = torch.full((5, H, N), 7.0, device=DEV)
    state[slots], nstate[slots] = 0.0, 0.0
    q, k, v, a, b, za, zb = [], [], [], [], [], [], []
    for r, n in enumerate(lens):
        q.append(rnd(n, G, N, seed=r))
        k.append(rnd(n, G, N, seed=10 + r))
        if delta:
            k[-1][n // 2:] = 0.3 * k[-1][n // 2:] + rnd(1, G, N, seed=40 + r)       # keys that overlap
        v.append(rnd(n, H, P, seed=20 + r))
        g = torch.Generator().manual_seed(30 + r)
        dec = torch.rand(n, H, generator=g) ** 0.2
        dec[torch.rand(n, H, generator=g) < 0.05] = 0.0
        dec[torch.rand(n, H, generator=g) < 0.2] = 1.0
        a.append(dec)
        b.append(torch.rand(n, H, generator=g))
        za.append(torch.log(torch.expm1(-torch.log(dec.double().clamp(1e-30, 1 - 1e-9)))).float())   # softplus(za) = -log of the decay
        zb.append(torch.logit(b[-1].double()).float())
    at, scale = [0] * 4, 0.37
    ys, nqs = [[] for _ in lens], [[] for _ in lens]
    zero = torch.zeros(H, device=DEV)
    for p in portions:
        sel = lambda t: torch.cat([t[r][at[r]:at[r] + p[r]] for r in range(4)]).float()
        T = sum(p)
        # q, k, v as columns of wider rows
        rows = torch.cat([sel(q).reshape(T, -1), sel(k).reshape(T, -1), sel(v).reshape(T, -1)], 1).to(DEV)
        qd, kd, vd = torch.split(rows, [G * N, G * N, H * P], 1)
        y, nq, batch = torch.empty(T, H * P, device=DEV), torch.empty(T, H, device=DEV), batch_of(p, at, slots)
        if delta:
            z = torch.cat([sel(za), sel(zb)], 1).to(DEV)
            scal = ops.ms_delta_prepare(qd, kd, z[:, :H], z[:, H:], zero, zero, batch, N, scale, 1e-6)
            ops.ms_delta_walk(qd, kd, vd, scal, state, batch, y)
        else:
            ops.ms_walk(qd, kd, vd, sel(a).contiguous().to(DEV), sel(b).contiguous().to(DEV), state, batch, y, scale, nstate, nq)
        o = 0
        for r in range(4):
            ys[r].append(y[o:o + p[r]].cpu())
            nqs[r].append(nq[o:o + p[r]].cpu())
            o += p[r]
            at[r] += p[r]
    assert bool((state[3] == 7.0).all()) and bool((nstate[3] == 7.0).all()), "a slot no request owns was written"
    for r, n in enumerate(lens):
        rep = lambda t: t.double().repeat_interleave(H // G, 1)
        if delta:
            A = torch.exp(-plain.softplus(za[r].double()))
            want = plain.gated_delta(plain.unit(rep(q[r])), plain.unit(rep(k[r])), v[r].double(), A, torch.sigmoid(zb[r].double()))
        else:
            S, nn = torch.zeros(H, N, P, dtype=F), torch.zeros(H, N, dtype=F)
            want, wn = torch.zeros(n, H, P, dtype=F), torch.zeros(n, H, dtype=F)
            Q, K, V, A, B = rep(q[r]), rep(k[r]), v[r].double(), a[r].double(), b[r].double()
            for t in range(n):
                S = A[t][:, None, None] * S + B[t][:, None, None] * K[t][:, :, None] * V[t][:, None, :]
                nn = A[t][:, None] * nn + B[t][:, None] * K[t]
                want[t], wn[t] = torch.einsum("hnp,hn->hp", S, Q[t]), (nn * Q[t]).sum(-1)
            close(torch.cat(nqs[r]), wn * scale, torch.float32, f"n . q of request {r}", 1e-4)
            close(state[slots[r]], S, torch.float32, "state")
        close(torch.cat(ys[r]).reshape(n, H, P), want * scale, torch.float32, f"request {r}", 1e-4)


def test_linear_walk_gives_the_same_bits_however_it_is_cut():
    from hipinfer_b200.kernels import ops

    H, N, P, n = 2, 64, 64, 100
    q, k, v = rnd(n, H * N, seed=1).to(DEV), rnd(n, H * N, seed=2).to(DEV), rnd(n, H * P, seed=3).to(DEV)
    a, b = torch.rand(n, H, generator=torch.Generator().manual_seed(4)).to(DEV) ** 0.1, torch.rand(n, H).to(DEV)
    res = []
    for cuts in ((100,), (1, 50, 16, 33), (3,) * 33 + (1,)):
        state, ns, at, ys = torch.zeros(1, H, N, P, device=DEV), torch.zeros(1, H, N, device=DEV), 0, []
        for c in cuts:
            y, nq, s = torch.empty(c, H * P, device=DEV), torch.empty(c, H, device=DEV), slice(at, at + c)
            ops.ms_walk(q[s], k[s], v[s], a[s].contiguous(), b[s].contiguous(), state, batch_of([c], [at]), y, 1.0, ns, nq)
            ys.append(y)
            at += c
        res.append((torch.cat(ys), state))
    assert all(torch.equal(res[0][0], r[0]) and torch.equal(res[0][1], r[1]) for r in res[1:])


@pytest.mark.parametrize("n", [1, 2, 31, 32, 33, 700, 1024, 1025, 2100])
@pytest.mark.parametrize("cap", [15.0, 1.0, 60.0])
def test_exponential_gates_and_their_running_maximum(n, cap):
    """a and b against the recurrence of m token by token, in one launch and in portions; the maximum starts at zero."""
    from hipinfer_b200.kernels import ops

    H = 3
    zi, zf = rnd(n, H, seed=1, scale=6.0), rnd(n, H, seed=2, scale=6.0)
    bi, bf = rnd(H, seed=3), 2 + rnd(H, seed=4)
    li, lf = plain.log_gates(torch.cat([zi, zf], 1).double(), {"i": torch.cat([torch.eye(H), torch.zeros(H, H)], 1).double(), "i.b": bi.double(),
                             "f": torch.cat([torch.zeros(H, H), torch.eye(H)], 1).double(), "f.b": bf.double()}, cap)
    m, A, B, E = torch.zeros(H, dtype=F), [], [], []
    for t in range(n):
        new = torch.maximum(lf[t] + m, li[t])
        A.append(torch.exp(lf[t] + m - new))
        B.append(torch.exp(li[t] - new))
        E.append(torch.exp(-new))
        m = new
    rows = torch.cat([zi, zf], 1).to(DEV)
    for cuts in ((n,), tuple([max(1, n // 3)] * (n // max(1, n // 3)) + ([n % max(1, n // 3)] if n % max(1, n // 3) else []))):
        ms, at, got = torch.zeros(2, H, device=DEV), 0, []
        for c in cuts:
            r = rows[at:at + c]
            got.append(ops.ms_exp_gates(r[:, :H], r[:, H:], bi.to(DEV), bf.to(DEV), cap, ms, batch_of([c], [at], [1])))
            at += c
        # the values lie within a factor of 1 + 1e-5 (or, where they vanish, within 1e-7)
        for got_t, want in zip(zip(*got), (A, B, E)):
            g, w = torch.cat(got_t).double().cpu(), torch.stack(want)
            assert float(((g - w).abs() / (w + 1e-2)).max()) < 2e-4
        assert float((ms[1].double().cpu() - m).abs().max()) < 1e-3 and bool((ms[0] == 0).all())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,N", [(4, 2, 64), (3, 3, 10), (6, 1, 130), (20, 10, 16)])
def test_unit_queries_and_keys_decay_and_write_strength(dtype, H, G, N):
    """The numbers of every token; the products with earlier tokens stop at the start of a request's portion."""
    from hipinfer_b200.kernels import ops

    lengths = [2, 1, 6]
    T = sum(lengths)
    qkv = rnd(T, 5 + 2 * G * N, seed=1)
    qkv[0] = 0.0                                                            # nothing to normalise: stays zero
    qkv[1] *= 1e-4                                                          # the constant under the root matters
    z = rnd(T, 2 * H, seed=2, scale=3.0)
    a_log, bias = (rnd(H, seed=3)).to(dtype), rnd(H, seed=4).to(dtype)
    rows, zd = qkv.to(DEV), z.to(DEV)
    qd, kd = rows[:, 5:5 + G * N], rows[:, 5 + G * N:]
    scal = ops.ms_delta_prepare(qd, kd, zd[:, :H], zd[:, H:], a_log.to(DEV), bias.to(DEV), batch_of(lengths), N, 0.25, 1e-6).cpu().double()
    raw_q, raw_k = (qkv[:, o:o + G * N].double().reshape(T, G, N) for o in (5, 5 + G * N))
    q, k = plain.unit(raw_q) * 0.25, plain.unit(raw_k)
    want = torch.zeros(T, H, 12, dtype=F)
    start = [sum(lengths[:i]) for i, n in enumerate(lengths) for _ in range(n)]
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            want[t, h, 0] = torch.exp(-torch.exp(a_log[h].double()) * plain.softplus(z[t, h].double() + bias[h].double()))
            want[t, h, 1] = torch.sigmoid(z[t, H + h].double())
            want[t, h, 2] = 1 / torch.sqrt((raw_k[t, g] ** 2).sum() + 1e-6)
            want[t, h, 3] = 0.25 / torch.sqrt((raw_q[t, g] ** 2).sum() + 1e-6)
            for i in range(4):
                if t - i >= start[t]:
                    if i:
                        want[t, h, 3 + i] = k[t, g] @ k[t - i, g]
                    want[t, h, 7 + i] = q[t, g] @ k[t - i, g]
    for i in range(12):
        if float(want[..., i].abs().max()) > 0:
            close(scal[..., i], want[..., i], torch.float32, f"number {i}", 5e-5)
        else:
            assert float(scal[..., i].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,P", [(4, 64), (2, 128), (3, 10), (1, 6), (2, 48), (5, 256)])
@pytest.mark.parametrize("shared,kind", [(True, "silu"), (False, "sigmoid")])
def test_head_norm_weight_and_gate(dtype, H, P, shared, kind):
    from hipinfer_b200.kernels import ops

    T, eps = 13, 1e-4
    y, gate = rnd(T, H * P, seed=1), rnd(T, 2 + H * P, seed=2, scale=2.0)
    y[3] *= 1e-3
    w = (1 + 0.3 * rnd(P if shared else H * P, seed=3)).to(dtype)
    nq, e = rnd(T, H, seed=4), rnd(T, H, seed=5).abs() * 0.5
    g64 = gate[:, 2:].double()
    act = plain.silu(g64) if kind == "silu" else torch.sigmoid(g64)
    w64 = (w.double().repeat(H) if shared else w.double())
    for norm in (False, True):
        o = y.double().reshape(T, H, P)
        if norm:
            o = o / (torch.maximum(nq.double().abs(), e.double()) + 1e-6)[..., None]
        want = plain.rms(o, eps).reshape(T, H * P) * w64 * act
        out = torch.empty(T, H * P, dtype=dtype, device=DEV)
        kw = dict(nq=nq.to(DEV), floor=e.to(DEV), den_eps=1e-6) if norm else {}
        ops.ms_finish(y.to(DEV), w.to(DEV), gate.to(DEV)[:, 2:], kind, out, H, eps, **kw)
        close(out, want, dtype)


def _run_mixer(p, h, plan, dtype, W):
    """A recurrent mixer over the sequences h (one per request) by `plan` (steps of (request, tokens))."""
    state = {n: torch.zeros((len(h),) + tuple(s), dtype=dt, device=DEV) for n, (s, dt) in p.state_need().items()}
    at, got = [0] * len(h), [[] for _ in h]
    for step in plan:
        rows = torch.cat([h[r][at[r]:at[r] + n] for r, n in step])
        b = batch_of([n for _, n in step], [at[r] for r, _ in step], [r for r, _ in step])
        x = torch.zeros(rows.shape[0], W, dtype=torch.float32, device=DEV)
        p.forward(rows.to(dtype).to(DEV), x, b, None, state)
        o = 0
        for r, n in step:
            got[r].append(x[o:o + n].cpu())
            o += n
            at[r] += n
    return [torch.cat(g) for g in got]


PLANS = {"whole": [[(0, 90)], [(1, 250)]], "token by token": [[(0, 1), (1, 1)]] * 90 + [[(1, 1)]] * 160,
         "portions": [[(0, 2), (1, 100)], [(0, 1), (1, 2)], [(1, 3)], [(0, 64), (1, 1)], [(0, 23), (1, 144)]]}


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,D,P,cap", [(4, 64, 64, 15.0), (3, 10, 6, 5.0), (2, 96, 32, 30.0), (2, 128, 128, 15.0)])
@pytest.mark.parametrize("plan", sorted(PLANS))
def test_matrix_memory_part(dtype, H, D, P, cap, plan):
    W = 64
    t = {"mix.q": rnd(H * D, W, seed=1, scale=0.15), "mix.k": rnd(H * D, W, seed=2, scale=0.15), "mix.v": rnd(H * P, W, seed=3, scale=0.15),
         "mix.g": rnd(H * P, W, seed=4, scale=0.15), "mix.i": rnd(H, W, seed=5, scale=0.4), "mix.i.b": rnd(H, seed=6),
         "mix.f": rnd(H, W, seed=7, scale=0.4), "mix.f.b": 3 + rnd(H, seed=8), "mix.norm": 1 + 0.3 * rnd(H * P, seed=9),
         "mix.o": rnd(W, H * P, seed=10, scale=0.1)}
    t = {n: v.to(dtype) for n, v in t.items()}
    p = part("mixer", "matrix_memory", dict(hidden_size=W, heads=H, dim=D, vdim=P, gate_cap=cap, eps=1e-5), dtype, t)
    h = [rnd(n, W, seed=20 + n).to(dtype).float() for n in (90, 250)]
    w = {n.split("mix.")[1]: v.double() for n, v in t.items()}
    for got, hh in zip(_run_mixer(p, h, PLANS[plan], dtype, W), h):
        close(got, plain.memory_mixer(hh.double(), w, dict(heads=H, dim=D, vdim=P, gate_cap=cap), 1e-5), dtype, tol=1e-4 if dtype == torch.float32 else 2e-2)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,P,taps", [(4, 2, 64, 64, 4), (3, 1, 10, 6, 1), (2, 2, 32, 96, 7), (2, 1, 128, 128, 3)])
@pytest.mark.parametrize("plan", sorted(PLANS))
def test_gated_delta_part(dtype, H, G, D, P, taps, plan):
    W = 64
    t = {"mix.q": rnd(G * D, W, seed=1, scale=0.15), "mix.k": rnd(G * D, W, seed=2, scale=0.15), "mix.v": rnd(H * P, W, seed=3, scale=0.15),
         "mix.q.conv": rnd(G * D, taps, seed=4, scale=0.6), "mix.k.conv": rnd(G * D, taps, seed=5, scale=0.6),
         "mix.v.conv": rnd(H * P, taps, seed=6, scale=0.6), "mix.b": rnd(H, W, seed=7, scale=0.2), "mix.a": rnd(H, W, seed=8, scale=0.2),
         "mix.dt_bias": rnd(H, seed=9) - 2, "mix.A_log": rnd(H, seed=10), "mix.g": rnd(H * P, W, seed=11, scale=0.15),
         "mix.norm": 1 + 0.3 * rnd(P, seed=12), "mix.o": rnd(W, H * P, seed=13, scale=0.1)}
    t = {n: v.to(dtype) for n, v in t.items()}
    p = part("mixer", "gated_delta", dict(hidden_size=W, heads=H, kv_heads=G, dim=D, vdim=P, conv=taps, eps=1e-5), dtype, t)
    h = [rnd(n, W, seed=20 + n).to(dtype).float() for n in (90, 250)]
    w = {n.split("mix.")[1]: v.double() for n, v in t.items()}
    for got, hh in zip(_run_mixer(p, h, PLANS[plan], dtype, W), h):
        close(got, plain.delta_mixer(hh.double(), w, dict(heads=H, kv_heads=G, dim=D, vdim=P), 1e-5), dtype, tol=1e-4 if dtype == torch.float32 else 2e-2)


# ------------------------------------------------------------------------------------------ feed-forwards
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W,ff", [(64, 96), (50, 30), (128, 320), (256, 1024)])
@pytest.mark.parametrize("T", [1, 7, 40, 64, 65, 300])
def test_dense_feed_forward_with_the_exact_gelu(dtype, W, ff, T):
    up, down, h = rnd(ff, W, seed=1, scale=2.0 / math.sqrt(W)).to(dtype), rnd(W, ff, seed=2, scale=1 / math.sqrt(ff)).to(dtype), rnd(T, W, seed=3).to(dtype)
    p = part("feed_forward", "activated", dict(hidden_size=W, intermediate_size=ff), dtype, {"mlp.up": up, "mlp.down": down})
    x = torch.zeros(T, W, device=DEV)
    p.forward(h.to(DEV), x, None)
    close(x, plain.dense(h.double(), {"up": up.double(), "down": down.double()}), dtype)


def test_exact_gelu_is_not_the_tanh_form():
    """The two forms differ by up to 5e-4; the 32-bit result must be the exact one."""
    from hipinfer_b200.kernels import ops

    z = torch.linspace(-6, 6, 2001)[None].contiguous()
    out = torch.empty_like(z, device=DEV)
    ops.bias_act(z.to(DEV), None, out, "gelu")
    exact = plain.gelu(z.double())
    tanh = 0.5 * z.double() * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z.double() + 0.044715 * z.double() ** 3)))
    assert float((out.double().cpu() - exact).abs().max()) < 1e-6 < 1e-4 < float((exact - tanh).abs().max())


ROUTERS = [dict(experts=15, top=4, groups=dict(count=5, keep=3), scale=1.3), dict(experts=16, top=2, groups=dict(count=8, keep=1), scale=0.7),
           dict(experts=5, top=2, scale=2.5), dict(experts=1, top=1), dict(experts=9, top=3, groups=dict(count=3, keep=2), scale=1.0),
           dict(experts=8, top=3, groups=dict(count=8, keep=4), scale=1.0), dict(experts=6, top=6, groups=dict(count=2, keep=2), scale=3.0)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("r", ROUTERS, ids=lambda r: f"{r['experts']}-{r['top']}-{(r.get('groups') or {}).get('count', 1)}")
@pytest.mark.parametrize("W", [64, 50, 2048])
def test_grouped_router(dtype, r, W):
    """Corrections of both signs move the choice but not the weights; groups that rank low lose even their best expert; choice
    scores below zero are still chosen. Rows whose call is close are left out."""
    from hipinfer_b200.kernels import ops

    T, E, top = 400, r["experts"], r["top"]
    h, router = rnd(T, W, seed=1).to(dtype), rnd(E, W, seed=2, scale=1.5 / math.sqrt(W)).to(dtype)
    corr, sg = (rnd(E, seed=3) * 0.5 - 0.7).to(dtype), rnd(1, W, seed=4, scale=1 / math.sqrt(W)).to(dtype)
    g = r.get("groups") or dict(count=1, keep=1)
    sw = torch.empty(T, device=DEV)
    expert, weight = ops.moe_route(h.to(DEV), router.to(DEV), top, None, "sigmoid_normed", corr.to(DEV), g["count"], g["keep"],
                                   r.get("scale", 1.0), sg.to(DEV), sw)
    chosen, want = plain.route(h.double(), router.double(), corr.double(), r)
    s = torch.sigmoid(h.double() @ router.double().T)
    c = s + corr.double()
    assert float(c.min()) < 0 or E < 5
    # how close the calls are: between the last group kept and the first dropped, between the last expert chosen and the next
    per = torch.sort(c.reshape(T, g["count"], -1), dim=-1, descending=True).values[..., :2].sum(-1)
    ordered = torch.sort(per, dim=-1, descending=True)
    margin = torch.full((T,), 1.0, dtype=F)
    if g["keep"] < g["count"]:
        margin = torch.minimum(margin, ordered.values[:, g["keep"] - 1] - ordered.values[:, g["keep"]])
    stay = torch.zeros(T, g["count"], dtype=torch.bool).scatter_(1, ordered.indices[:, :g["keep"]], True)
    left = torch.sort(c.masked_fill(~stay.repeat_interleave(E // g["count"], 1), -9.0), dim=-1, descending=True).values
    margin = torch.minimum(margin, (left[:, :top] - torch.cat([left, torch.full((T, 1), -10.0, dtype=F)], 1)[:, 1:top + 1]).min(-1).values)
    sure = margin > 1e-4
    assert int(sure.sum()) > T // 2
    assert torch.equal(expert.cpu().long()[sure], chosen[sure])
    close(weight.cpu()[sure], want[sure], torch.float32)
    close(sw, torch.sigmoid(h.double() @ sg.double()[0]), torch.float32)
    if g["keep"] < g["count"] and E > g["count"]:            # groups of one decide nothing that the experts do not
        ungrouped = torch.sort(c, dim=-1, descending=True).indices[:, :top]
        assert float((ungrouped.sort(-1).values != chosen.sort(-1).values).any(-1).double().mean()) > 0.05, "the groups decide nothing: not tested"


def test_router_ties_go_to_the_lower_index():
    from hipinfer_b200.kernels import ops

    h, router, corr = torch.ones(1, 16, device=DEV), torch.zeros(8, 16, device=DEV), torch.zeros(8, device=DEV)
    expert, weight = ops.moe_route(h, router, 3, None, "sigmoid_normed", corr, 4, 2, 1.0)
    assert expert.tolist() == [[0, 1, 2]] and float((weight - 1 / 3).abs().max()) < 1e-6


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W,Fe,Fs,r", [(64, 32, 48, ROUTERS[0]), (50, 10, 6, ROUTERS[2]), (128, 96, None, ROUTERS[4]), (96, 40, 200, ROUTERS[3])])
@pytest.mark.parametrize("T,prompt", [(1, False), (3, False), (8, False), (9, False), (40, False), (70, True), (200, True)])
def test_experts_with_a_gated_shared_expert(dtype, W, Fe, Fs, r, T, prompt):
    """The three ways a step runs the experts and the two ways it runs the shared one. Every token's code sits in the first
    channels, so that no call is close."""
    E, top = r["experts"], r["top"]
    g = r.get("groups")
    t = {"mlp.router": torch.cat([3.0 * torch.eye(E), torch.zeros(E, W - E)], 1), "mlp.correction": 0.3 * rnd(E, seed=2) - 0.4}
    for e in range(E):
        t.update({f"mlp.e{e}.gate": rnd(Fe, W, seed=10 + e, scale=0.3), f"mlp.e{e}.up": rnd(Fe, W, seed=40 + e, scale=0.3),
                  f"mlp.e{e}.down": rnd(W, Fe, seed=70 + e, scale=0.2)})
    if Fs:
        t.update({"mlp.shared.gate": rnd(Fs, W, seed=3, scale=0.3), "mlp.shared.up": rnd(Fs, W, seed=4, scale=0.3),
                  "mlp.shared.down": rnd(W, Fs, seed=5, scale=0.2), "mlp.shared.sg": rnd(1, W, seed=6, scale=0.2)})
    t = {n: v.to(dtype) for n, v in t.items()}
    h = rnd(T, W, seed=7)
    gen = torch.Generator().manual_seed(8)
    for row in range(T):
        for _ in range(200):
            h[row, :E] = torch.randn(E, generator=gen)
            c = torch.sigmoid(3.0 * h[row, :E]) + t["mlp.correction"].float()
            n, keep = (g["count"], g["keep"]) if g else (1, 1)
            per = torch.sort(c.reshape(n, -1), -1, descending=True).values[:, :2].sum(-1)
            so = torch.sort(per, descending=True)
            ok = keep == n or float(so.values[keep - 1] - so.values[keep]) > 0.03
            c2 = torch.sort(torch.cat([c.reshape(n, -1)[i] for i in so.indices[:keep]]), descending=True).values
            if ok and (c2.numel() == top or float(c2[top - 1] - c2[top]) > 0.03):
                break
    h = h.to(dtype)
    p = part("feed_forward", "routed", dict(hidden_size=W, experts=E, top=top, expert_size=Fe, score="sigmoid_normed", weight_at="output",
                                            groups=(g["count"], g["keep"]) if g else None, weight_scale=r.get("scale", 1.0), shared_size=Fs,
                                            shared_gate=True), dtype, t)
    x = torch.full((T, W), 0.5, device=DEV)
    p.forward(h.to(DEV), x, SimpleNamespace(max_q_len=T if prompt else 1, dump=None))
    want = 0.5 + plain.experts(h.double(), {n.split("mlp.")[1]: v.double() for n, v in t.items()}, r)
    close(x, want, dtype)


# ------------------------------------------------------------------------------------------ side by side, the block
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_two_mixers_with_constant_scales_in_any_block(dtype):
    """The join as a pair (a block that sums on its own way) and as a plain addition into x."""
    from hipinfer_b200.kernels import ops
    from hipinfer_b200.parts.spec import PartSpec

    W = 32
    side = lambda s: PartSpec("matrix_memory", dict(hidden_size=W, heads=2, dim=8, vdim=8, gate_cap=15.0, eps=1e-5, **{
        k + "_name": f"mix.{s}.{n}" for k, n in dict(q="q", k="k", v="v", g="g", i="i", i_bias="i.b", f="f", f_bias="f.b", norm="norm", o="o").items()}))
    shapes = dict(q=(16, W), k=(16, W), v=(16, W), g=(16, W), i=(2, W), f=(2, W), o=(W, 16), norm=(16,), **{"i.b": (2,), "f.b": (2,)})
    t = {f"mix.{s}.{n}": rnd(*shape, seed=hash_of(s, n), scale=0.3).to(dtype) for s in ("left", "right") for n, shape in shapes.items()}
    p = part("mixer", "side_by_side", dict(hidden_size=W, left=side("left"), right=side("right"), join="scaled", left_scale=0.65, right_scale=-1.2), dtype, t)
    h = rnd(20, W, seed=1).to(dtype)
    state = lambda: {n: torch.zeros((1,) + tuple(s), dtype=dt, device=DEV) for n, (s, dt) in p.state_need().items()}
    m = dict(heads=2, dim=8, vdim=8, gate_cap=15.0)
    want = sum(c * plain.memory_mixer(h.double(), {n.split(s + ".", 1)[1]: v.double() for n, v in t.items() if f".{s}." in n}, m, 1e-5)
               for s, c in (("left", 0.65), ("right", -1.2)))
    pair = p.forward_pair(h.to(DEV), batch_of([20]), None, state())
    assert isinstance(pair, ops.ScaledPair)
    close(pair.ca * pair.a.cpu() + pair.cb * pair.b.cpu(), want, dtype, tol=5e-5 if dtype == torch.float32 else 2e-2)
    x = torch.full((20, W), 2.0, device=DEV)
    p.forward(h.to(DEV), x, batch_of([20]), None, state())
    close(x, 2.0 + want, dtype)


def hash_of(*parts):
    return sum(ord(c) * (i + 1) for i, c in enumerate("/".join(parts)))


def test_history_with_a_layer_that_does_not_average(tmp_path):
    """A model whose middle layer has a block without an average: its result is a state of the later layers' averages all the
    same (the decoder keeps it)."""
    from hipinfer_b200.engine.batch import StepEntry
    from hipinfer_b200.engine.runner import ModelRunner
    from hipinfer_b200.config import config_from_dict, get_architecture
    from hipinfer_b200.config.base import register_architecture
    import dataclasses
    import gakupel_models as tm
    import tiny

    cfg = tm.model(64, 32, [tm.attention(2, 1, 16, mlp=tm.dense(32)), tm.attention(2, 2, 16, rot_dims=8, mlp=tm.dense(48)),
                            tm.delta(2, 1, 16, 16, 2)], max_positions=100)
    w = tm.draw_weights(cfg, 3, torch.float32)

    def spec(c):
        s = get_architecture("Gakupel").build_spec(c)
        mid = dataclasses.replace(s.layers[1], params=dict(s.layers[1].params, average=0))
        return dataclasses.replace(s, layers=(s.layers[0], mid, s.layers[2]))

    register_architecture("GakupelMiddle", type(config_from_dict(cfg)), spec)
    c = dataclasses.replace(config_from_dict(cfg), architecture="GakupelMiddle")
    tensors = {n: t.to(DEV) for n, t in w.items() if n != "l1.dwa"}
    toks = tiny.random_tokens(40, 64, 2)
    runner = ModelRunner(c, tensors, dtype="float32", num_pages=8, max_num_seqs=1)
    got = runner.step([StepEntry("a", toks, list(range(40)))]).cpu()
    plain_w = dict(w)
    plain_w["l1.dwa"] = torch.tensor([0.0, 0.0, 1.0])                      # what goes on is the layer's own result
    close(got, plain.forward(cfg, plain_w, toks), torch.float32, tol=5e-5)
