"""One kernel at given sizes, timed with CUDA events: for profiling a kernel alone and for the
roofline figures under `profiles/` (the reference times its kernels one by one the same way,
scripts/bench.py:126-212, and reports GB/s or TFLOP/s from algorithmic bytes and flops).

    python -m hipinfer_b200.kernels.microbench gemm_tc --m 2048 --n 16384 --k 2048 --epi swiglu
    python -m hipinfer_b200.kernels.microbench gemm_stream --m 8 --n 65536 --k 2048
    python -m hipinfer_b200.kernels.microbench attn_decode --batch 64 --context 2176
    python -m hipinfer_b200.kernels.microbench flash_prefill --tokens 2048
    python -m hipinfer_b200.kernels.microbench rmsnorm --m 2048 --n 2048
    python -m hipinfer_b200.kernels.microbench delta_rule --tokens 2048 --batch 1 --heads 32 --head-dim 64
    python -m hipinfer_b200.kernels.microbench attn_window --batch 8 --context 2048 --window 1024        (single rows)
    python -m hipinfer_b200.kernels.microbench attn_window --portion --tokens 2048 --window 1024         (a prompt portion)
    python -m hipinfer_b200.kernels.microbench attn_window --keep 0 ...                                  (the same without kept first tokens)
    python -m hipinfer_b200.kernels.microbench two_norms --m 2048 --n 2048
    python -m hipinfer_b200.kernels.microbench rope_maps --m 2048 --heads 32 --kv-heads 8 --head-dim 64  (two maps a head, values --value-dim wide)
    python -m hipinfer_b200.kernels.microbench router --m 2048 --k 2048 --experts 12
    python -m hipinfer_b200.kernels.microbench experts --batch 64 --k 2048 --n 4096 --experts 8          (single rows, two experts each)
    python -m hipinfer_b200.kernels.microbench layernorm|polynorm|scale_add --m 2048 --n 2048
    python -m hipinfer_b200.kernels.microbench selective_scan --tokens 2048 --batch 1 --n 2048 --states 16   (a prompt portion)
    python -m hipinfer_b200.kernels.microbench selective_scan --tokens 1 --batch 64 --n 2048 --states 16     (single rows)
    python -m hipinfer_b200.kernels.microbench residual_norm --m 2048 --n 2048 [--pair]
    python -m hipinfer_b200.kernels.microbench matrix_memory|gated_delta --tokens 2048 --batch 1 --heads 32 --head-dim 64  (the walk of a portion)
    python -m hipinfer_b200.kernels.microbench matrix_memory|gated_delta --tokens 1 --batch 64   (single tokens: the whole mixer's kernel)
    python -m hipinfer_b200.kernels.microbench output_norm --m 2048 --n 2048 --states 9          (states of the depth average)

Between timed launches of kernels whose inputs fit in L2 a buffer larger than L2 is written
(`--flush`, on by default) so that the figures are for operands coming from HBM.
"""
from __future__ import annotations

import argparse
import json
import math
import sys

import torch

EPI = {"f32": 0, "bf16": 1, "add": 2, "swiglu": 3}


def timeit(fn, iters, flush):
    """Median milliseconds of `fn` over `iters` launches, each bracketed by events."""
    scratch = torch.empty(256 << 20, dtype=torch.uint8, device="cuda") if flush else None
    for _ in range(3):
        fn()
    torch.cuda.synchronize()
    times = []
    for _ in range(iters):
        if scratch is not None:
            scratch.zero_()
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        start.record()
        fn()
        stop.record()
        stop.synchronize()
        times.append(start.elapsed_time(stop))
    times.sort()
    return times[len(times) // 2]


def _prepared(fast, x, nw):
    """A filled NormFeed for residual rows x: what a product with the residual add in its epilogue leaves for the next norm."""
    M, K = x.shape
    feed = fast.NormFeed(nw, 1e-5, M)
    feed.xb.copy_((x * nw.float()).bfloat16())
    feed.ssq.zero_()
    feed.ssq[:, :M] = (x * x).reshape(M, K // 16, 16).sum(-1).T
    feed.filled = True
    return feed


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawTextHelpFormatter)
    ap.add_argument("kernel", choices=["gemm_tc", "gemm_stream", "rows_add", "rows_swiglu", "rows_qkv", "attn_decode", "flash_prefill", "flash_prefill_tc", "rmsnorm",
                                       "delta_rule", "attn_window", "layernorm", "polynorm", "scale_add", "selective_scan", "residual_norm",
                                       "matrix_memory", "gated_delta", "output_norm", "two_norms", "rope_maps", "router", "experts"])
    ap.add_argument("--m", type=int, default=8)
    ap.add_argument("--n", type=int, default=16384)
    ap.add_argument("--k", type=int, default=2048)
    ap.add_argument("--epi", default="f32", choices=sorted(EPI))
    ap.add_argument("--tile-n", type=int, default=0)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--context", type=int, default=2176)
    ap.add_argument("--tokens", type=int, default=2048)
    ap.add_argument("--heads", type=int, default=32)
    ap.add_argument("--kv-heads", type=int, default=8)
    ap.add_argument("--head-dim", type=int, default=64)
    ap.add_argument("--page-size", type=int, default=16)
    ap.add_argument("--window", type=int, default=1024, help="attn_window: the window (0: none)")
    ap.add_argument("--keep", type=int, default=4, help="attn_window: first tokens that the window keeps (0: the TMA and tcgen05 kernels)")
    ap.add_argument("--experts", type=int, default=8, help="experts, router: how many (--n is their width, --k the rows')")
    ap.add_argument("--value-dim", type=int, default=64, help="attn_window: width of a head's values (a score map is --head-dim / 2 wide)")
    ap.add_argument("--portion", action="store_true", help="attn_window: one request's portion of --tokens rows instead of --batch single rows")
    ap.add_argument("--states", type=int, default=16, help="selective_scan: states a channel (--n is the number of channels)")
    ap.add_argument("--pair", action="store_true", help="residual_norm: two side-by-side results that are normed and joined")
    ap.add_argument("--iters", type=int, default=20)
    ap.add_argument("--no-flush", dest="flush", action="store_false")
    ap.add_argument("--prepared-norm", action="store_true",
                    help="rows_swiglu, rows_qkv: the rows come as a prepared norm (x times the norm's weight and the pieces of "
                         "the sums of squares, as the product before leaves them) instead of the residual rows")
    a = ap.parse_args(argv)

    from . import fast, ops

    dev = "cuda:0"
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s: torch.randn(*s, generator=g, device=dev)
    out = {"kernel": a.kernel}
    if a.kernel == "selective_scan":
        from types import SimpleNamespace

        R, L, I, N = a.batch, a.tokens, a.n, a.states
        T = R * L
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
        x, dt, z, bc = rnd(T, I), rnd(T, I), rnd(T, I), rnd(T, 2 * N)
        a_log = (torch.rand(I, N, generator=g, device=dev) * 5 - 4).bfloat16()
        dt_bias, d = rnd(I).bfloat16(), rnd(I).bfloat16()
        state, y = torch.zeros(R, I, N, device=dev), torch.empty(T, I, dtype=torch.bfloat16, device=dev)
        batch = SimpleNamespace(n_requests=R, max_q_len=L, req_q_start=i32([r * L for r in range(R)]), req_q_len=i32([L] * R),
                                req_state_slot=i32(list(range(R))))
        fn = lambda: ops.selective_scan(x, dt, bc, z, dt_bias, a_log, d, state, batch, y)
        ms = timeit(fn, a.iters, a.flush)
        pieces = L >= 3 * ops.SEL_PIECE_TOKENS > 0
        # rows in (x, dt, B | C, and z once) and out, the states in and out; in pieces x, dt and B are read twice
        nbytes = T * (I * 4 * (5 if pieces else 3) + 2 * N * 4 * (1.5 if pieces else 1) + I * 2) + 2 * R * I * N * 4
        out.update(requests=R, tokens=L, channels=I, states=N, pieces=bool(pieces), ms=ms, gbs=nbytes / ms / 1e6,
                   us_per_token=ms * 1e3 / L)
    elif a.kernel in ("matrix_memory", "gated_delta"):
        from types import SimpleNamespace

        R, L, H, D, delta = a.batch, a.tokens, a.heads, a.head_dim, a.kernel == "gated_delta"
        T = R * L
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
        q, k, v, gate = (rnd(T, H * D) for _ in range(4))
        dec, add = torch.rand(T, H, generator=g, device=dev) * 0.1 + 0.9, torch.rand(T, H, generator=g, device=dev)
        state, y = torch.zeros(R, H, D, D, device=dev), torch.empty(T, H * D, device=dev)
        ns, ms, nq = (torch.zeros(*s, device=dev) for s in ((R, H, D), (R, H), (T, H)))
        batch = SimpleNamespace(n_requests=R, max_q_len=L, req_q_start=i32([r * L for r in range(R)]), req_q_len=i32([L] * R),
                                req_state_slot=i32(list(range(R))), row_request=i32([r for r in range(R) for _ in range(L)]))
        if L == 1:
            vec, nw = rnd(H).bfloat16(), torch.ones(D if delta else H * D, device=dev).bfloat16()
            out16 = torch.empty(T, H * D, dtype=torch.bfloat16, device=dev)
            fn = lambda: ops.ms_single(q, k, v, dec, add, vec, vec, state, nw, gate, "silu" if delta else "sigmoid", out16, batch, D ** -0.5, 1e-5,
                                       None if delta else ns, None if delta else ms, 15.0, 1e-6, 1e-6)
            nbytes = R * H * (2 * D * D * 4 + 4 * D * 4 + 2 * D + (0 if delta else 8 * D))
        else:
            vec = torch.zeros(H, device=dev)
            scal = ops.ms_delta_prepare(q, k, dec * -6.0, add, vec, vec, batch, D, D ** -0.5, 1e-6) if delta else None
            fn = ((lambda: ops.ms_delta_walk(q, k, v, scal, state, batch, y)) if delta
                  else lambda: ops.ms_walk(q, k, v, dec, add, state, batch, y, D ** -0.5, ns, nq))
            pieces = not delta and L >= 3 * ops.MS_PIECE_TOKENS > 0
            nbytes = T * H * D * 4 * (6 if pieces else 4) + 2 * R * H * D * D * 4
        ms_ = timeit(fn, a.iters, a.flush)
        out.update(requests=R, tokens=L, heads=H, head_dim=D, ms=ms_, gbs=nbytes / ms_ / 1e6, us_per_token=ms_ * 1e3 / L)
    elif a.kernel == "output_norm":
        M, W, n = a.m, a.n, a.states
        x, y, states, coef = rnd(M, W), rnd(M, W), rnd(n + 1, M, W), rnd(n + 1)
        w, b = torch.ones(W, device=dev).bfloat16(), torch.zeros(W, device=dev).bfloat16()
        rounded = torch.empty(M, W, dtype=torch.bfloat16, device=dev)
        fn = lambda: ops.output_norm(x, y, w, b, 1e-5, rounded, None, states[n], states[:n] if n else None, coef if n else None)
        ms = timeit(fn, a.iters, a.flush)
        out.update(m=M, n=W, states=n, ms=ms, gbs=M * W * (4 * (n + 4) + 2) / ms / 1e6)
    elif a.kernel == "residual_norm":
        M, W = a.m, a.n
        x, y, w = rnd(M, W), rnd(M, W), 1 + 0.1 * rnd(W)
        pair = ops.NormedPair(rnd(M, W), rnd(M, W), torch.ones(W, device=dev).bfloat16(), torch.ones(W, device=dev).bfloat16(), 0.5, 1e-5) if a.pair else None
        rounded = torch.empty(M, W, dtype=torch.bfloat16, device=dev)
        fn = lambda: ops.residual_norm(x, None if a.pair else y, pair, 2.0, w, 1e-5, rounded)
        ms = timeit(fn, a.iters, a.flush)
        out.update(m=M, n=W, pair=a.pair, ms=ms, gbs=M * W * (4 * (3 if a.pair else 2) + 4 + 2) / ms / 1e6)
    elif a.kernel.startswith("rows"):
        M, N, K = a.m, a.n, a.k
        w = (rnd(N, K) * 0.02).bfloat16()
        nw = torch.ones(K, device=dev, dtype=torch.bfloat16)
        if a.kernel == "rows_add":
            act, acc = rnd(M, K).bfloat16(), torch.zeros(M, N, device=dev)
            fn = lambda: fast.rows_add(act, w, acc)
        elif a.kernel == "rows_swiglu":
            x, act = rnd(M, K), torch.empty(M, N // 2, device=dev, dtype=torch.bfloat16)
            fn = lambda: fast.rows_norm_swiglu(x, nw, 1e-5, w, act, 16)
            if a.prepared_norm:
                feed = _prepared(fast, x, nw)
                fn = lambda: fast.rows_scaled_swiglu(feed, M, w, act, 16)
        else:
            Hq, Hkv, D = a.heads, a.kv_heads, a.head_dim
            N = (Hq + 2 * Hkv) * D
            w = (rnd(N, K) * 0.02).bfloat16()
            x, q = rnd(M, K), torch.empty(M, Hq * D, device=dev, dtype=torch.bfloat16)
            table = ops.rope_table((10000.0 ** (-torch.arange(0, D, 2, dtype=torch.float64) / D)).float().to(dev), 4096)
            pos = torch.arange(M, dtype=torch.int32, device=dev) + 2048
            kc = torch.zeros(M + 4, Hkv, a.page_size, D, device=dev, dtype=torch.bfloat16)
            vc = torch.zeros_like(kc)
            slots = (torch.arange(M, dtype=torch.int32, device=dev) * a.page_size)
            fn = lambda: fast.rows_norm_qkv_rope(x, nw, 1e-5, w, pos, slots, table, q, kc, vc, Hq, Hkv, D, D, a.page_size)
            if a.prepared_norm:
                feed = _prepared(fast, x, nw)
                fn = lambda: fast.rows_scaled_qkv_rope(feed, M, w, pos, slots, table, q, kc, vc, Hq, Hkv, D, D, a.page_size)
        assert fn(), "the rows kernel does not take these sizes"
        ms = timeit(fn, a.iters, a.flush)
        out.update(M=M, N=N, K=K, ms=ms, gbs=N * K * 2 / ms / 1e6)
    elif a.kernel.startswith("gemm"):
        M, N, K, epi = a.m, a.n, a.k, EPI[a.epi]
        x, w = rnd(M, K).bfloat16(), (rnd(N, K) * 0.02).bfloat16()
        c = torch.zeros(M, N // 2 if epi == 3 else N, device=dev, dtype=torch.bfloat16 if epi in (1, 3) else torch.float32)
        if a.kernel == "gemm_tc":
            fn = lambda: fast.gemm_tc(x, w, c, epi, a.tile_n)
        else:
            fn = lambda: fast.gemm_stream(x, w, c, epi)
        ms = timeit(fn, a.iters, a.flush)
        nbytes = N * K * 2 + M * K * 2 + c.numel() * c.element_size()
        out.update(M=M, N=N, K=K, epi=a.epi, ms=ms, tflops=2.0 * M * N * K / ms / 1e9, gbs=nbytes / ms / 1e6)
    elif a.kernel in ("layernorm", "polynorm", "scale_add"):
        x, w = rnd(a.m, a.n), torch.ones(a.n, device=dev, dtype=torch.bfloat16)
        y = torch.empty(a.m, a.n, device=dev, dtype=torch.bfloat16)
        if a.kernel == "layernorm":
            fn, nbytes = (lambda: ops.layernorm(x, w, 1e-5, y)), a.m * a.n * 6
        elif a.kernel == "polynorm":
            fn, nbytes = (lambda: ops.polynorm(x, [1.0, 1.0, 1.0, 1.0], 1e-5, y)), a.m * a.n * 6
        else:
            x2 = rnd(a.m, a.n)
            fn, nbytes = (lambda: ops.scale_add(x, x2, w)), a.m * a.n * 12
        ms = timeit(fn, a.iters, a.flush)
        out.update(M=a.m, H=a.n, ms=ms, gbs=nbytes / ms / 1e6)
    elif a.kernel == "delta_rule":
        from types import SimpleNamespace

        T, R, Hh, D = a.tokens * a.batch if a.tokens < 16 else a.tokens, a.batch, a.heads, a.head_dim
        n, HD = T // R, a.heads * a.head_dim
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
        proj, w_raw = rnd(R * n, 5 * HD), rnd(R * n, HD)
        vec = [rnd(HD).bfloat16() for _ in range(3)]
        state, y = torch.zeros(R, Hh, D, D, device=dev), torch.empty(R * n, HD, device=dev, dtype=torch.bfloat16)
        batch = SimpleNamespace(req_q_start=i32([i * n for i in range(R)]), req_q_len=i32([n] * R),
                                req_state_slot=i32(list(range(R))), n_requests=R)
        fn = lambda: ops.delta_rule(proj, (0, HD, 2 * HD, 3 * HD, 4 * HD), w_raw, *vec, state, batch, y, Hh, D, 0.6, 1e-6, 1e-5)
        ms = timeit(fn, a.iters, a.flush)
        nbytes = R * n * HD * (5 * 4 + 4 + 2) + 2 * R * Hh * D * D * 4
        out.update(requests=R, tokens_each=n, heads=Hh, head_dim=D, ms=ms, us_per_token=ms * 1e3 / n, gbs=nbytes / ms / 1e6)
    elif a.kernel == "attn_window":
        from types import SimpleNamespace

        H, G, D, E, ps, window = a.heads, a.kv_heads, a.head_dim // 2, a.value_dim, a.page_size, a.window
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
        rows = a.portion                                       # a portion of --tokens rows, else --batch single rows at --context
        R, T, ctx = (1, a.tokens, a.tokens) if rows else (a.batch, a.batch, a.context)
        pages = ctx // ps + 1
        kc, vc = rnd(R * pages, G, ps, 2 * D).bfloat16(), rnd(R * pages, G, ps, E).bfloat16()
        bt = torch.arange(R * pages, dtype=torch.int32, device=dev).view(R, pages)
        q, gate, y = rnd(T, H * 2 * D).bfloat16(), rnd(T, H * E), torch.empty(T, H * E, device=dev, dtype=torch.bfloat16)
        if rows:
            batch = SimpleNamespace(block_tables=[bt], row_request=i32([0] * T), positions=i32(list(range(T))), max_q_len=T,
                                    n_requests=1, req_q_start=i32([0]), req_q_len=i32([T]), req_ctx_len=i32([0]), h_q_len=[T],
                                    max_pos=T - 1)
            pairs = sum(min(p + 1, window + a.keep) if window else p + 1 for p in range(T))
        else:
            batch = SimpleNamespace(block_tables=[bt], row_request=i32(list(range(R))), positions=i32([ctx] * R), max_q_len=1,
                                    max_pos=ctx, n_requests=R, req_ctx_len=i32([ctx] * R))
            pairs = R * (min(ctx + 1, window + a.keep) if window else ctx + 1)
        fn = lambda: ops.attention_window(q, kc, vc, batch, 0, y, H, G, D, E, 2, ps, window, a.keep, D ** -0.5, 0.5, 0.5, 1e-5, True,
                                          gate=gate)
        ms = timeit(fn, a.iters, a.flush)
        nbytes = pairs * G * (2 * D + E) * 2                   # single rows: every visible key and value once a kv head
        out.update(rows=T, requests=R, heads=H, kv_heads=G, map_dim=D, value_dim=E, window=window, ms=ms,
                   tflops=pairs * H * (4 * D + 4 * E) / ms / 1e9)
        if not rows:
            out.update(gbs=nbytes / ms / 1e6)
    elif a.kernel == "two_norms":
        x, w1, w2 = rnd(a.m, a.n), rnd(a.n), rnd(a.n)
        ms = timeit(lambda: ops.two_norms(x, w1, w2, 1e-5, torch.bfloat16), a.iters, a.flush)
        out.update(M=a.m, H=a.n, ms=ms, gbs=a.m * a.n * 8 / ms / 1e6)
    elif a.kernel == "rope_maps":
        H, G, D, E, ps, T = a.heads, a.kv_heads, a.head_dim // 2, a.value_dim, a.page_size, a.m
        cols = H * 2 * D + G * 2 * D + G * E
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
        proj, q, table = rnd(T, cols), torch.empty(T, H * 2 * D, device=dev, dtype=torch.bfloat16), ops.shared_rope_table(D, 10000.0, T, dev)
        kc, vc = (torch.empty(-(-T // ps), G, ps, n, device=dev, dtype=torch.bfloat16) for n in (2 * D, E))
        pos, slots = i32(list(range(T))), i32(list(range(T)))
        ms = timeit(lambda: ops.rope_norm_store(proj, (0, H * 2 * D, H * 2 * D + G * 2 * D), pos, slots, table, D, "half", False, 0.0, q, kc,
                                                vc, H * 2, G * 2, D, E, ps, maps=2), a.iters, a.flush)
        out.update(rows=T, heads=H, kv_heads=G, map_dim=D, value_dim=E, ms=ms, gbs=T * cols * 6 / ms / 1e6)
    elif a.kernel == "router":
        x, w, c = rnd(a.m, a.k).bfloat16(), rnd(a.experts, a.k).bfloat16() * 0.02, rnd(a.experts).bfloat16() * 0.01
        ms = timeit(lambda: ops.moe_route(x, w, 2, None, "softmax", c), a.iters, a.flush)
        out.update(rows=a.m, experts=a.experts, K=a.k, ms=ms, gbs=(a.m + a.experts) * a.k * 2 / ms / 1e6)
    elif a.kernel == "experts":
        T, W, F, E = a.batch, a.k, a.n, a.experts
        wgu, wd = rnd(E, 2 * F, W).bfloat16() * 0.02, rnd(E, W, F).bfloat16() * 0.02
        ex = torch.stack([torch.randperm(E, generator=g, device=dev)[:2] for _ in range(T)]).to(torch.int32)
        x, y, sc = rnd(T, W).bfloat16(), rnd(T, W), torch.rand(T, 2, generator=g, device=dev)
        offsets, pos, src = ops.moe_sort(ex, E)
        act, ys = torch.empty(2 * T, F, device=dev, dtype=torch.bfloat16), torch.empty(2 * T, W, device=dev)
        used = int(ex.unique().numel())
        up = timeit(lambda: ops.moe_grouped_act(x, src, 2, wgu, offsets, sc, act, True), a.iters, a.flush)
        down = timeit(lambda: ops.moe_grouped(act, None, 1, wd, offsets, ys), a.iters, a.flush)
        out.update(rows=T, experts=E, experts_used=used, gate_up_ms=up, gate_up_gbs=used * 4 * F * W / up / 1e6, down_ms=down,
                   down_gbs=used * 2 * F * W / down / 1e6)
    elif a.kernel == "rmsnorm":
        x, w = rnd(a.m, a.n), torch.ones(a.n, device=dev, dtype=torch.bfloat16)
        y = torch.empty(a.m, a.n, device=dev, dtype=torch.bfloat16)
        ms = timeit(lambda: ops.rmsnorm(x, w, 1e-5, y), a.iters, a.flush)
        out.update(M=a.m, H=a.n, ms=ms, gbs=a.m * a.n * 6 / ms / 1e6)
    else:
        Hq, Hkv, D, ps = a.heads, a.kv_heads, a.head_dim, a.page_size
        if a.kernel == "attn_decode":
            R, ctx, T = a.batch, a.context, a.batch
            q_len, ctx_len = [1] * R, [ctx - 1] * R
        else:
            R, T, ctx = 1, a.tokens, a.tokens
            q_len, ctx_len = [T], [0]
        pages = -(-ctx // ps)
        kc = (rnd(R * pages, Hkv, ps, D)).bfloat16()
        vc = (rnd(R * pages, Hkv, ps, D)).bfloat16()
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
        bt = torch.arange(R * pages, dtype=torch.int32, device=dev).view(R, pages)
        q = rnd(T, Hq * D).bfloat16()
        o = torch.empty_like(q)
        scale = 1.0 / math.sqrt(D)
        if a.kernel == "attn_decode":
            rr, pos, cl = i32(list(range(R))), i32([ctx - 1] * R), i32(ctx_len)
            fn = lambda: fast.attention_decode(q, kc, vc, bt, None, pos, o, Hq, Hkv, D, ps, 0, scale, ctx - 1, ctx_len=cl)   # row t = request t, as in a decode step
            nbytes = 2 * R * ctx * Hkv * D * 2
            flops = 4.0 * R * ctx * Hq * D
        else:
            qs, ql, cl = i32([0]), i32(q_len), i32(ctx_len)
            impl = fast.flash_prefill_tc if a.kernel == "flash_prefill_tc" else fast.flash_prefill
            fn = lambda: impl(q, kc, vc, bt, qs, ql, cl, o, T, Hq, Hkv, D, ps, 0, scale)
            nbytes = 2 * ctx * Hkv * D * 2 + 2 * T * Hq * D * 2
            flops = 4.0 * Hq * D * (T * (T + 1) / 2)
        ms = timeit(fn, a.iters, a.flush)
        out.update(requests=R, context=ctx, heads=Hq, kv_heads=Hkv, head_dim=D, ms=ms, tflops=flops / ms / 1e9,
                   gbs=nbytes / ms / 1e6)
    torch.cuda.synchronize()
    fast.check_status()
    print(json.dumps({k: (round(v, 4) if isinstance(v, float) else v) for k, v in out.items()}))
    return 0


if __name__ == "__main__":
    sys.exit(main())
