"""A plain, slow statement of the Selovik decoder on the CPU, one function per mechanism, written from the design's
equations and sharing no code with the engine. Everything is float64 torch on whole sequences; nothing is paged, batched,
cached or fused. The GPU tests compare the engine with these functions.

Notation: T tokens at positions p = 0..T-1 of one sequence, W the model's width.

  norm              N_w(x) = x / sqrt(mean x^2 + eps) * (1 + w)
  embedding         N_en(scale embed[t_p] + bigram[(t_(p-1) mp + t_p mc) mod B]),  row B for the first token
  run order         layers before the loop; the loop's layers `times` times, each pass starting with
                    x <- x (+ embedding output, from the second pass on) + step[pass];  the layers after it
  layer             x <- x + mixer(N1(x)) + ff(N2(x)), both of the same x
  attention         per head two maps: q_m, k_m rotated on their first dims; s_m = scale q_m k_m^T over 0 <= i - j < window;
                    a_m = softmax(s_m) v;  lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff;  o = a_1 - lambda a_2;
                    o / rms(o) (1 - diff) per head;  Wo (concat(o) sigmoid(Wg h))
  rotation          pairs (i, i + dims/2) by p f_i, with YaRN: f_i / factor r_i + f_i (1 - r_i), cos and sin times
                    0.1 ln(factor) + 1
  dense             Wdown relu(Wup h)^2
  experts           s = softmax(Wr h) over experts and identity experts, c = s + correction;  groups of neighbours ranked by
                    their largest c, the best `keep` stay;  the `top` largest c there;  weights s;
                    sum_e weight_e (Wd_e (silu(Wg_e h) * Wu_e h), or h for an identity expert) + shared(h)
  output            logits = logit_scale embed N_f(x)
"""
from __future__ import annotations

import math

import torch

F = torch.float64


def norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * (1.0 + w)


def silu(z):
    return z * torch.sigmoid(z)


def bigram_rows(tokens, b):
    """The bigram table's row of every token; b: buckets, mul_prev, mul_cur."""
    rows = [b["buckets"]]
    for prev, cur in zip(tokens[:-1], tokens[1:]):
        rows.append((prev * b["mul_prev"] + cur * b["mul_cur"]) % b["buckets"])
    return rows


def embedding(tokens, w, cfg):
    tokens = [int(t) for t in tokens]
    e = cfg.get("embedding") or {}
    x = w["embed"].to(F)[tokens] * e.get("scale", 1.0)
    if e.get("bigram"):
        x = x + w["bigram"].to(F)[bigram_rows(tokens, e["bigram"])]
    return norm(x, w["embed.norm"].to(F), cfg["norm"]["eps"])


def frequencies(rot):
    """([dims / 2] turns per position, magnitude of cos and sin); rot: dims, base, scaling {factor, original, fast, slow}."""
    dims, base, sc = rot["dims"], float(rot["base"]), rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return f, 1.0
    at = lambda t: dims * math.log(sc["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo, hi = max(math.floor(at(sc["fast"])), 0), min(math.ceil(at(sc["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * r + fi * (1 - r))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(t, positions, rot):
    """t [T, ..., D]: dimension i < dims / 2 is paired with i + dims / 2."""
    f, mag = frequencies(rot)
    out, n = t.clone(), len(f)
    shape = (-1,) + (1,) * (t.dim() - 2)
    for i in range(n):
        ang = positions.to(F) * f[i]
        c, s = (mag * torch.cos(ang)).view(shape), (mag * torch.sin(ang)).view(shape)
        u, v = t[..., i], t[..., i + n]
        out[..., i] = u * c - v * s
        out[..., i + n] = v * c + u * s
    return out


def window_softmax(s, window):
    """Rows of softmax over the keys 0 <= i - j < window (None: every j <= i)."""
    T = s.shape[0]
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    hide = (d < 0) if not window else (d < 0) | (d >= window)
    return torch.softmax(s.masked_fill(hide, float("-inf")), -1)


def combination(w, diff):
    dot = lambda a, b: float((w[a].double() * w[b].double()).sum())
    return math.exp(dot("lq1", "lk1")) - math.exp(dot("lq2", "lk2")) + diff


def head_norm(o, eps):
    return o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps)


def attention(h, w, m, eps):
    """w: q, k, v, g, o, lq1, lk1, lq2, lk2; m: heads, kv_heads, dim, vdim, scale, diff, rot, mask {size}."""
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    pos = torch.arange(T)
    q, k = (h @ w["q"].T).reshape(T, H, 2, D), (h @ w["k"].T).reshape(T, G, 2, D)
    v = (h @ w["v"].T).reshape(T, G, E)
    rot = m.get("rot")
    if rot and rot["dims"]:
        q, k = rotate(q, pos, rot), rotate(k, pos, rot)
    lam, window = combination(w, m["diff"]), (m.get("mask") or {}).get("size")
    out = torch.zeros(T, H, E, dtype=F)
    for hd in range(H):
        g = hd // (H // G)
        a1, a2 = (window_softmax((q[:, hd, j] @ k[:, g, j].T) * m["scale"], window) @ v[:, g] for j in (0, 1))
        out[:, hd] = head_norm(a1 - lam * a2, eps) * (1.0 - m["diff"])
    return (out.reshape(T, H * E) * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def dense(h, w):
    return torch.clamp(h @ w["up"].T, min=0.0) ** 2 @ w["down"].T


def expert(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def route(h, router, correction, r):
    """(chosen [T, top], weights [T, top]); r: top, groups {count, keep} or none. Ties: the lower index."""
    s = torch.softmax(h @ router.T, -1)
    c = s + correction
    T, E = s.shape
    g = r.get("groups")
    if g:
        best = torch.sort(c.reshape(T, g["count"], -1).amax(-1), dim=-1, descending=True, stable=True).indices[:, :g["keep"]]
        stay = torch.zeros(T, g["count"], dtype=torch.bool)
        stay.scatter_(1, best, True)
        c = c.masked_fill(~stay.repeat_interleave(E // g["count"], 1), float("-inf"))
    chosen = torch.sort(c, dim=-1, descending=True, stable=True).indices[:, :r["top"]]
    return chosen, torch.gather(s, 1, chosen)


def closest_call(h, router, correction, r):
    """Per token, how far the closest of the router's calls is from going the other way (the last group kept against the first
    one dropped, the last expert chosen against the next)."""
    c = torch.softmax(h @ router.T, -1) + correction
    T, E = c.shape
    g, margin = r.get("groups"), torch.full((T,), float("inf"), dtype=F)
    if g and g["keep"] < g["count"]:
        best = torch.sort(c.reshape(T, g["count"], -1).amax(-1), dim=-1, descending=True)
        margin = best.values[:, g["keep"] - 1] - best.values[:, g["keep"]]
        stay = torch.zeros(T, g["count"], dtype=torch.bool).scatter_(1, best.indices[:, :g["keep"]], True)
        c = c.masked_fill(~stay.repeat_interleave(E // g["count"], 1), float("-inf"))
    c = torch.sort(c, dim=-1, descending=True).values
    if r["top"] < E:
        margin = torch.minimum(margin, c[:, r["top"] - 1] - c[:, r["top"]])
    return margin


def experts(h, w, r):
    """w: router, correction, e<i>.gate / up / down, shared.gate / up / down; r also: experts, identity."""
    chosen, weight = route(h, w["router"], w["correction"], r)
    out = torch.zeros_like(h)
    for e in range(r["experts"] + r.get("identity", 0)):
        rows, col = (chosen == e).nonzero(as_tuple=True)
        if rows.numel():
            out[rows] += weight[rows, col][:, None] * (expert(h[rows], sub(w, f"e{e}.")) if e < r["experts"] else h[rows])
    if "shared.gate" in w:
        out = out + expert(h, sub(w, "shared."))
    return out


def feed_forward(h, w, mlp):
    return dense(h, w) if mlp["kind"] == "dense" else experts(h, w, mlp["router"])


def run_order(cfg):
    """[(layer, pass or None)]: pass t at the first layer of the loop's pass t."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        out += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return out + [(i, None) for i in range(loop["stop"], n)]


def sub(tensors, prefix):
    return {k[len(prefix):]: v.to(F) for k, v in tensors.items() if k.startswith(prefix)}


def forward(cfg, tensors, tokens, layers_out=None, round_to=None, calls=None):
    """Logits [T, vocab] of one sequence from position 0. cfg: the config.json dictionary; tensors: name -> tensor.
    layers_out (a list): the residual rows after every layer run are appended. round_to (a function): every sublayer's input
    and result go through it; the difference to the exact logits measures how sensitive each position is to rounding. calls (a
    list): every router's closest call per position is appended."""
    rd = round_to or (lambda t: t)
    eps = cfg["norm"]["eps"]
    x = x0 = embedding(tokens, tensors, cfg)
    layers = [sub(tensors, f"l{i}.") for i in range(len(cfg["layers"]))]
    for i, t in run_order(cfg):
        if t is not None:
            if t > 0:
                x = x + x0
            x = x + tensors["loop.step"].to(F)[t]
        L, w = cfg["layers"][i], layers[i]
        y = rd(attention(rd(norm(x, w["norm1"], eps)), sub(w, "mix."), L["mixer"], eps))
        if L.get("mlp") is not None:
            h = rd(norm(x, w["norm2"], eps))
            if calls is not None and L["mlp"]["kind"] == "moe":
                calls.append(closest_call(h, w["mlp.router"], w["mlp.correction"], L["mlp"]["router"]))
            y = y + rd(feed_forward(h, sub(w, "mlp."), L["mlp"]))
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm(x, tensors["final.norm"].to(F), eps) @ tensors["embed"].to(F).T * cfg.get("logit_scale", 1.0)
