"""A plain, slow statement of the Gakupel decoder on the CPU, one function per mechanism, written from the design's
equations and sharing no code with the engine. Everything is float64 torch on whole sequences (the recurrences token by
token); nothing is paged, batched, cached or fused. The GPU tests compare the engine with these functions.

Notation: T tokens at positions p = 0..T-1 of one sequence, W the model's width.

  layer norm        LN(x) = (x - mean x) / sqrt(mean (x - mean x)^2 + eps) * w + b;    rms(x) = x / sqrt(mean x^2 + eps)
  layer i           z = x + LN1(mixer(x));  X_(i+1) = z + LN2(ff(z)) (no ff: z);  x <- sum_(j <= i+1) a_i[j] X_j,
                    X_0 the embedding rows
  attention         q = rms(Wq h) nq, k = rms(Wk h) nk per head, rotated on the first dims of each head, pairs
                    (i, i + dims/2); values are Wk h itself;  softmax over j <= i of q . k * scale;  Wo
  delta             q, k, v = silu(conv(W h));  q, k to unit length, q / sqrt(dim);  b = sigmoid(Wb h);
                    g = exp(-exp(A_log) softplus(Wa h + dt_bias));  S <- g S;  u = b (v - S^T k);  S <- S + k u^T;  o = S^T q;
                    rms(o) n silu(Wg h) per head;  Wo
  parallel          cl left(h) + cr right(h)
  left              q = rms(Wq h) nq, k = rms(Wk h) nk over the whole rows, no rotation;  q times 1 + c ln(floor((p+1)/n) + 1);
                    s = q . k * scale - r1 ln(1 + r2 (i - j));  exp(s) / (1 + sum exp(s));  Wo
  right             q = Wq h / sqrt(dim), k, v;  li = cap tanh((Wi h + bi) / cap), lf = -softplus(-cap tanh((Wf h + bf) / cap));
                    m' = max(lf + m, li);  S, n <- exp(lf + m - m') (S, n) + exp(li - m') k (v, 1)^T;
                    o = S^T q / (max(|n . q|, exp(-m')) + 1e-6);  rms(o) per head, times n sigmoid(Wg h);  Wo
  dense             Wdown gelu(Wup h), gelu(z) = z Phi(z)
  experts           s = sigmoid(Wr h), c = s + correction;  groups of neighbours ranked by the sum of their two largest c, the
                    best `keep` stay;  the `top` largest c there;  weights s / (sum + 1e-20) * scale;
                    sum_e weight_e Wd_e (silu(Wg_e h) * Wu_e h) + sigmoid(wsg . h) shared(h)
  output            logits = head LN(x)
"""
from __future__ import annotations

import math

import torch

F = torch.float64


def rms(t, eps):
    return t / torch.sqrt((t * t).mean(-1, keepdim=True) + eps)


def layer_norm(t, w, b, eps):
    d = t - t.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def gelu(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def rotate_half(t, positions, dims, base):
    """t [T, ..., D]: dimension i < dims / 2 is paired with i + dims / 2 and turned by position * base^(-2i / dims)."""
    out = t.clone()
    shape = (-1,) + (1,) * (t.dim() - 2)
    for i in range(dims // 2):
        ang = positions.to(F) * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(ang).view(shape), torch.sin(ang).view(shape)
        u, v = t[..., i], t[..., i + dims // 2]
        out[..., i] = u * c - v * s
        out[..., i + dims // 2] = v * c + u * s
    return out


def causal_softmax(s, one_more=False):
    """Rows of softmax over the keys up to the row; one_more: the denominator also holds exp(0)."""
    T = s.shape[0]
    s = s.masked_fill(torch.arange(T)[None, :] > torch.arange(T)[:, None], float("-inf"))
    top = s.max(-1, keepdim=True).values
    if one_more:
        top = torch.clamp(top, min=0.0)
    e = torch.exp(s - top)
    den = e.sum(-1, keepdim=True)
    if one_more:
        den = den + torch.exp(-top)
    return e / den


def shared_key_attention(h, w, m, eps):
    """w: q, k, q.norm, k.norm, o; m: heads, kv_heads, dim, vdim = dim, scale, rot {base, dims}. Values are the raw keys."""
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    T = h.shape[0]
    pos = torch.arange(T)
    raw = (h @ w["k"].T).reshape(T, G, D)
    q, k = rms((h @ w["q"].T).reshape(T, H, D), eps) * w["q.norm"], rms(raw, eps) * w["k.norm"]
    rot = m.get("rot") or dict(base=1.0, dims=0)
    q, k = rotate_half(q, pos, rot["dims"], rot["base"]), rotate_half(k, pos, rot["dims"], rot["base"])
    out = torch.zeros(T, H, D, dtype=F)
    for hd in range(H):
        g = hd // (H // G)
        out[:, hd] = causal_softmax((q[:, hd] @ k[:, g].T) * m["scale"]) @ raw[:, g]
    return out.reshape(T, H * D) @ w["o"].T


def temperature(T, m):
    t = m.get("q_temp")
    if not t:
        return torch.ones(T, dtype=F)
    return torch.tensor([1.0 + t["coef"] * math.log((p + 1) // t["every"] + 1) for p in range(T)], dtype=F)


def distance_bias(T, r1, r2):
    d = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).clamp(min=0).to(F)
    return r1 * torch.log(1.0 + r2 * d)


def distance_attention(h, w, m, eps):
    """w: q, k, v, q.norm, k.norm (whole rows), r1, r2, o; m: heads, kv_heads, dim, vdim, scale, q_temp {coef, every}."""
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = (rms(h @ w["q"].T, eps) * w["q.norm"] * temperature(T, m)[:, None]).reshape(T, H, D)
    k = (rms(h @ w["k"].T, eps) * w["k.norm"]).reshape(T, G, D)
    v = (h @ w["v"].T).reshape(T, G, E)
    out = torch.zeros(T, H, E, dtype=F)
    for hd in range(H):
        g = hd // (H // G)
        s = (q[:, hd] @ k[:, g].T) * m["scale"] - distance_bias(T, w["r1"][hd], w["r2"][hd])
        out[:, hd] = causal_softmax(s, one_more=True) @ v[:, g]
    return out.reshape(T, H * E) @ w["o"].T


def matrix_memory(q, k, v, li, lf):
    """q, k [T, H, D] (q scaled), v [T, H, E], li, lf [T, H] log gates: o [T, H, E]; S and n start at zero, m at zero."""
    T, H, D = q.shape
    S, n, m = torch.zeros(H, D, v.shape[-1], dtype=F), torch.zeros(H, D, dtype=F), torch.zeros(H, dtype=F)
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for t in range(T):
        new = torch.maximum(lf[t] + m, li[t])
        keep, add = torch.exp(lf[t] + m - new), torch.exp(li[t] - new)
        m = new
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = torch.einsum("hde,hd->he", S, q[t]) / den[:, None]
    return out


def log_gates(h, w, cap):
    soft = lambda z: cap * torch.tanh(z / cap)
    return soft(h @ w["i"].T + w["i.b"]), -softplus(-soft(h @ w["f"].T + w["f.b"]))


def memory_mixer(h, w, m, eps):
    """w: q, k, v, i, i.b, f, f.b, g, norm, o; m: heads, dim, vdim, gate_cap."""
    H, D, E = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q, k, v = (h @ w["q"].T).reshape(T, H, D) * D ** -0.5, (h @ w["k"].T).reshape(T, H, D), (h @ w["v"].T).reshape(T, H, E)
    li, lf = log_gates(h, w, m["gate_cap"])
    o = rms(matrix_memory(q, k, v, li, lf), eps).reshape(T, H * E)
    return (o * w["norm"] * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def parallel_mixer(h, w, m, eps):
    return (m["left_scale"] * distance_attention(h, sub(w, "left."), m["left"], eps)
            + m["right_scale"] * memory_mixer(h, sub(w, "right."), m["right"], eps))


def causal_conv(x, weight):
    """x [T, C], weight [C, K] (the last column multiplies the current token); zeros before the sequence."""
    T, C = x.shape
    K = weight.shape[1]
    padded = torch.cat([torch.zeros(K - 1, C, dtype=F), x], 0)
    return sum(padded[j:j + T] * weight[:, j] for j in range(K))


def unit(t):
    return t / torch.sqrt((t * t).sum(-1, keepdim=True) + 1e-6)


def gated_delta(q, k, v, g, b):
    """q, k [T, H, D], v [T, H, E], g, b [T, H]: o [T, H, E]; the state starts at zero."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=F)
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for t in range(T):
        S = g[t][:, None, None] * S
        u = b[t][:, None] * (v[t] - torch.einsum("hde,hd->he", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hde,hd->he", S, q[t])
    return out


def delta_mixer(h, w, m, eps):
    """w: q, k, v, <each>.conv, b, a, dt_bias, A_log, g, norm, o; m: heads, kv_heads, dim, vdim, conv."""
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q, k, v = (silu(causal_conv(h @ w[n].T, w[n + ".conv"])) for n in ("q", "k", "v"))
    q, k = unit(q.reshape(T, G, D)) * D ** -0.5, unit(k.reshape(T, G, D))
    q, k = q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1)
    b = torch.sigmoid(h @ w["b"].T)
    g = torch.exp(-torch.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))
    o = rms(gated_delta(q, k, v.reshape(T, H, E), g, b), eps) * w["norm"]
    return (o.reshape(T, H * E) * silu(h @ w["g"].T)) @ w["o"].T


MIXERS = {"attention": shared_key_attention, "delta": delta_mixer, "parallel": parallel_mixer}


def dense(h, w):
    return gelu(h @ w["up"].T) @ w["down"].T


def expert(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def route(h, router, correction, r):
    """(chosen experts [T, top], weights [T, top]); r: top, scale, groups {count, keep} or none. Ties: the lower index."""
    s = torch.sigmoid(h @ router.T)
    c = s + correction
    T, E = s.shape
    groups = r.get("groups")
    if groups:
        per = c.reshape(T, groups["count"], E // groups["count"])
        rank = torch.sort(per, dim=-1, descending=True).values[..., :2].sum(-1)
        best = torch.sort(rank, dim=-1, descending=True, stable=True).indices[:, :groups["keep"]]
        stay = torch.zeros(T, groups["count"], dtype=torch.bool)
        stay.scatter_(1, best, True)
        c = c.masked_fill(~stay.repeat_interleave(E // groups["count"], 1), float("-inf"))
    chosen = torch.sort(c, dim=-1, descending=True, stable=True).indices[:, :r["top"]]
    weight = torch.gather(s, 1, chosen)
    return chosen, weight / (weight.sum(-1, keepdim=True) + 1e-20) * r.get("scale", 1.0)


def experts(h, w, r):
    """w: router, correction, e<i>.gate / up / down, shared.gate / up / down / sg."""
    chosen, weight = route(h, w["router"], w["correction"], r)
    out = torch.zeros(h.shape[0], w["e0.down"].shape[0], dtype=F)
    for e in range(r["experts"]):
        rows, col = (chosen == e).nonzero(as_tuple=True)
        if rows.numel():
            out[rows] += weight[rows, col][:, None] * expert(h[rows], sub(w, f"e{e}."))
    if "shared.gate" in w:
        out = out + torch.sigmoid(h @ w["shared.sg"].T) * expert(h, sub(w, "shared."))
    return out


def feed_forward(h, w, mlp):
    return dense(h, w) if mlp["kind"] == "dense" else experts(h, w, mlp["router"])


def depth_average(states, weights):
    return sum(a * X for a, X in zip(weights, states))


def sub(tensors, prefix):
    return {k[len(prefix):]: v.to(F) for k, v in tensors.items() if k.startswith(prefix)}


def forward(cfg, tensors, tokens, layers_out=None, round_to=None):
    """Logits [T, vocab] of one sequence from position 0. cfg: the config.json dictionary; tensors: name -> tensor.
    layers_out (a list): the residual rows after every layer (averaged over the depth) are appended.
    round_to (a dtype, or a function): every sublayer's input and result are rounded to it; the difference to the exact
    logits measures how sensitive each position is to rounding."""
    rd = (lambda t: t) if round_to is None else round_to if callable(round_to) else (lambda t: t.to(round_to).to(F))
    eps = cfg["norm"]["eps"]
    x = tensors["embed"].to(F)[torch.as_tensor(tokens, dtype=torch.long)]
    states = [x]
    for i, L in enumerate(cfg["layers"]):
        t = sub(tensors, f"l{i}.")
        x = x + layer_norm(rd(MIXERS[L["type"]](rd(x), sub(t, "mix."), L["mixer"], eps)), t["norm1"], t["norm1.b"], eps)
        if L.get("mlp") is not None:
            x = x + layer_norm(rd(feed_forward(rd(x), sub(t, "mlp."), L["mlp"])), t["norm2"], t["norm2.b"], eps)
        states.append(x)
        x = depth_average(states, t["dwa"])
        if layers_out is not None:
            layers_out.append(x.clone())
    f = sub(tensors, "final.")
    return layer_norm(x, f["norm"], f["norm.b"], eps) @ tensors["head"].to(F).T
