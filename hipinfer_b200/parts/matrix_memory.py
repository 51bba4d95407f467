"""The matrix memory of an exponentially gated LSTM (mLSTM): a linear recurrence with one state matrix per head, a normaliser
beside it and a running maximum that keeps the exponential gates in range.

For each head, with S [dim, vdim], n [dim] and m that start at zero and are carried from token to token in 32-bit:

    q, k, v = Wq h / sqrt(dim), Wk h, Wv h                      (heads x dim, heads x dim, heads x vdim)
    li = cap tanh((Wi h + bi) / cap);   lf = log sigmoid(cap tanh((Wf h + bf) / cap))
    m' = max(lf + m, li)
    S <- exp(lf + m - m') S + exp(li - m') k v^T;   n <- exp(lf + m - m') n + exp(li - m') k
    o = S^T q / (max(|n . q|, exp(-m')) + den_eps)

then o of each head is divided by its root mean square (eps inside the root), the heads are concatenated, multiplied by a
weight vector and by sigmoid(Wg h), and projected by Wo. All projections that read h are one product whose 32-bit result
feeds the recurrence directly; gates, the running maximum, the state and the head norm are 32-bit (csrc/matrix_state.cu).
A request's state slot holds S, n and m (`state_need`), zeroed at admission; there is no cache.

params: hidden_size, heads, dim, vdim, gate_cap, eps, den_eps (default 1e-6), and the tensor names q, k, v, g, i, i_bias, f,
f_bias, norm, o (`<key>_name`, relative to the prefix).
"""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights import ParamSpec
from . import planes
from .registry import Mixer, register_part, to_compute

_DEFAULT_NAMES = dict(q="mix.q", k="mix.k", v="mix.v", g="mix.g", i="mix.i", i_bias="mix.i.b", f="mix.f", f_bias="mix.f.b",
                      norm="mix.norm", o="mix.o")


class MatrixMemoryMixer(Mixer):
    def __init__(self, params, ctx, prefix=""):
        super().__init__(params, ctx, prefix)
        p = params
        self.hidden, self.heads, self.dim, self.vdim = int(p["hidden_size"]), int(p["heads"]), int(p["dim"]), int(p["vdim"])
        self.cap, self.eps, self.den_eps = float(p["gate_cap"]), float(p["eps"]), float(p.get("den_eps", 1e-6))
        self.names = {k: prefix + p.get(k + "_name", d) for k, d in _DEFAULT_NAMES.items()}
        self.w_in = self.wo = None

    def param_specs(self):
        n, W, HD, HP, H = self.names, self.hidden, self.heads * self.dim, self.heads * self.vdim, self.heads
        return [ParamSpec(n["q"], (HD, W)), ParamSpec(n["k"], (HD, W)), ParamSpec(n["v"], (HP, W)), ParamSpec(n["g"], (HP, W)),
                ParamSpec(n["i"], (H, W)), ParamSpec(n["i_bias"], (H,), init="zeros"), ParamSpec(n["f"], (H, W)),
                ParamSpec(n["f_bias"], (H,), init="zeros"), ParamSpec(n["norm"], (HP,), init="ones"), ParamSpec(n["o"], (W, HP))]

    def load(self, tensors):
        t = {k: to_compute(tensors[n], self.ctx) for k, n in self.names.items()}
        mats = [t[k] for k in ("q", "k", "v", "g", "i", "f")]
        dt = mats[0].dtype if all(m.dtype == mats[0].dtype for m in mats) else torch.float32
        self.w_in = ops.Weight(torch.cat([m.to(dt) for m in mats], 0).contiguous())     # rows [q | k | v | g | i | f]
        self.wo, self.norm_w = ops.Weight(t["o"]), t["norm"]
        self.b_i, self.b_f = t["i_bias"], t["f_bias"].to(t["i_bias"].dtype)

    def weight_bytes(self):
        return self.w_in.nbytes + self.wo.nbytes + self.norm_w.numel() * self.norm_w.element_size()

    def state_need(self):
        return {"S": ((self.heads, self.dim, self.vdim), torch.float32), "n": ((self.heads, self.dim), torch.float32),
                "m": ((self.heads,), torch.float32)}

    def forward(self, xn, x, batch, cache, state):
        T, H, HD, HP, dev = xn.shape[0], self.heads, self.heads * self.dim, self.heads * self.vdim, xn.device
        proj = torch.empty(T, 2 * HD + 2 * HP + 2 * H, dtype=torch.float32, device=dev)
        ops.linear_rows32(xn, self.w_in, proj)
        q, k, v, g, zi, zf = torch.split(proj, [HD, HD, HP, HP, H, H], 1)
        out = torch.empty(T, HP, dtype=self.ctx.dtype, device=dev)
        if not ops.ms_single(q, k, v, zi, zf, self.b_i, self.b_f, state["S"], self.norm_w, g, "sigmoid", out, batch, self.dim ** -0.5,
                             self.eps, state["n"], state["m"], self.cap, self.den_eps):
            a, b, e = ops.ms_exp_gates(zi, zf, self.b_i, self.b_f, self.cap, state["m"], batch)
            y = torch.empty(T, HP, dtype=torch.float32, device=dev)
            nq = torch.empty(T, H, dtype=torch.float32, device=dev)
            ops.ms_walk(q, k, v, a, b, state["S"], batch, y, self.dim ** -0.5, nstate=state["n"], nq=nq)
            ops.ms_finish(y, self.norm_w, g, "sigmoid", out, H, self.eps, nq, e, self.den_eps)
        planes.record(batch, "attention", out)
        ops.linear_into_stream(out, self.wo, x)
        return None


register_part("mixer", "matrix_memory", MatrixMemoryMixer)
