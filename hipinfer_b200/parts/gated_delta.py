"""The gated delta-rule mixer: a recurrence with one state matrix per head, a scalar decay per head and token, and a write
that replaces what the state holds under the token's key.

For each head h (query/key head h // (heads / kv_heads)), with a state S [dim, vdim] that starts at zero and is carried from
token to token in 32-bit:

    q, k, v = silu(conv(Wq h)), silu(conv(Wk h)), silu(conv(Wv h))       causal, `conv` taps a channel, no bias
    q, k to unit length: x / sqrt(sum x^2 + unit_eps); q also times dim^(-1/2)
    beta = sigmoid(Wb h);  g = exp(-exp(A_log) softplus(Wa h + dt_bias))   one number per head
    S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q

then o of each head is divided by its root mean square over vdim (eps inside the root), multiplied by a weight shared by the
heads and by silu(Wg h), and projected by Wo. All projections that read h are one product whose 32-bit result feeds the
convolution and the recurrence directly; decays, write strengths, unit keys, the state and the head norm are 32-bit
(csrc/matrix_state.cu, ssd.cu). A request's state slot holds S and the last `conv` - 1 raw inputs of the convolution.

params: hidden_size, heads, kv_heads, dim, vdim, conv, eps, unit_eps (default 1e-6), and the tensor names q, k, v, q_conv, k_conv,
v_conv, b, a, dt_bias, a_log, g, norm, o (`<key>_name`, relative to the prefix).
"""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights import ParamSpec
from . import planes
from .registry import Mixer, register_part, to_compute

_DEFAULT_NAMES = dict(q="mix.q", k="mix.k", v="mix.v", q_conv="mix.q.conv", k_conv="mix.k.conv", v_conv="mix.v.conv", b="mix.b",
                      a="mix.a", dt_bias="mix.dt_bias", a_log="mix.A_log", g="mix.g", norm="mix.norm", o="mix.o")


class GatedDeltaMixer(Mixer):
    def __init__(self, params, ctx, prefix=""):
        super().__init__(params, ctx, prefix)
        p = params
        self.hidden, self.heads, self.kv_heads = int(p["hidden_size"]), int(p["heads"]), int(p["kv_heads"])
        self.dim, self.vdim, self.taps = int(p["dim"]), int(p["vdim"]), int(p["conv"])
        if self.heads % self.kv_heads:
            raise ValueError(f"gated delta rule: {self.heads} heads are not a multiple of {self.kv_heads} query/key heads")
        self.eps, self.unit_eps = float(p["eps"]), float(p.get("unit_eps", 1e-6))
        self.n_qk, self.n_v = self.kv_heads * self.dim, self.heads * self.vdim
        self.channels = 2 * self.n_qk + self.n_v
        self.names = {k: prefix + p.get(k + "_name", d) for k, d in _DEFAULT_NAMES.items()}
        self.w_in = self.wo = None

    def param_specs(self):
        n, W, H, K = self.names, self.hidden, self.heads, self.taps
        return [ParamSpec(n["q"], (self.n_qk, W)), ParamSpec(n["q_conv"], (self.n_qk, K)), ParamSpec(n["k"], (self.n_qk, W)),
                ParamSpec(n["k_conv"], (self.n_qk, K)), ParamSpec(n["v"], (self.n_v, W)), ParamSpec(n["v_conv"], (self.n_v, K)),
                ParamSpec(n["b"], (H, W)), ParamSpec(n["a"], (H, W)), ParamSpec(n["dt_bias"], (H,), init="zeros"),
                ParamSpec(n["a_log"], (H,), init="zeros"), ParamSpec(n["g"], (self.n_v, W)),
                ParamSpec(n["norm"], (self.vdim,), init="ones"), ParamSpec(n["o"], (W, self.n_v))]

    def load(self, tensors):
        t = {k: to_compute(tensors[n], self.ctx) for k, n in self.names.items()}
        mats = [t[k] for k in ("q", "k", "v", "g", "a", "b")]
        dt = mats[0].dtype if all(m.dtype == mats[0].dtype for m in mats) else torch.float32
        self.w_in = ops.Weight(torch.cat([m.to(dt) for m in mats], 0).contiguous())     # rows [q | k | v | g | a | b]
        self.wo, self.norm_w = ops.Weight(t["o"]), t["norm"]
        convs = [t[k] for k in ("q_conv", "k_conv", "v_conv")]
        cdt = convs[0].dtype if all(c.dtype == convs[0].dtype for c in convs) else torch.float32
        self.conv_w = torch.cat([c.to(cdt) for c in convs], 0).contiguous()
        self.conv_b = torch.zeros(self.channels, dtype=cdt, device=self.conv_w.device)
        self.dt_bias, self.a_log = t["dt_bias"], t["a_log"].to(t["dt_bias"].dtype)

    def weight_bytes(self):
        return self.w_in.nbytes + self.wo.nbytes + self.conv_w.numel() * self.conv_w.element_size()

    def state_need(self):
        return {"S": ((self.heads, self.dim, self.vdim), torch.float32), "conv": ((self.taps - 1, self.channels), torch.float32)}

    def forward(self, xn, x, batch, cache, state):
        T, H, C, dev = xn.shape[0], self.heads, self.channels, xn.device
        proj = torch.empty(T, C + self.n_v + 2 * H, dtype=torch.float32, device=dev)
        ops.linear_rows32(xn, self.w_in, proj)
        g, za, zb = torch.split(proj[:, C:], [self.n_v, H, H], 1)
        qkv = torch.empty(T, C, dtype=torch.float32, device=dev)
        ops.ssd_conv(proj, 0, self.conv_w, self.conv_b, state["conv"], batch, qkv)
        q, k, v = torch.split(qkv, [self.n_qk, self.n_qk, self.n_v], 1)
        out = torch.empty(T, self.n_v, dtype=self.ctx.dtype, device=dev)
        if not ops.ms_single(q, k, v, za, zb, self.dt_bias, self.a_log, state["S"], self.norm_w, g, "silu", out, batch, self.dim ** -0.5,
                             self.eps, unit_eps=self.unit_eps):
            scal = ops.ms_delta_prepare(q, k, za, zb, self.a_log, self.dt_bias, batch, self.dim, self.dim ** -0.5, self.unit_eps)
            y = torch.empty(T, self.n_v, dtype=torch.float32, device=dev)
            ops.ms_delta_walk(q, k, v, scal, state["S"], batch, y)
            ops.ms_finish(y, self.norm_w, g, "silu", out, H, self.eps)
        planes.record(batch, "attention", out)
        ops.linear_into_stream(out, self.wo, x)
        return None


register_part("mixer", "gated_delta", GatedDeltaMixer)
