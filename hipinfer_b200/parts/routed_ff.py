"""A routed feed-forward (mixture of experts): E small gated feed-forward layers without biases, of which every token
runs `top`.

    s = sigmoid(Wr h)                             router scores, 32-bit sums
    the `top` largest s choose the experts (ties: the lower index); the weights are the chosen scores, not renormalised
    out = sum over the chosen e of Wdown_e (silu(Wgate_e v) * (Wup_e v)),  v = s_e h     the score multiplies the INPUT

Without biases Wgate_e (s h) = s (Wgate_e h): the products run on h and the score enters the activation in 32-bit.

A second form is chosen by parameters: `router_bias` adds a bias to the router's logits; `score` "softmax_chosen" lets the
`top` largest LOGITS choose and takes as weights the softmax over the chosen logits alone; `weight_at` "output" multiplies
the expert's RESULT by the weight (brought in at the activation too: the down product is linear).
A third: `score` "sigmoid_normed" chooses by sigmoid(z) + a correction per expert, where `groups` (count, keep) is given
only within the `keep` groups of neighbouring experts that rank best by the sum of their two largest; the weights are the
chosen sigmoid(z), without the correction, over their sum, times `weight_scale`.

A fourth: `score` "softmax" chooses by softmax(z) over all experts + the correction, where `groups` is given only within the
`keep` groups that rank best by their LARGEST; the weights are the chosen softmax(z) as they are.
With `identity` the last that many of the experts + identity router rows are experts without tensors whose result is h itself
(times the weight; kinds of score that are not normalised). Groups are formed over all of them together.

With `shared_size` a shared expert of the same form and that size runs for every token and is added; with `shared_gate` its
result is multiplied by sigmoid(w . h), one number per token (made beside the router's logits). One without a gate is a gated
feed-forward like any other and runs on its kernels (parts/feed_forward.py).
A step's (row, choice) pairs are sorted by expert, so that an expert's weights are read once for all of its rows, and in
bfloat16 all of it runs on the device alone (csrc/moe.cu, gemm_tc.cu), so that it replays from a CUDA graph: where the experts
have few rows each, warp-MMA kernels stream their weights (gate/up product with its activation, then the down product); where they
have more, two tcgen05 kernels do the same over tiles of 128 rows. In 32-bit (and at sizes those kernels do not take) a few rows
run one by one, single rows of a larger step on any-size kernels, and in a step with prompt portions each expert's block of rows
goes to the ordinary products, for which the host reads the experts' row counts once a layer.

params: hidden_size, experts, top, expert_size, score (default "sigmoid"), weight_at (default "input"), router_bias
(default False), groups (count, keep) (default none), identity (default 0), weight_scale (default 1), shared_size (default none), shared_gate (default
False), router_name (default "mlp.router"), router_bias_name (default "mlp.router.b"), correction_name (default
"mlp.correction"), expert_prefix (default "mlp.e": expert i's tensors are <expert_prefix><i>.gate / .up / .down),
shared_prefix (default "mlp.shared": .gate / .up / .down, and .sg for its gate).
"""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights import ParamSpec
from . import planes
from .feed_forward import GatedFF
from .registry import Part, register_part, to_compute

SORTED_MIN_PAIRS = 64     # fewer (row, choice) pairs than this never go to the ordinary products
TILES_MIN_ROWS = 16       # from this many pairs a choice on, on average, the experts' rows go to the tcgen05 kernels
GROUP = 16                # gate and up rows in turn, as the gated epilogues want them
SHARED_MIN_ROWS = 9       # fewer rows run the shared expert row by row
GROUPED_MIN_PAIRS = 20    # fewer than this run row by row where the grouped kernels are the any-size ones


class RoutedFF(Part):
    def __init__(self, params, ctx, prefix=""):
        super().__init__(params, ctx, prefix)
        self.hidden, self.experts, self.top = int(params["hidden_size"]), int(params["experts"]), int(params["top"])
        self.inter = int(params["expert_size"])
        self.identity = int(params.get("identity") or 0)
        self.choices = self.experts + self.identity          # what the router chooses from
        if not 1 <= self.top <= self.choices:
            raise ValueError(f"routed feed-forward: top {self.top} of {self.choices} experts")
        self.score, self.weight_at = params.get("score", "sigmoid"), params.get("weight_at", "input")
        if self.score not in ops.MOE_SCORES or self.weight_at not in ("input", "output"):
            raise ValueError(f"routed feed-forward: score {self.score!r} (known: {sorted(ops.MOE_SCORES)}), weight_at "
                             f"{self.weight_at!r} (known: 'input', 'output')")
        self.at_output = self.weight_at == "output"
        self.router_name = prefix + params.get("router_name", "mlp.router")
        self.router_bias_name = prefix + params.get("router_bias_name", "mlp.router.b") if params.get("router_bias") else None
        self.router_bias = None
        self.expert_prefix = prefix + params.get("expert_prefix", "mlp.e")
        self.router = self.wgu = self.wdown = self.correction = None
        corrected = self.score in ("sigmoid_normed", "softmax")
        self.correction_name = (prefix + params.get("correction_name", "mlp.correction")) if corrected else None
        self.groups, self.keep = (int(g) for g in (params.get("groups") or (1, 1)))
        self.weight_scale = float(params.get("weight_scale", 1.0))
        if self.choices % self.groups or not 1 <= self.keep <= self.groups or self.keep * (self.choices // self.groups) < self.top:
            raise ValueError(f"routed feed-forward: {self.choices} experts in {self.groups} groups of which {self.keep} stay, "
                             f"{self.top} chosen")
        if self.groups > 1 and not corrected:
            raise ValueError(f"routed feed-forward: groups go with scores 'sigmoid_normed' and 'softmax', not {self.score!r}")
        if self.identity and (self.score not in ("sigmoid", "softmax") or not self.at_output):
            raise ValueError("routed feed-forward: identity experts go with weights that are not normalised, on the experts' results")
        self.shared = int(params.get("shared_size") or 0)
        self.shared_gated = bool(params.get("shared_gate", False)) and self.shared > 0
        self.shared_prefix = prefix + params.get("shared_prefix", "mlp.shared")
        self.shared_gate = self.s_gu = self.s_down = self.index = self.bounds = self.shared_ff = None
        if self.shared and not self.shared_gated:
            self.shared_ff = GatedFF(dict(hidden_size=self.hidden, intermediate_size=self.shared, activation="silu",
                                          **{k + "_name": f"{params.get('shared_prefix', 'mlp.shared')}.{k}" for k in ("gate", "up", "down")}),
                                     ctx, prefix)

    def _expert(self, i, key):
        return f"{self.expert_prefix}{i}.{key}"

    def param_specs(self):
        specs = [ParamSpec(self.router_name, (self.choices, self.hidden))]
        if self.router_bias_name:
            specs.append(ParamSpec(self.router_bias_name, (self.choices,), init="zeros"))
        if self.correction_name:
            specs.append(ParamSpec(self.correction_name, (self.choices,), init="zeros"))
        if self.shared_ff is not None:
            specs += self.shared_ff.param_specs()
        elif self.shared:
            s = self.shared_prefix
            specs += [ParamSpec(s + ".gate", (self.shared, self.hidden)), ParamSpec(s + ".up", (self.shared, self.hidden)),
                      ParamSpec(s + ".down", (self.hidden, self.shared))]
            specs.append(ParamSpec(s + ".sg", (1, self.hidden)))
        for i in range(self.experts):
            specs += [ParamSpec(self._expert(i, "gate"), (self.inter, self.hidden)),
                      ParamSpec(self._expert(i, "up"), (self.inter, self.hidden)),
                      ParamSpec(self._expert(i, "down"), (self.hidden, self.inter))]
        return specs

    def load(self, tensors):
        t = lambda name: to_compute(tensors[name], self.ctx)
        self.router = t(self.router_name)
        if self.router_bias_name:
            self.router_bias = t(self.router_bias_name).to(self.router.dtype).contiguous()
        if self.correction_name:
            self.correction = t(self.correction_name).to(self.router.dtype).contiguous()
        if self.shared_ff is not None:
            self.shared_ff.load(tensors)
        elif self.shared:
            g, u, d = (t(f"{self.shared_prefix}.{k}") for k in ("gate", "up", "down"))
            sdt = g.dtype if g.dtype == u.dtype == d.dtype else torch.float32
            self.s_gu = ops.Weight(torch.cat([g.to(sdt), u.to(sdt)], 0).contiguous())        # gate rows, then up rows
            self.s_down = ops.Weight(d.to(sdt).contiguous())
            self.shared_gate = t(self.shared_prefix + ".sg").to(self.router.dtype).reshape(-1).contiguous()
        mats = [t(self._expert(i, k)) for i in range(self.experts) for k in ("gate", "up", "down")]
        dt = mats[0].dtype if all(m.dtype == mats[0].dtype for m in mats) else torch.float32
        E, F, W = self.experts, self.inter, self.hidden
        G = self.group = GROUP if F % GROUP == 0 else F
        turn = lambda gate, up: torch.stack([gate.to(dt).reshape(F // G, G, W), up.to(dt).reshape(F // G, G, W)], 1).reshape(2 * F, W)
        self.wgu = torch.stack([turn(mats[3 * i], mats[3 * i + 1]) for i in range(E)], 0).contiguous()
        self.wdown = torch.stack([mats[3 * i + 2].to(dt) for i in range(E)], 0).contiguous()      # [E, W, F]
        assert self.wgu.shape == (E, 2 * F, W) and self.wdown.shape == (E, W, F)
        self.w_gu_e = [ops.Weight(self.wgu[i]) for i in range(E)]
        self.w_down_e = [ops.Weight(self.wdown[i]) for i in range(E)]

    def weight_bytes(self):
        """What a single row reads: the router and `top` experts."""
        per = (self.wgu.numel() + self.wdown.numel()) * self.wgu.element_size() // self.experts
        shared = self.shared_ff.weight_bytes() if self.shared_ff else self.s_gu.nbytes + self.s_down.nbytes if self.shared else 0
        return self.router.numel() * self.router.element_size() + self.top * per + shared

    def _row_index(self, T, dev):
        """(0 .. T-1, zeros): a shared expert as the one expert of every row."""
        if self.index is None or self.index[0].numel() < T:
            n = max(T, 2048)
            self.index = (torch.arange(n, dtype=torch.int32, device=dev), torch.zeros(n, 1, dtype=torch.int32, device=dev))
            self.bounds = torch.tensor([[0, t] for t in range(SHARED_MIN_ROWS)], dtype=torch.int32, device=dev)
        return tuple(t[:T] for t in self.index)

    def _add_shared(self, xn, x, weight):
        """x += weight * shared expert: the weight enters at the activation in 32-bit (the down product is linear)."""
        T, F = xn.shape[0], self.shared
        rows, zeros = self._row_index(T, xn.device)
        act = torch.empty(T, F, dtype=self.ctx.dtype, device=xn.device)
        if T < SHARED_MIN_ROWS:
            if ops.moe_grouped_act(xn, rows, 1, self.s_gu.t.unsqueeze(0), self.bounds[T], weight, act, True):
                ops.linear_into_stream(act, self.s_down, x)
                return
            ops.moe_rows(xn, self.s_gu.t.unsqueeze(0), self.s_down.t.unsqueeze(0), zeros, weight, x, True)
            return
        gu = torch.empty(T, 2 * F, dtype=torch.float32, device=xn.device)
        ops.linear(xn, self.s_gu, gu)
        ops.moe_act(gu, rows, weight, act, True)
        ops.linear_into_stream(act, self.s_down, x)

    def forward(self, xn, x, batch):
        T, top, F = xn.shape[0], self.top, self.inter
        shared_weight = torch.empty(T, dtype=torch.float32, device=xn.device) if self.shared_gated else None
        idw = torch.empty(T, dtype=torch.float32, device=xn.device) if self.identity else None
        expert, score = ops.moe_route(xn, self.router, top, self.router_bias, self.score, self.correction, self.groups, self.keep,
                                      self.weight_scale, self.shared_gate, shared_weight, self.identity, idw)
        if self.shared_ff is not None:
            self.shared_ff.forward(xn, x, None)
        elif self.shared:
            self._add_shared(xn, x, shared_weight)
        if T * top < GROUPED_MIN_PAIRS and not ops.moe_grouped_fast(xn, self.wgu, self.wdown):
            ops.moe_rows(xn, self.wgu, self.wdown, expert, score, x, self.at_output, idw, self.group)
            return None
        offsets, pos, src = ops.moe_sort(expert, self.choices)
        # identity experts come last in the order: their sorted rows hold nothing
        limit, rows_in = (offsets[self.experts:], xn) if self.identity else (None, None)
        tiles = self.group == GROUP and ops.moe_sorted_fast(xn, self.wgu, self.wdown)
        if T * top < TILES_MIN_ROWS * self.choices if tiles else getattr(batch, "max_q_len", 1) <= 1 or T * top < SORTED_MIN_PAIRS:
            act = torch.empty(T * top, F, dtype=self.ctx.dtype, device=xn.device)
            if not ops.moe_grouped_act(xn, src, top, self.wgu, offsets, score, act, self.at_output, group=self.group):
                gu = torch.empty(T * top, 2 * F, dtype=torch.float32, device=xn.device)
                ops.moe_grouped(xn, src, top, self.wgu, offsets, gu)
                ops.moe_act(gu, src, score, act, self.at_output, limit, self.group)
            planes.record(batch, "activation", act)
            ys = torch.empty(T * top, self.hidden, dtype=torch.float32, device=xn.device)
            ops.moe_grouped(act, None, 1, self.wdown, offsets, ys)
            ops.moe_combine(ys, pos, x, top, limit, rows_in, idw)
            return None
        xs = ops.moe_gather(xn, src, top, limit)
        act = torch.empty(T * top, F, dtype=self.ctx.dtype, device=xn.device)
        ys = torch.empty(T * top, self.hidden, dtype=torch.float32, device=xn.device)
        if tiles:
            ops.moe_sorted_linear(xs, self.wgu, offsets, act, src, score, self.at_output)
            planes.record(batch, "activation", act)
            ops.moe_sorted_linear(act, self.wdown, offsets, ys)
            ops.moe_combine(ys, pos, x, top, limit, rows_in, idw)
            return None
        bounds = offsets.tolist()                      # the one read by the host: how many rows each expert has
        gu = torch.empty(T * top, 2 * F, dtype=torch.float32, device=xn.device)
        for e in range(self.experts):
            lo, hi = bounds[e], bounds[e + 1]
            if hi > lo:
                ops.linear(xs[lo:hi], self.w_gu_e[e], gu[lo:hi])
        ops.moe_act(gu, src, score, act, self.at_output, limit, self.group)
        planes.record(batch, "activation", act)
        for e in range(self.experts):
            lo, hi = bounds[e], bounds[e + 1]
            if hi > lo:
                ops.linear(act[lo:hi], self.w_down_e[e], ys[lo:hi])
        ops.moe_combine(ys, pos, x, top, limit, rows_in, idw)
        return None


register_part("feed_forward", "routed", RoutedFF)
