"""Small Gakupel configurations of the tests' own, with weights drawn so that faults show: matrices of unit gain, decays and
gates from nearly closed to nearly open, distance biases that matter within a page, norm weights away from one, router
corrections (also large negative ones) that move the choice, depth weights of both signs."""
from __future__ import annotations

import json
import math
import os

import torch

import plain_gakupel as plain


def attention(heads, kv_heads, dim, rot_dims=0, base=10000.0, scale=None, mlp=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=scale or 1.0 / math.sqrt(dim))
    if rot_dims:
        m["rot"] = dict(base=base, dims=rot_dims)
    return dict(type="attention", mixer=m, mlp=mlp)


def delta(heads, kv_heads, dim, vdim, conv, mlp=None):
    return dict(type="delta", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv), mlp=mlp)


def parallel(left, right, left_scale=0.7, right_scale=0.8, mlp=None):
    """left: (heads, kv_heads, dim, vdim[, coef, every]); right: (heads, dim, vdim, gate_cap)."""
    H, G, D, E = left[:4]
    a = dict(heads=H, kv_heads=G, dim=D, vdim=E, scale=1.0 / math.sqrt(D))
    if len(left) > 4:
        a["q_temp"] = dict(coef=left[4], every=left[5])
    b = dict(zip(("heads", "dim", "vdim", "gate_cap"), right))
    return dict(type="parallel", mixer=dict(left=a, right=b, left_scale=left_scale, right_scale=right_scale), mlp=mlp)


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(ff, experts, top, groups=None, scale=1.0, shared=None):
    r = dict(experts=experts, top=top, scale=scale)
    if groups:
        r["groups"] = dict(count=groups[0], keep=groups[1])
    d = dict(kind="moe", expert=dict(ff=ff), router=r)
    if shared:
        d["shared"] = dict(ff=shared)
    return d


def model(vocab, width, layers, eps=1e-5, max_positions=None):
    d = dict(architecture="Gakupel", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)
    if max_positions:
        d["max_positions"] = max_positions
    return d


# A: every kind of layer and feed-forward; more value heads than query/key heads in both attentions and in the delta rule;
#    six experts in three groups of two; a layer without a feed-forward; a temperature that steps every 10 positions
A = model(150, 64, [parallel((4, 2, 16, 24, 0.4, 10), (3, 16, 8, 12.0), mlp=moe(32, 6, 2, (3, 2), 1.7, 24)),
                    attention(6, 2, 16, rot_dims=8, mlp=dense(80)),
                    delta(4, 2, 16, 24, 4, mlp=moe(24, 5, 2, None, 2.5, 40)),
                    parallel((3, 1, 24, 16, 0.7, 33), (2, 24, 40, 8.0), left_scale=-0.5, right_scale=1.3)], max_positions=700)
# B: the delta rule first, one tap (no carried inputs) and seven; every head its own; no rotation, no temperature, no shared
#    expert, one expert of one; gate caps that bind; four groups of which one stays
B = model(97, 48, [delta(3, 3, 8, 8, 1, mlp=moe(40, 1, 1)), attention(3, 3, 8, mlp=moe(16, 8, 2, (4, 1), 0.5)),
                   parallel((2, 2, 8, 8), (4, 8, 16, 1.5), mlp=dense(50)), delta(2, 1, 24, 8, 7), attention(2, 1, 24, rot_dims=24, base=100.0)],
          eps=1e-6, max_positions=600)
# C: heads of 64, 96 and 128 (the tensor-core kernels, one of their sizes only in part); sixteen experts in four groups
C = model(211, 128, [parallel((8, 2, 64, 64, 0.2, 100), (2, 64, 64, 15.0), mlp=moe(64, 16, 4, (4, 2), 1.3, 64)),
                     attention(4, 1, 128, rot_dims=64, mlp=dense(256)), delta(2, 2, 64, 128, 3, mlp=dense(96)),
                     parallel((4, 4, 96, 96, 0.25, 48), (2, 96, 32, 15.0), mlp=moe(96, 4, 2, (2, 1), 1.0, 32)),
                     attention(20, 1, 32, rot_dims=16)], max_positions=900)
# D: sizes no vectorised kernel takes: a width that is no multiple of 4, heads of 10, 6 and 7
D = model(90, 50, [attention(2, 1, 10, rot_dims=6, mlp=moe(30, 3, 2, None, 1.0, 10)),
                   parallel((3, 1, 10, 6, 0.5, 7), (2, 7, 10, 10.0), mlp=dense(30)), delta(4, 2, 6, 14, 5, mlp=moe(22, 6, 1, (2, 1), 2.0, 6)),
                   delta(2, 2, 70, 6, 2)], max_positions=300)

MODELS = {"a": A, "b": B, "c": C, "d": D}


def _routers(config):
    return [L["mlp"]["router"] for L in config["layers"] if L.get("mlp") and L["mlp"]["kind"] == "moe"]


ROUTER_GAIN = 2.5


def _margin(levels, corrections, r):
    """How far the closest call of a router is from going the other way, for a row whose first channels hold `levels`."""
    E, g = r["experts"], r.get("groups") or dict(count=1, keep=1)
    c = torch.sigmoid(ROUTER_GAIN * levels[:E]) + corrections
    m = math.inf
    if g["keep"] < g["count"]:
        per = torch.sort(c.reshape(g["count"], -1), dim=-1, descending=True).values[:, :2].sum(-1)
        order = torch.sort(per, descending=True)
        m = min(m, float(order.values[g["keep"] - 1] - order.values[g["keep"]]))
        stay = torch.zeros(g["count"], dtype=torch.bool)
        stay[order.indices[:g["keep"]]] = True
        c = c[stay.repeat_interleave(E // g["count"])]
    c = torch.sort(c, descending=True).values
    if c.numel() > r["top"]:                                   # the order among the chosen decides nothing; the last one does
        m = min(m, float(c[r["top"] - 1] - c[r["top"]]))
    return m


def draw_weights(config: dict, seed: int, dtype=torch.bfloat16):
    """{name: tensor} for `config` from the product's own list of tensors, rounded to `dtype` (so that the engine and the
    plain implementation start from the same numbers).

    With random routers two choices nearly tie at a few positions of every sequence; inputs that differ by rounding alone
    then choose another expert, and a recurrent layer carries the difference to every later position. So the first E
    channels of the width (E the largest number of experts) carry a code that only the embedding writes: the norms after the
    sublayers have zero weight and bias there, the depth weights of a layer sum to one, and router row e reads channel e
    alone. A token's code is drawn again until no router's choice, of a group or of an expert, is a close call. (Random
    routers are compared in tests/test_gpu_gakupel_parts.py, row by row, with the nearly tied rows left out.)"""
    from hipinfer_b200.config import config_from_dict, get_architecture
    from hipinfer_b200.parts.spec import spec_param_specs

    c = config_from_dict(config)
    g = torch.Generator().manual_seed(seed)
    routers = _routers(config)
    code = max([r["experts"] for r in routers], default=0)
    out, corrections = {}, []
    for s in spec_param_specs(get_architecture(c.architecture).build_spec(c)):
        n, shape = s.name, tuple(s.shape)
        rnd = torch.randn(shape, generator=g)
        leaf = n.split(".", 1)[1] if n.startswith("l") and "." in n else n
        if n == "embed":
            t = rnd * 0.7
        elif leaf == "dwa":
            t = 0.4 * rnd
            t[-1] = 0.8
            t = t / t.sum() if float(t.sum()) > 0.3 else torch.cat([t[:-1] * 0.0, torch.ones(1)])
        elif leaf.endswith("A_log"):
            t = torch.rand(shape, generator=g) * 4.0 - 3.0          # decays from exp(-0.05 dt) to exp(-2.7 dt)
        elif leaf.endswith("dt_bias"):
            t = 0.7 * rnd - 1.0
        elif leaf.endswith(".f.b"):
            t = 2.0 + 1.5 * rnd                                     # forget gates mostly open
        elif leaf.endswith(".i.b"):
            t = 1.5 * rnd
        elif leaf.endswith(".r1"):
            t = 0.2 + rnd.abs()
        elif leaf.endswith(".r2"):
            t = 0.05 + 0.5 * rnd.abs()
        elif leaf.endswith(".conv"):
            t = 0.6 * rnd
        elif leaf == "mlp.router":
            t = torch.zeros(shape)
            t[:, :shape[0]] = ROUTER_GAIN * torch.eye(shape[0])
        elif leaf == "mlp.correction":
            t = 0.5 * rnd - 0.6                                     # choice scores of both signs
            corrections.append(t.to(dtype).float())
        elif len(shape) == 2:
            t = rnd * (1.2 / math.sqrt(shape[1]))
        elif leaf in ("norm1.b", "norm2.b") or n == "final.norm.b":
            t = 0.2 * rnd
        else:                                                       # norm weights
            t = 1.0 + 0.3 * rnd
        if code and leaf in ("norm1", "norm2", "norm1.b", "norm2.b"):
            t[:code] = 0.0
        out[n] = t.to(dtype)
    if code:
        embed = out["embed"].float()
        for tok in range(embed.shape[0]):
            best, best_m = None, -1.0
            for _ in range(60):
                levels = (torch.randperm(code, generator=g) + 0.5) * (2.0 / code) + 0.3 * torch.rand(code, generator=g) - 0.5
                m = min(_margin(levels, cr, r) for cr, r in zip(corrections, routers))
                if m > best_m:
                    best, best_m = levels, m
                if m > 0.04:
                    break
            embed[tok, :code] = best
        out["embed"] = embed.to(dtype)
    return out


def make_folder(folder, which, seed=1, dtype=torch.bfloat16):
    from hipinfer_b200.weights.safetensors_io import save_safetensors

    cfg = MODELS[which] if isinstance(which, str) else which
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    w = draw_weights(cfg, seed, dtype)
    save_safetensors(w, os.path.join(folder, "model.safetensors"), {"format": "pt"})
    return str(folder), cfg, w


class PlainGakupel:
    """The plain implementation with the interface the engine tests use: logits of every position of a sequence; a call
    continues the sequence of the calls before it (by running the whole sequence again), `reset` starts a new one."""

    def __init__(self, cfg, weights):
        self.cfg, self.w, self.tokens = cfg, weights, []

    def reset(self):
        self.tokens = []

    def forward(self, tokens):
        n = len(self.tokens)
        self.tokens = self.tokens + list(tokens)
        return plain.forward(self.cfg, self.w, self.tokens)[n:].float()


def sensitivity(cfg, weights, tokens, ref=None, dtype="bfloat16"):
    """Per position, how far the plain logits move (largest difference over the vocabulary, over the largest logit) when
    every sublayer's input and result are rounded to bfloat16, or (dtype "float32") when the plain implementation itself runs
    in 32-bit: large where a norm divides by nearly nothing or sums cancel (a first token whose query and key are nearly
    orthogonal reads out nearly nothing, which the head's norm then makes large; a query nearly orthogonal to the memory's
    normaliser, whose read-out changes its sign). For bfloat16 the largest of that and of a quarter of what noise of four times
    the size does, in a few draws: such a point may lie just beyond one draw of rounding."""
    ref = plain.forward(cfg, weights, tokens) if ref is None else ref.double()
    if dtype == "bfloat16":
        err = (plain.forward(cfg, weights, tokens, round_to=torch.bfloat16) - ref).abs().amax(-1)
        g = torch.Generator().manual_seed(5)
        for _ in range(4):
            noisy = lambda t: t * (1.0 + (torch.rand(t.shape, generator=g, dtype=torch.float64) - 0.5) * 2.0 ** -6)
            err = torch.maximum(err, (plain.forward(cfg, weights, tokens, round_to=noisy) - ref).abs().amax(-1) / 4)
    else:
        plain.F = torch.float32
        try:
            err = (plain.forward(cfg, weights, tokens).double() - ref).abs().amax(-1)
        finally:
            plain.F = torch.float64
    return (err / ref.abs().max()).float()
