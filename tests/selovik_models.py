"""Small Selovik configurations of the tests' own, with weights drawn so that faults show: matrices of unit gain, queries and
keys large enough for single scores to stand out, norm weights away from zero, a bigram table and a step vector per pass as large
as the embedding, corrections (also large negative ones) that move the choice."""
from __future__ import annotations

import json
import math
import os

import torch

import plain_selovik as plain


def yarn(factor, original, fast=32.0, slow=1.0):
    return dict(factor=factor, original=original, fast=fast, slow=slow)


def layer(heads, kv_heads, dim, vdim, window=None, rot_dims=0, base=10000.0, scaling=None, scale=None, diff=0.4, mlp=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale or 1.0 / math.sqrt(dim), diff=diff)
    if rot_dims:
        m["rot"] = dict(base=base, dims=rot_dims)
        if scaling:
            m["rot"]["scaling"] = scaling
    if window:
        m["mask"] = dict(size=window)
    return dict(type="attention", mixer=m, mlp=mlp)


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(ff, experts, top, identity=0, groups=None, shared=None):
    r = dict(experts=experts, top=top)
    if identity:
        r["identity"] = identity
    if groups:
        r["groups"] = dict(count=groups[0], keep=groups[1])
    d = dict(kind="moe", expert=dict(ff=ff), router=r)
    if shared:
        d["shared"] = dict(ff=shared)
    return d


def model(vocab, width, layers, loop=None, bigram=(101, 7, 3), scale=1.0, logit_scale=1.0, eps=1e-5, max_positions=None):
    """loop: (start, stop, times) or None; bigram: (buckets, mul_prev, mul_cur) or None."""
    d = dict(architecture="Selovik", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=scale), logit_scale=logit_scale,
             layers=layers)
    if bigram:
        d["embedding"]["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    if max_positions:
        d["max_positions"] = max_positions
    return d


# A: every kind of feed-forward and none; a window of 24, of one token, wider than a key tile, and none; a rotation of part of a
#    map, of all of it, with and without scaling, and none; six experts and three identity ones in three groups; three passes
A = model(150, 64, [layer(4, 2, 16, 24, 24, 8, scaling=yarn(4.0, 64), mlp=dense(80)),
                    layer(6, 2, 8, 32, 70, 8, base=100.0, diff=0.7, mlp=moe(32, 6, 2, 3, (3, 2), 24)),
                    layer(3, 1, 24, 16, None, 24, scaling=yarn(8.0, 256, 16.0, 2.0), mlp=moe(24, 5, 3, 1)),
                    layer(2, 2, 16, 16, 1), layer(4, 4, 8, 8, 33, diff=-0.2, mlp=moe(40, 4, 1, 0, (2, 1), 8))],
          loop=(1, 3, 3), scale=2.5, logit_scale=0.6, max_positions=700)
# B: the loop is the whole model, one pass twice; every head its own keys; one expert of one; all choices made at once; multipliers
#    whose products need more than 32 bits are of no effect on the row's rule
B = model(97, 48, [layer(3, 3, 8, 8, 17, 4, base=50.0, mlp=moe(40, 1, 1, 3, None, 16)), layer(2, 1, 12, 20, 64, 12, mlp=dense(50)),
                   layer(4, 1, 8, 40, 65, 2, mlp=moe(16, 6, 4, 2, (4, 2)))],
          loop=(0, 3, 2), bigram=(13, 4000000007, 2500000001), scale=0.7, eps=1e-6, max_positions=600)
# C: maps of 32, 64 and 128 with values of 64 and 128 (the warp-MMA kernels); sixteen choices in four groups; a loop at the end
C = model(211, 128, [layer(8, 2, 64, 64, 100, 64, base=500000.0, scaling=yarn(16.0, 300), mlp=moe(64, 12, 4, 4, (4, 2), 64)),
                     layer(4, 1, 32, 128, 63, 16, mlp=dense(256)), layer(2, 2, 128, 64, None, 64, mlp=moe(96, 5, 2, 3, (2, 1), 32)),
                     layer(20, 2, 32, 64, 130, 32, scaling=yarn(2.0, 128, 8.0, 1.0), mlp=moe(64, 3, 2, 1))],
          loop=(2, 4, 2), bigram=(499, 211, 1), scale=4.0, logit_scale=1.7, max_positions=900)
# D: sizes no vectorised kernel takes: a width that is no multiple of 4, maps of 10, 6 and 7; no loop, no bigram table
D = model(90, 50, [layer(2, 1, 10, 6, 20, 6, scaling=yarn(3.0, 100), mlp=moe(30, 3, 2, 1, None, 10)), layer(3, 1, 6, 14, 50, 6, mlp=dense(30)),
                   layer(4, 2, 7, 10, 9, 4, mlp=moe(22, 4, 1, 2, (3, 1), 6)), layer(2, 2, 70, 6)], bigram=None, max_positions=300)
# E: a loop of one pass (its vector is added all the same), a single layer
E = model(64, 32, [layer(2, 1, 16, 16, 40, 16, mlp=moe(32, 4, 2, 2, (3, 2), 16))], loop=(0, 1, 1), max_positions=300)

MODELS = {"a": A, "b": B, "c": C, "d": D, "e": E}
ROUTER_GAIN = 3.0


def _choices(config):
    return max([L["mlp"]["router"]["experts"] + L["mlp"]["router"].get("identity", 0)
                for L in config["layers"] if L.get("mlp") and L["mlp"]["kind"] == "moe"], default=0)


def draw_weights(config: dict, seed: int, dtype=torch.bfloat16):
    """{name: tensor} for `config` from the product's own list of tensors, rounded to `dtype` (so that the engine and the
    plain implementation start from the same numbers).

    With random routers two choices nearly tie at a few positions of every sequence, where inputs that differ by rounding alone
    choose another expert. So the first E channels of the width (E the largest number of choices) carry a code that the
    embedding alone writes (no sublayer, bigram row or step vector does; an identity expert scales all of it alike) and router
    row e reads channel e; `safe_tokens` then leaves out tokens whose calls are close. (Random routers are compared in
    tests/test_gpu_selovik_parts.py, row by row, with the nearly tied rows left out.)"""
    from hipinfer_b200.config import config_from_dict, get_architecture
    from hipinfer_b200.parts.spec import spec_param_specs

    c = config_from_dict(config)
    g = torch.Generator().manual_seed(seed)
    code, W = _choices(config), config["width"]
    out = {}
    for s in spec_param_specs(get_architecture(c.architecture).build_spec(c)):
        n, shape = s.name, tuple(s.shape)
        rnd = torch.randn(shape, generator=g)
        leaf = n.split(".", 1)[1] if n.startswith("l") and n[1].isdigit() else n
        if n == "embed":
            t = rnd * 0.7
            if code:
                for row in t:
                    row[:code] = (torch.randperm(code, generator=g) / (code - 1.0) * 2.0 - 1.0) if code > 1 else 1.0
        elif n == "bigram":
            t = rnd * 0.7 * config["embedding"]["scale"]
        elif n == "loop.step":
            t = rnd * 0.7
        elif leaf in ("mix.lq1", "mix.lk1", "mix.lq2", "mix.lk2"):
            t = rnd * 0.5 / shape[0] ** 0.25
        elif leaf == "mlp.router":
            t = torch.zeros(shape)
            t[:, :shape[0]] = ROUTER_GAIN * torch.eye(shape[0])
        elif leaf == "mlp.correction":
            t = 0.15 * rnd - 0.3                                    # choice scores of both signs
        elif leaf in ("mix.q", "mix.k"):
            t = rnd * (1.6 / math.sqrt(shape[1]))                   # single keys stand out
        elif len(shape) == 2:
            t = rnd * (1.2 / math.sqrt(shape[1]))
        else:                                                       # norm weights, around zero
            t = 0.3 * rnd
        if code and n == "bigram" or n == "loop.step":
            t[:, :code] = 0.0
        elif code and (leaf == "mix.o" or leaf.endswith(".down")):
            t[:code] = 0.0
        elif code and (leaf == "norm2" or n == "embed.norm"):
            t[:code] = 0.0
        out[n] = t.to(dtype)
    return out


def safe_tokens(cfg, weights, n, seed, margin=0.012, rounds=40):
    """n random tokens none of whose router calls is closer than `margin`; tokens with a close call are drawn again until there
    are none (a token moves later ones' calls a little, so more than one round may be needed)."""
    g = torch.Generator().manual_seed(seed)
    toks = torch.randint(0, cfg["vocab"], (n,), generator=g)
    if not _choices(cfg):
        return toks.tolist()
    for _ in range(rounds):
        calls = []
        plain.forward(cfg, weights, toks.tolist(), calls=calls)
        bad = torch.stack(calls).amin(0) < margin
        if not bool(bad.any()):
            return toks.tolist()
        toks[bad] = torch.randint(0, cfg["vocab"], (int(bad.sum()),), generator=g)
    raise AssertionError("no tokens without a close call were found")


def make_folder(folder, which, seed=1, dtype=torch.bfloat16):
    from hipinfer_b200.weights.safetensors_io import save_safetensors

    cfg = MODELS[which] if isinstance(which, str) else which
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    w = draw_weights(cfg, seed, dtype)
    save_safetensors(w, os.path.join(folder, "model.safetensors"), {"format": "pt"})
    return str(folder), cfg, w


def sensitivity(cfg, weights, tokens, ref=None):
    """Per position, how far the plain logits move (largest difference over the vocabulary, over the largest logit) when every
    sublayer's input and result are rounded to bfloat16: large where the two maps nearly cancel before the head's norm."""
    ref = plain.forward(cfg, weights, tokens) if ref is None else ref.double()
    err = (plain.forward(cfg, weights, tokens, round_to=lambda t: t.to(torch.bfloat16).double()) - ref).abs().amax(-1)
    return (err / ref.abs().max()).float()
