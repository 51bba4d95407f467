"""The Gakupel decoder as a ModelSpec: a token embedding; layers in the order config.json lists them, each with the norm (a
layer norm with weight and bias) on the sublayer's RESULT only, x <- x + norm1(mixer(x)) and, where the layer has a
feed-forward, x <- x + norm2(ff(x)); what goes on to the next layer (and after the last one to the output) is a learned
average over the embedding rows and every layer's result so far. The mixer is grouped-query attention whose values are the
keys as projected (per-head query and key norms, rotation of part of a head), the gated delta rule with short convolutions,
or two mixers side by side with constant scales: attention without rotation whose score is lowered by the logarithm of the
distance, with a norm over whole query and key rows, a query temperature that grows with the position and a constant sink,
beside the matrix memory of an exponentially gated LSTM. The feed-forward is dense with the exact GELU and no gate, or a
mixture of experts (sigmoid scores with a correction for the choice, chosen within the best groups, renormalised) with a
gated shared expert. The model's norm and an untied head.

Tensor names: embed, final.norm(.b), head, and per layer i under "l<i>.": norm1(.b), norm2(.b), dwa, mix.* (a parallel layer:
mix.left.*, mix.right.*), mlp.up / .down, or mlp.router, mlp.correction, mlp.e<j>.*, mlp.shared.*.
"""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.gakupel import GakupelConfig, GeluFFConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, RunStep


def _mixer_spec(c: GakupelConfig, L) -> PartSpec:
    W, eps, m = c.width, c.norm_eps, L.mixer
    if L.type == "attention":
        return PartSpec("masked_attention", dict(
            hidden_size=W, heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale, eps=eps,
            rot_dims=m.rot.dims, rot_base=m.rot.base, pairing="half", head_norm=True, values="keys"))
    if L.type == "delta":
        return PartSpec("gated_delta", dict(hidden_size=W, heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, conv=m.conv,
                                            eps=eps))
    a, b = m.left, m.right
    left = PartSpec("masked_attention", dict(
        hidden_size=W, heads=a.heads, kv_heads=a.kv_heads, dim=a.dim, vdim=a.vdim, scale=a.scale, eps=eps, rot_dims=0,
        row_norm=True, q_temp=(a.q_temp.coef, a.q_temp.every) if a.q_temp else None, distance_bias=True, sink="one",
        **{k + "_name": "mix.left." + n for k, n in dict(q="q", k="k", v="v", o="o", q_norm="q.norm", k_norm="k.norm", r1="r1",
                                                         r2="r2").items()}))
    right = PartSpec("matrix_memory", dict(
        hidden_size=W, heads=b.heads, dim=b.dim, vdim=b.vdim, gate_cap=b.gate_cap, eps=eps,
        **{k + "_name": "mix.right." + n for k, n in dict(q="q", k="k", v="v", g="g", i="i", i_bias="i.b", f="f", f_bias="f.b",
                                                          norm="norm", o="o").items()}))
    return PartSpec("side_by_side", dict(hidden_size=W, left=left, right=right, join="scaled", left_scale=m.left_scale,
                                         right_scale=m.right_scale))


def _ff_spec(c: GakupelConfig, ff) -> PartSpec:
    if isinstance(ff, GeluFFConfig):
        return PartSpec("activated", dict(hidden_size=c.width, intermediate_size=ff.ff, activation="gelu"))
    return PartSpec("routed", dict(hidden_size=c.width, experts=ff.experts, top=ff.top, expert_size=ff.ff, score="sigmoid_normed",
                                   weight_at="output", groups=ff.groups, weight_scale=ff.scale, shared_size=ff.shared_ff,
                                   shared_gate=True))


def gakupel_spec(c: GakupelConfig) -> ModelSpec:
    W = c.width
    norm = lambda name: PartSpec("layernorm", dict(name=name, size=W, eps=c.norm_eps, bias_name=name + ".b"))
    layers = []
    for i, L in enumerate(c.layers):
        parts = dict(mixer=_mixer_spec(c, L), mixer_norm=norm("norm1"))
        if L.mlp is not None:
            parts.update(feed_forward=_ff_spec(c, L.mlp), feed_forward_norm=norm("norm2"))
        layers.append(LayerSpec(prefix=f"l{i}.", block="output_norm", parts=parts, params=dict(hidden_size=W, average=i + 2)))
    return ModelSpec(
        architecture=c.architecture, hidden_size=W, vocab_size=c.vocab, max_position=c.max_positions,
        embedding=PartSpec("token", dict(name="embed", vocab_size=c.vocab, hidden_size=W)),
        layers=tuple(layers), order=tuple(RunStep(i) for i in range(len(layers))), final_norm=norm("final.norm"),
        head=PartSpec("linear", dict(name="head", vocab_size=c.vocab, hidden_size=W)), eos_token_ids=c.eos_token_ids)


register_architecture("Gakupel", GakupelConfig, gakupel_spec)
