"""The Selovik decoder as a ModelSpec: a scaled token embedding plus a bigram embedding, normed; layers in the order config.json
lists them, each with two norms of the same rows, one read by differential attention with rotation (YaRN scaling), a sliding
window and an output gate, the other by the feed-forward, x <- x + (mixer(norm1(x)) + ff(norm2(x))); a run of neighbouring
layers is gone through several times with the same weights, every pass with caches of its own, starting with a vector per pass
and, from the second pass on, the embedding rows added once more. The feed-forward is dense with the square of relu, or a
mixture of experts (softmax scores with a correction for the choice, chosen within the groups whose best expert is best, not
renormalised, some experts being the identity) with a shared expert. RMS norms with weights stored around zero; the head is the
embedding table, its logits scaled.

Tensor names: embed, bigram, embed.norm, loop.step, final.norm, and per layer i under "l<i>.": norm1, norm2, mix.q / .k / .v /
.g / .o / .lq1 / .lk1 / .lq2 / .lk2, mlp.up / .down, or mlp.router, mlp.correction, mlp.e<j>.*, mlp.shared.*.
"""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.selovik import SelovikConfig, SquaredReluFFConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, RunStep


def _mixer_spec(c: SelovikConfig, m) -> PartSpec:
    scaling = dict(m.rot.scaling_dict(), kind="yarn") if m.rot.scaling else None
    return PartSpec("differential_attention", dict(
        hidden_size=c.width, heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale, diff=m.diff, eps=c.norm_eps,
        window=m.window, biases=False, rot_dims=m.rot.dims, rot_base=m.rot.base, rot_scaling=scaling))


def _ff_spec(c: SelovikConfig, ff) -> PartSpec:
    if isinstance(ff, SquaredReluFFConfig):
        return PartSpec("activated", dict(hidden_size=c.width, intermediate_size=ff.ff, activation="relu2"))
    return PartSpec("routed", dict(hidden_size=c.width, experts=ff.experts, identity=ff.identity, top=ff.top, expert_size=ff.ff,
                                   score="softmax", weight_at="output", groups=ff.groups, shared_size=ff.shared_ff))


def selovik_spec(c: SelovikConfig) -> ModelSpec:
    W = c.width
    norm = lambda name, **kw: PartSpec("rmsnorm", dict(name=name, size=W, eps=c.norm_eps, one_plus=True, **kw))
    layers = []
    for i, L in enumerate(c.layers):
        parts = dict(mixer_norm=norm("norm1"), mixer=_mixer_spec(c, L.mixer))
        if L.mlp is not None:
            parts.update(feed_forward_norm=norm("norm2"), feed_forward=_ff_spec(c, L.mlp))
        layers.append(LayerSpec(prefix=f"l{i}.", block="parallel_two_norms", parts=parts))
    return ModelSpec(
        architecture=c.architecture, hidden_size=W, vocab_size=c.vocab, max_position=c.max_positions,
        embedding=PartSpec("token_bigram", dict(name="embed", vocab_size=c.vocab, hidden_size=W, scale=c.embedding_scale,
                                                bigram=c.bigram, norm=norm("embed.norm"))),
        layers=tuple(layers), order=tuple(RunStep(i, enters_pass=t) for i, t in c.run_order()),
        # the head is linear: the logits' scale multiplies its input, in the norm's 32-bit weight
        final_norm=norm("final.norm", gain=c.logit_scale), head=PartSpec("linear", dict(tied_to="embed", vocab_size=c.vocab, hidden_size=W)),
        pass_entry=None if c.loop is None else PartSpec("loop", dict(name="loop.step", passes=c.loop.times, hidden_size=W)),
        eos_token_ids=c.eos_token_ids)


register_architecture("Selovik", SelovikConfig, selovik_spec)
