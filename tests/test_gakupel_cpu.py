"""The Gakupel design without a GPU: its configuration, its description as parts, the cache and state plan the decoder
derives from it, and the plain implementation against hand-made cases (both recurrences against their unrolled sums, the
running maximum, the temperature's steps, the bias, the router's groups, the average over the depth)."""
import json
import math

import pytest
import torch

import gakupel_models as tm
import plain_gakupel as plain

F = torch.float64


def rnd(*shape, seed=0):
    return torch.randn(*shape, dtype=F, generator=torch.Generator().manual_seed(seed))


def test_config_round_trip_and_refusals():
    from hipinfer_b200.config import ConfigError, config_from_dict

    for name, cfg in tm.MODELS.items():
        c = config_from_dict(cfg)
        assert c.architecture == "Gakupel" and config_from_dict(json.loads(json.dumps(c.to_dict()))) == c, name
        assert c.to_dict()["layers"] == cfg["layers"], name
    c = config_from_dict(tm.A)
    assert c.layers[0].mixer.left.q_temp.every == 10 and c.layers[0].mlp.groups == (3, 2) and c.layers[2].mlp.groups is None
    assert c.layers[3].mlp is None and c.layers[3].mixer.left_scale == -0.5 and c.layers[0].mlp.shared_ff == 24

    def broken(change, base=tm.A):
        bad = json.loads(json.dumps(base))
        change(bad)
        with pytest.raises(ConfigError):
            config_from_dict(bad)

    broken(lambda d: d["layers"][0]["mixer"]["left"].update(kv_heads=3))
    broken(lambda d: d["layers"][1]["mixer"].update(vdim=8))                        # the values are the keys
    broken(lambda d: d["layers"][1]["mixer"]["rot"].update(dims=18))
    broken(lambda d: d["layers"][2]["mixer"].update(kv_heads=3))
    broken(lambda d: d["layers"][2]["mixer"].pop("conv"))
    broken(lambda d: d["layers"][2].update(type="convolution"))
    broken(lambda d: d["layers"][0]["mixer"].pop("right"))
    broken(lambda d: d["layers"][0]["mixer"]["right"].update(gate_cap=0.0))
    broken(lambda d: d["layers"][0]["mixer"]["left"]["q_temp"].update(every=0))
    broken(lambda d: d["layers"][0]["mlp"]["router"].update(top=7))
    broken(lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(count=4))     # six experts in four groups
    broken(lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(keep=4))
    broken(lambda d: d["layers"][0]["mlp"]["router"].update(top=5))                 # five of the four experts that stay
    broken(lambda d: d["layers"][1]["mlp"].update(kind="sparse"))
    broken(lambda d: d.pop("norm"))


def test_spec_caches_states_and_tensors():
    from hipinfer_b200.config import config_from_dict, get_architecture
    from hipinfer_b200.models.decoder import DecoderModel
    from hipinfer_b200.parts.registry import BuildContext

    build = lambda cfg: DecoderModel(get_architecture("Gakupel").build_spec(config_from_dict(cfg)), BuildContext.meta())
    m = build(tm.A)
    assert [p is not None for p in m.cache_plan] == [True, True, False, True]
    assert {k: v[0] for k, v in m.state_specs.items()} == {
        (0, "right.S"): (3, 16, 8), (0, "right.n"): (3, 16), (0, "right.m"): (3,), (2, "S"): (4, 16, 24), (2, "conv"): (3, 160),
        (3, "right.S"): (2, 24, 40), (3, "right.n"): (2, 24), (3, "right.m"): (2,)}
    names = {s.name: tuple(s.shape) for s in m.param_specs()}
    assert [names[f"l{i}.dwa"] for i in range(4)] == [(2,), (3,), (4,), (5,)]
    assert names["l0.mix.left.q.norm"] == (64,) and names["l0.mix.left.k.norm"] == (32,) and names["l0.mix.left.r1"] == (4,)
    assert names["l1.mix.q.norm"] == names["l1.mix.k.norm"] == (16,) and "l1.mix.v" not in names and "l1.mix.g" not in names
    assert names["l0.mix.right.i"] == (3, 64) and names["l0.mix.right.f.b"] == (3,) and names["l0.mix.right.norm"] == (24,)
    assert names["l2.mix.q.conv"] == (32, 4) and names["l2.mix.v.conv"] == (96, 4) and names["l2.mix.norm"] == (24,)
    assert names["l0.mlp.correction"] == (6,) and names["l0.mlp.shared.sg"] == (1, 64) and names["l2.mlp.shared.down"] == (64, 40)
    assert "l3.norm2" not in names and names["l0.norm2.b"] == names["final.norm.b"] == (64,) and names["head"] == (150, 64)
    assert all(getattr(layer, "takes_history") for layer in m.layers)
    m = build(tm.B)
    assert m.state_specs[(0, "conv")][0] == (0, 72) and m.state_specs[(3, "conv")][0] == (6, 64)
    names = {s.name for s in m.param_specs()}
    assert "l0.mlp.shared.gate" not in names and "l0.mlp.correction" in names and "l3.mlp.up" not in names


def test_parts_refuse_what_they_cannot_do():
    from hipinfer_b200.parts.registry import BuildContext, build_part
    from hipinfer_b200.parts.spec import PartSpec

    ctx = BuildContext.meta()
    base = dict(hidden_size=16, heads=2, kv_heads=1, dim=8, vdim=8, scale=1.0, eps=1e-5)
    for bad in (dict(values="keys", vdim=4), dict(values="keys", reads_cache=True), dict(head_norm=True, row_norm=True), dict(q_temp=(1.0, 0.0))):
        with pytest.raises(ValueError):
            build_part("mixer", PartSpec("masked_attention", dict(base, **bad)), ctx)
    routed = dict(hidden_size=16, experts=6, top=2, expert_size=8, score="sigmoid_normed")
    for bad in (dict(groups=(4, 2)), dict(groups=(3, 4)), dict(groups=(6, 1)), dict(groups=(3, 2), score="sigmoid")):
        with pytest.raises(ValueError):
            build_part("feed_forward", PartSpec("routed", dict(routed, **bad)), ctx)


def test_matrix_memory_is_its_unrolled_sum():
    """S_t / exp(-m_t) is the sum over s of exp(li_s + sum of lf after s) k_s v_s^T, whatever the running maximum was."""
    T, H, D, E = 12, 2, 3, 4
    q, k, v = rnd(T, H, D, seed=1), rnd(T, H, D, seed=2), rnd(T, H, E, seed=3)
    li, lf = 3 * rnd(T, H, seed=4), -plain.softplus(rnd(T, H, seed=5))
    got = plain.matrix_memory(q, k, v, li, lf)
    for t in range(T):
        for h in range(H):
            w = torch.stack([torch.exp(li[s, h] + lf[s + 1:t + 1, h].sum()) for s in range(t + 1)])
            m = max([float(lf[:t + 1, h].sum())] + [float(li[s, h] + lf[s + 1:t + 1, h].sum()) for s in range(t + 1)])
            dots = k[:t + 1, h] @ q[t, h] * w
            den = max(abs(float(dots.sum())), 1.0) + 1e-6 * math.exp(m)
            assert float((got[t, h] - (dots[:, None] * v[:t + 1, h]).sum(0) / den).abs().max()) < 1e-9


def test_delta_rule_replaces_what_a_key_holds():
    """With unit keys, beta 1 and no decay, writing a second value under the same key reads back that value alone; a decay of
    zero forgets everything."""
    k = plain.unit(rnd(1, 1, 5, seed=1)).expand(3, 1, 5)
    v, one = rnd(3, 1, 4, seed=2), torch.ones(3, 1, dtype=F)
    out = plain.gated_delta(k, k, v, one, one)
    assert float((out - v).abs().max()) < 1e-5
    g = torch.tensor([[1.0], [0.0], [1.0]], dtype=F)
    half = torch.full((3, 1), 0.5, dtype=F)
    out = plain.gated_delta(k, k, v, g, half)
    assert float((out[1] - 0.5 * v[1]).abs().max()) < 1e-5 and float((out[2] - 0.5 * v[2] - 0.25 * v[1]).abs().max()) < 1e-5


def test_temperature_bias_and_sink_by_hand():
    t = plain.temperature(9, dict(q_temp=dict(coef=0.5, every=4)))
    want = [1.0] * 3 + [1 + 0.5 * math.log(2)] * 4 + [1 + 0.5 * math.log(3)] * 2
    assert float((t - torch.tensor(want, dtype=F)).abs().max()) < 1e-12
    b = plain.distance_bias(4, torch.tensor(2.0, dtype=F), torch.tensor(0.5, dtype=F))
    assert abs(float(b[3, 1]) - 2 * math.log(2.0)) < 1e-12 and float(b.diagonal().abs().max()) == 0.0
    p = plain.causal_softmax(torch.zeros(3, 3, dtype=F), True)
    assert torch.allclose(p[2], torch.full((3,), 0.25, dtype=F)) and torch.allclose(p[0], torch.tensor([0.5, 0, 0], dtype=F))


def test_rotation_by_hand():
    t = torch.zeros(1, 6, dtype=F)
    t[0, 0], t[0, 1], t[0, 5] = 1.0, 2.0, 9.0
    r = plain.rotate_half(t, torch.tensor([3]), 4, 100.0)              # pairs (0, 2) and (1, 3); frequencies 1 and 0.1
    want = [math.cos(3), 2 * math.cos(0.3), math.sin(3), 2 * math.sin(0.3), 0.0, 9.0]
    assert float((r[0] - torch.tensor(want, dtype=F)).abs().max()) < 1e-12


def test_router_groups_by_hand():
    """Four experts in two groups: the second group's two together beat the first's, which holds the single largest."""
    logit = lambda s: math.log(s / (1 - s))
    z = torch.tensor([[logit(0.9), logit(0.1), logit(0.6), logit(0.7)]], dtype=F)
    router, zero = torch.eye(4, dtype=F), torch.zeros(4, dtype=F)
    c, w = plain.route(z, router, zero, dict(top=1, groups=dict(count=2, keep=1), scale=2.0))
    assert c.tolist() == [[3]] and abs(float(w) - 2.0) < 1e-9
    # corrections decide the choice (here all below zero), the weights are made without them
    corr = torch.tensor([-2.0, -2.0, -1.0, -3.0], dtype=F)
    c, w = plain.route(z, router, corr, dict(top=2, groups=dict(count=2, keep=2)))
    assert c.tolist() == [[2, 0]] and torch.allclose(w, torch.tensor([[0.4, 0.6]], dtype=F))


def test_plain_layers_are_averaged_over_the_depth():
    """With depth weights that keep only the embedding rows the layers change nothing; with ones on the last state the average
    is the plain residual chain."""
    cfg = tm.model(30, 16, [tm.attention(2, 1, 8, mlp=tm.dense(12)), tm.delta(1, 1, 8, 8, 2)])
    w = tm.draw_weights(cfg, 1)
    toks = [3, 7, 7, 1, 29]
    w["l0.dwa"], w["l1.dwa"] = torch.tensor([1.0, 0.0]), torch.tensor([1.0, 0.0, 0.0])
    out = plain.forward(cfg, w, toks)
    f = plain.sub(w, "final.")
    want = plain.layer_norm(w["embed"].double()[toks], f["norm"], f["norm.b"], 1e-5) @ w["head"].double().T
    assert float((out - want).abs().max()) < 1e-12
    layers = []
    w["l0.dwa"], w["l1.dwa"] = torch.tensor([0.0, 1.0]), torch.tensor([0.0, 0.5, 1.0])
    plain.forward(cfg, w, toks, layers)
    chain = []
    w["l1.dwa"] = torch.tensor([0.0, 0.0, 1.0])
    plain.forward(cfg, w, toks, chain)
    assert float((layers[1] - (0.5 * chain[0] + chain[1])).abs().max()) < 1e-12


def test_tokens_after_a_position_change_nothing_before_it():
    for name, cfg in tm.MODELS.items():
        w = tm.draw_weights(cfg, 2)
        toks = [int(t) for t in torch.randint(0, cfg["vocab"], (24,), generator=torch.Generator().manual_seed(1))]
        a, b = plain.forward(cfg, w, toks), plain.forward(cfg, w, toks[:15])
        assert float((a[:15] - b).abs().max()) < 1e-9, name


def test_random_weights_mode_writes_a_loadable_folder(tmp_path):
    from hipinfer_b200.config import config_from_dict, get_architecture, load_config
    from hipinfer_b200.parts.spec import spec_param_specs
    from hipinfer_b200.weights import load_weights, write_random_model

    write_random_model(config_from_dict(tm.A), str(tmp_path), 3)
    c = load_config(str(tmp_path))
    t = load_weights(str(tmp_path), spec_param_specs(get_architecture("Gakupel").build_spec(c)), device="cpu")
    assert torch.allclose(t["l1.dwa"].float(), torch.full((3,), 1 / 3), atol=2e-3) and t["l0.mlp.e5.down"].shape == (64, 32)
