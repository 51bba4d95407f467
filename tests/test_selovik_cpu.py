"""The Selovik design without a GPU: its configuration, its description as parts, the cache and state plan the decoder
derives from it, and the plain implementation against hand-made cases (the bigram rows, the rotation's scaling, the window, the
combination of two maps, the router's groups and identity experts, the loop)."""
import json
import math

import pytest
import torch

import selovik_models as tm
import plain_selovik as plain

F = torch.float64


def rnd(*shape, seed=0):
    return torch.randn(*shape, dtype=F, generator=torch.Generator().manual_seed(seed))


def test_config_round_trip_and_refusals():
    from hipinfer_b200.config import ConfigError, config_from_dict

    for name, cfg in tm.MODELS.items():
        c = config_from_dict(cfg)
        assert c.architecture == "Selovik" and config_from_dict(json.loads(json.dumps(c.to_dict()))) == c, name
        assert c.to_dict()["layers"] == cfg["layers"] and c.to_dict().get("loop") == cfg.get("loop"), name
        assert c.to_dict()["embedding"] == cfg["embedding"] and c.logit_scale == cfg["logit_scale"]
        assert c.run_order() == plain.run_order(cfg), name
    c = config_from_dict(tm.A)
    assert c.loop.times == 3 and c.bigram == (101, 7, 3) and c.layers[0].mixer.rot.scaling_dict()["original"] == 64.0
    assert c.layers[1].mlp.groups == (3, 2) and c.layers[2].mlp.groups is None and c.layers[2].mlp.identity == 1
    assert c.layers[3].mlp is None and c.layers[3].mixer.window == 1 and c.layers[2].mixer.window is None and c.layers[3].mixer.rot.dims == 0
    assert config_from_dict(tm.D).bigram is None and config_from_dict(tm.D).loop is None

    def broken(change, base=tm.A):
        bad = json.loads(json.dumps(base))
        change(bad)
        with pytest.raises(ConfigError):
            config_from_dict(bad)

    broken(lambda d: d["layers"][1]["mixer"].update(kv_heads=4))
    broken(lambda d: d["layers"][0]["mixer"]["rot"].update(dims=18))
    broken(lambda d: d["layers"][0]["mixer"]["rot"].update(dims=7))
    broken(lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].pop("fast"))
    broken(lambda d: d["layers"][0]["mixer"].pop("diff"))
    broken(lambda d: d["layers"][0]["mixer"]["mask"].update(size=0))
    broken(lambda d: d["layers"][0].update(type="convolution"))
    broken(lambda d: d["layers"][1]["mlp"]["router"].update(top=7))                # seven of the six choices that stay
    broken(lambda d: d["layers"][1]["mlp"]["router"]["groups"].update(count=4))    # nine choices in four groups
    broken(lambda d: d["layers"][1]["mlp"]["router"]["groups"].update(keep=4))
    broken(lambda d: d["layers"][1]["mlp"]["router"].update(identity=-1))
    broken(lambda d: d["layers"][0]["mlp"].update(kind="sparse"))
    broken(lambda d: d["loop"].update(stop=6))
    broken(lambda d: d["loop"].update(start=3))
    broken(lambda d: d["loop"].update(times=0))
    broken(lambda d: d["embedding"]["bigram"].update(buckets=0))
    broken(lambda d: d["embedding"]["bigram"].update(mul_cur=-1))
    broken(lambda d: d.pop("norm"))


def test_spec_caches_states_and_tensors():
    from hipinfer_b200.config import config_from_dict, get_architecture
    from hipinfer_b200.models.decoder import EMBEDDING_STATE, DecoderModel
    from hipinfer_b200.parts.registry import BuildContext

    build = lambda cfg: DecoderModel(get_architecture("Selovik").build_spec(config_from_dict(cfg)), BuildContext.meta())
    m = build(tm.A)
    assert [s.layer for s in m.spec.order] == [0, 1, 2, 1, 2, 1, 2, 3, 4]
    assert [s.enters_pass for s in m.spec.order] == [None, 0, None, 1, None, 2, None, None, None]
    # every pass writes a cache of its own: the looped layers' groups hold one per pass
    assert len({(p.group, p.slot) for p in m.cache_plan}) == 9 and all(p.write for p in m.cache_plan)
    assert sorted(g.n_layers for g in m.cache_groups) == [1, 1, 1, 3, 3]
    assert m.state_specs == {(EMBEDDING_STATE, "previous"): ((), torch.int32)}
    names = {s.name: tuple(s.shape) for s in m.param_specs()}
    assert names["bigram"] == (102, 64) and names["loop.step"] == (3, 64) and names["embed.norm"] == names["final.norm"] == (64,)
    assert names["l1.mix.q"] == (96, 64) and names["l1.mix.k"] == (32, 64) and names["l1.mix.v"] == (64, 64) and names["l1.mix.lk2"] == (8,)
    assert names["l1.mlp.router"] == (9, 64) and names["l1.mlp.correction"] == (9,) and "l1.mlp.e6.up" not in names and "l1.mlp.e5.up" in names
    assert names["l1.mlp.shared.down"] == (64, 24) and "l1.mlp.shared.sg" not in names and "l2.mlp.shared.up" not in names
    assert "l3.norm2" not in names and names["l0.norm2"] == (64,) and "head" not in names and "l0.mix.q.b" not in names
    m = build(tm.D)
    assert not m.state_specs and m.pass_entry is None and "bigram" not in {s.name for s in m.param_specs()}


def test_parts_refuse_what_they_cannot_do():
    from hipinfer_b200.parts.registry import BuildContext, build_part
    from hipinfer_b200.parts.spec import LayerSpec, ModelSpec, PartSpec, RunStep

    ctx = BuildContext.meta()
    attn = dict(hidden_size=16, heads=2, kv_heads=1, dim=8, vdim=8, scale=1.0, diff=0.5, eps=1e-5)
    for bad in (dict(rot_dims=4), dict(rot_dims=10, biases=False), dict(rot_dims=3, biases=False)):
        with pytest.raises(ValueError):
            build_part("mixer", PartSpec("differential_attention", dict(attn, **bad)), ctx)
    routed = dict(hidden_size=16, experts=4, identity=2, top=2, expert_size=8, score="softmax", weight_at="output")
    build_part("feed_forward", PartSpec("routed", dict(routed, groups=(3, 1))), ctx)
    for bad in (dict(groups=(4, 2)), dict(groups=(6, 1)), dict(top=7), dict(score="sigmoid_normed"), dict(weight_at="input")):
        with pytest.raises(ValueError):
            build_part("feed_forward", PartSpec("routed", dict(routed, **bad)), ctx)
    with pytest.raises(ValueError):
        build_part("embedding", PartSpec("token_bigram", dict(name="e", vocab_size=4, hidden_size=8, bigram=(0, 1, 1))), ctx)
    with pytest.raises(ValueError):
        build_part("feed_forward", PartSpec("activated", dict(hidden_size=8, intermediate_size=8, activation="relu3")), ctx)
    layer = LayerSpec("l0.", "parallel", dict(norm=PartSpec("rmsnorm", dict(name="n", size=8, eps=1e-5)),
                                              mixer=PartSpec("differential_attention", dict(attn, hidden_size=8))))
    spec = ModelSpec("X", 8, 8, 8, PartSpec("token", dict(name="e", vocab_size=8, hidden_size=8)), (layer,), (RunStep(0, enters_pass=0),),
                     PartSpec("rmsnorm", dict(name="f", size=8, eps=1e-5)), PartSpec("linear", dict(tied_to="e", vocab_size=8, hidden_size=8)))
    with pytest.raises(ValueError, match="pass_entry"):
        spec.validate()


def test_bigram_rows_by_hand():
    b = dict(buckets=10, mul_prev=7, mul_cur=3)
    assert plain.bigram_rows([4, 4, 9, 0], b) == [10, (28 + 12) % 10, (28 + 27) % 10, 63 % 10]
    assert plain.bigram_rows([2], b) == [10]
    big = dict(buckets=13, mul_prev=4000000007, mul_cur=2500000001)
    assert plain.bigram_rows([96, 95], big)[1] == (96 * (4000000007 % 13) + 95 * (2500000001 % 13)) % 13


def test_embedding_by_hand():
    cfg = dict(embedding=dict(scale=3.0, bigram=dict(buckets=2, mul_prev=1, mul_cur=1)), norm=dict(eps=0.0))
    w = {"embed": torch.tensor([[1.0, 0.0], [0.0, 2.0]]), "bigram": torch.tensor([[0.0, 1.0], [5.0, 0.0], [1.0, -4.0]]),
         "embed.norm": torch.tensor([0.0, 1.0])}
    got = plain.embedding([1, 0, 0], w, cfg)
    raw = torch.tensor([[1.0, 2.0], [8.0, 0.0], [3.0, 1.0]], dtype=F)      # rows 2 (first), (1 + 0) mod 2, (0 + 0) mod 2
    want = raw / torch.sqrt((raw ** 2).mean(-1, keepdim=True)) * torch.tensor([1.0, 2.0], dtype=F)
    assert float((got - want).abs().max()) < 1e-12


def test_rotation_and_its_scaling_by_hand():
    t = torch.zeros(1, 6, dtype=F)
    t[0, 0], t[0, 1], t[0, 5] = 1.0, 2.0, 9.0
    r = plain.rotate(t, torch.tensor([3]), dict(dims=4, base=100.0))       # pairs (0, 2) and (1, 3); frequencies 1 and 0.1
    want = [math.cos(3), 2 * math.cos(0.3), math.sin(3), 2 * math.sin(0.3), 0.0, 9.0]
    assert float((r[0] - torch.tensor(want, dtype=F)).abs().max()) < 1e-12
    # base 2, eight dims: a wavelength of original / t positions is reached at dimension 4 log2(original / (2 pi t)); fast and slow
    # chosen so that this is 0.5 and 2.5: frequencies from 1 on keep, from 3 on fall by the factor
    orig = 64.0
    at = lambda d: orig / (2 * math.pi * 2 ** (d / 4))
    f, mag = plain.frequencies(dict(dims=8, base=2.0, scaling=dict(factor=4.0, original=orig, fast=at(0.5), slow=at(2.5))))
    plain_f = [2.0 ** (-i / 4) for i in range(4)]
    ramp = [0.0, 1 / 3, 2 / 3, 1.0]                                         # lo = 0, hi = 3
    assert all(abs(a - (b / 4 * r + b * (1 - r))) < 1e-12 for a, b, r in zip(f, plain_f, ramp))
    assert abs(mag - (0.1 * math.log(4) + 1)) < 1e-12
    # both bounds below the first dimension, and equal ones: no division by zero
    f, _ = plain.frequencies(dict(dims=8, base=10.0, scaling=dict(factor=2.0, original=1.0, fast=32.0, slow=1.0)))
    assert all(math.isfinite(x) for x in f)


def test_the_product_computes_the_same_frequencies():
    from hipinfer_b200.kernels import ops

    for rot in (dict(dims=32, base=10000.0, scaling=tm.yarn(4.0, 512)), dict(dims=8, base=500000.0, scaling=tm.yarn(16.0, 77, 8.0, 0.5)),
                dict(dims=64, base=100.0, scaling=tm.yarn(2.0, 4.0)), dict(dims=6, base=3.0, scaling=tm.yarn(1.0, 4096)), dict(dims=10, base=77.0)):
        sc = dict(rot["scaling"], kind="yarn") if rot.get("scaling") else None
        got, mag = ops.rope_frequencies(rot["dims"], rot["base"], sc)
        want, want_mag = plain.frequencies(rot)
        assert mag == pytest.approx(want_mag) and torch.allclose(got, torch.tensor(want, dtype=F), rtol=1e-12), rot


def test_window_and_combination_by_hand():
    p = plain.window_softmax(torch.zeros(5, 5, dtype=F), 2)
    assert torch.allclose(p[0], torch.tensor([1.0, 0, 0, 0, 0], dtype=F)) and torch.allclose(p[4], torch.tensor([0, 0, 0, 0.5, 0.5], dtype=F))
    assert torch.allclose(plain.window_softmax(torch.zeros(3, 3, dtype=F), None)[2], torch.full((3,), 1 / 3, dtype=F))
    assert torch.equal(plain.window_softmax(rnd(4, 4), 1), torch.eye(4, dtype=F))
    w = dict(lq1=torch.tensor([1.0, 2.0]), lk1=torch.tensor([0.5, 0.0]), lq2=torch.tensor([0.0, 1.0]), lk2=torch.tensor([3.0, -1.0]))
    assert plain.combination(w, 0.3) == pytest.approx(math.exp(0.5) - math.exp(-1.0) + 0.3)


def test_two_equal_maps_leave_a_multiple_of_one():
    """With both maps alike the head's result is (1 - lambda) a, whose norm forgets the factor but not its sign."""
    m = dict(heads=1, kv_heads=1, dim=4, vdim=4, scale=0.5, diff=0.25, mask=dict(size=3))
    half = rnd(4, 6, seed=1)
    w = dict(q=torch.cat([half, half]), k=torch.cat([half, half]), v=rnd(4, 6, seed=2), g=torch.zeros(4, 6, dtype=F), o=torch.eye(4, dtype=F))
    h = rnd(7, 6, seed=3)
    for sign, lq in ((1.0, -3.0), (-1.0, 2.0)):
        w.update(lq1=torch.tensor([lq] + [0.0] * 3), lk1=torch.ones(4), lq2=torch.full((4,), -9.0), lk2=torch.ones(4))
        one = plain.window_softmax((h @ half.T) @ (h @ half.T).T * 0.5, 3) @ (h @ w["v"].T)
        want = sign * one / torch.sqrt((one ** 2).mean(-1, keepdim=True)) * 0.75 * 0.5        # the gate is sigmoid(0)
        assert float((plain.attention(h, w, m, 1e-12) - want).abs().max()) < 1e-6


def test_router_by_hand():
    """Six choices in three groups: a group is as good as its best; the corrections decide the choice, not the weights."""
    s = torch.tensor([[0.30, 0.02, 0.16, 0.17, 0.25, 0.10]], dtype=F)
    z, router = torch.log(s), torch.eye(6, dtype=F)
    zero = torch.zeros(6, dtype=F)
    c, w = plain.route(z, router, zero, dict(top=2, groups=dict(count=3, keep=1)))
    assert c.tolist() == [[0, 1]] and torch.allclose(w, s[:, [0, 1]])          # by the sum of two, group 2 would be the best
    c, w = plain.route(z, router, zero, dict(top=3, groups=dict(count=3, keep=2)))
    assert c.tolist() == [[0, 4, 5]]
    corr = torch.tensor([-0.9, -0.5, -0.7, -0.8, -0.6, -0.45], dtype=F)        # every choice score below zero
    c, w = plain.route(z, router, corr, dict(top=2))
    assert c.tolist() == [[4, 5]] and torch.allclose(w, s[:, [4, 5]])
    assert float(plain.closest_call(z, router, zero, dict(top=1))) == pytest.approx(0.05)
    assert float(plain.closest_call(z, router, zero, dict(top=1, groups=dict(count=3, keep=2)))) == pytest.approx(0.05)


def test_identity_experts_return_their_input():
    h = rnd(5, 4, seed=1)
    w = {"router": torch.zeros(3, 4, dtype=F), "correction": torch.tensor([0.0, 0.1, 0.2], dtype=F)}
    w.update({f"e0.{k}": rnd(*s, seed=i) for i, (k, s) in enumerate((("gate", (6, 4)), ("up", (6, 4)), ("down", (4, 6))))})
    got = plain.experts(h, w, dict(experts=1, identity=2, top=2))
    assert torch.allclose(got, 2.0 / 3.0 * h)
    got = plain.experts(h, w, dict(experts=1, identity=2, top=3))
    assert torch.allclose(got, 2.0 / 3.0 * h + plain.expert(h, plain.sub(w, "e0.")) / 3.0)


def test_the_loop_adds_the_embedding_from_the_second_pass_on():
    """With layers that add nothing (zero output projections) the stream at the end is the embedding times the passes plus every
    pass's vector."""
    cfg = tm.model(30, 16, [tm.layer(2, 1, 8, 8), tm.layer(1, 1, 8, 8), tm.layer(2, 2, 8, 8)], loop=(1, 2, 3))
    w = tm.draw_weights(cfg, 1)
    for i in range(3):
        w[f"l{i}.mix.o"] = torch.zeros_like(w[f"l{i}.mix.o"])
    toks, layers = [3, 7, 7, 1, 29], []
    plain.forward(cfg, w, toks, layers)
    x0, step = plain.embedding(toks, w, cfg), w["loop.step"].double()
    assert len(layers) == 5
    for i, want in enumerate((x0, x0 + step[0], 2 * x0 + step[0] + step[1], 3 * x0 + step.sum(0), 3 * x0 + step.sum(0))):
        assert float((layers[i] - want).abs().max()) < 1e-12, i


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
    t = load_weights(str(tmp_path), spec_param_specs(get_architecture("Selovik").build_spec(c)), device="cpu")
    assert t["loop.step"].shape == (3, 64) and t["l1.mlp.e5.down"].shape == (64, 32) and t["bigram"].shape == (102, 64)
