"""Seredra on the CPU: configuration, names, cache plan and schedule of the engine's description, and properties of the
plain implementation that the GPU tests measure against."""

import copy
import math

import pytest
import torch

import plain_seredra as plain
from matricxon_b200.config import ConfigError, config_from_dict, resolve_architecture
from matricxon_b200.config.seredra import SeredraConfig
from matricxon_b200.models.decoder import model_weight_specs, plan_cache
from matricxon_b200.parts.base import Runtime, StateRequest, part_class
from matricxon_b200.parts.rotary import interpolated_frequencies
from matricxon_b200.parts.spec import InterpolatedRotarySpec, ParallelMixerSpec, RoutedExpertsSpec
from seredra_configs import MODELS, conv_attention, dense, draw, ids, model, moe, parallel, retention, single_layer, turned

F64 = torch.float64


def doubles(tensors):
    return {name: value.double() for name, value in tensors.items()}


@pytest.mark.parametrize("name", list(MODELS))
def test_registry_and_round_trip(name):
    raw = MODELS[name]
    assert resolve_architecture(raw).config_class is SeredraConfig
    config = config_from_dict(copy.deepcopy(raw))
    assert config.to_dict() == raw
    assert config_from_dict(config.to_dict()) == config


def test_tensor_names_and_shapes():
    spec = config_from_dict(copy.deepcopy(MODELS["A"])).model_spec()
    shapes = {w.name: tuple(w.shape) for w in model_weight_specs(spec)}
    assert shapes["embed"] == (211, 96) and shapes["head"] == (211, 96) and shapes["final.norm"] == ()
    assert shapes["l0.norm1"] == () and "l0.norm2" not in shapes and "l0.mlp.up" not in shapes
    assert shapes["l0.mix.q"] == (144, 96) and shapes["l0.mix.k"] == (72, 96) and shapes["l0.mix.v"] == (120, 96)
    for name, rows in (("q", 144), ("k", 72), ("v", 120)):
        assert shapes[f"l0.mix.{name}.b"] == (rows,) and shapes[f"l0.mix.{name}.conv"] == (rows, 4)
    assert shapes["l0.mix.q.norm"] == (144,) and shapes["l0.mix.k.norm"] == (72,) and "l0.mix.v.norm" not in shapes
    assert shapes["l0.mix.r1"] == (6,) and shapes["l0.mix.r2"] == (6,)
    assert shapes["l0.mix.o"] == (96, 240) and shapes["l0.mix.o.b"] == (96,)
    assert shapes["l1.mix.q"] == (60, 96) and shapes["l1.mix.k"] == (60, 96) and shapes["l1.mix.v"] == (84, 96)
    assert shapes["l1.mix.g"] == (84, 96) and shapes["l1.mix.o"] == (96, 84) and shapes["l1.norm2"] == ()
    assert shapes["l1.mlp.router"] == (5, 96) and shapes["l1.mlp.e4.gate"] == (40, 96) and shapes["l1.mlp.e4.down"] == (96, 40)
    assert shapes["l2.mix.left.q"] == (160, 96) and shapes["l2.mix.left.k"] == (40, 96) and "l2.mix.left.v" not in shapes
    assert shapes["l2.mix.left.q.norm"] == (40,) and shapes["l2.mix.left.k.norm"] == (40,)
    assert shapes["l2.mix.left.o"] == (96, 160)
    assert shapes["l2.mix.right.in"] == (144, 96) and shapes["l2.mix.right.conv"] == (72, 3)
    assert shapes["l2.mix.right.conv.b"] == (72,) and shapes["l2.mix.right.x"] == (35, 72)
    assert shapes["l2.mix.right.dt"] == (72, 9) and shapes["l2.mix.right.dt.b"] == (72,)
    assert shapes["l2.mix.right.A_log"] == (72, 13) and shapes["l2.mix.right.D"] == (72,)
    assert shapes["l2.mix.right.o"] == (96, 72)
    assert shapes["l2.mlp.up"] == (72, 96) and shapes["l2.mlp.down"] == (96, 72) and "l2.mlp.gate" not in shapes
    # a layer on another one's keys and values has none of their tensors
    assert shapes["l3.mix.q.conv"] == (72, 2) and shapes["l3.mix.q.norm"] == (72,) and shapes["l3.mix.r1"] == (3,)
    assert not any(name.startswith(("l3.mix.k", "l3.mix.v")) for name in shapes)
    assert not any(name.endswith(".weight") for name in shapes)


def test_schedule_cache_and_state_plan():
    spec = config_from_dict(copy.deepcopy(MODELS["A"])).model_spec()
    assert [(e.layer, e.cache_of) for e in spec.schedule] == [(0, None), (1, None), (2, None), (3, 0)]
    plan = plan_cache(spec)
    by_request = {(g.request.num_kv_heads, g.request.head_dim, g.request.window, g.request.planes): g.entries
                  for g in plan.groups}
    assert by_request == {(3, 48, None, 2): (0,), (1, 48, None, 2): (2,)}
    assert plan.kv_of_entry[3] == plan.kv_of_entry[0] and plan.writes == (True, True, True, False)
    assert plan.state_of_entry == (StateRequest((3, 144 + 72 + 120)), StateRequest((3, 20, 28)),
                                   StateRequest((72 * (2 + 13),)), StateRequest((1, 72)))
    # one tap keeps nothing; a model of recurrent layers has no paged cache
    c = plan_cache(config_from_dict(copy.deepcopy(MODELS["C"])).model_spec())
    assert c.state_of_entry[2] is None and c.state_of_entry[1] == StateRequest((60,))
    d = plan_cache(config_from_dict(copy.deepcopy(MODELS["D"])).model_spec())
    assert d.groups == () and all(state is not None for state in d.state_of_entry)
    b = plan_cache(config_from_dict(copy.deepcopy(MODELS["B"])).model_spec())
    assert [b.kv_of_entry[i] for i in (2, 4)] == [b.kv_of_entry[1]] * 2


def test_what_the_description_says_of_the_mechanisms():
    spec = config_from_dict(copy.deepcopy(MODELS["A"])).model_spec()
    first, second, third, fourth = (layer.mixer for layer in spec.layers)
    assert first.temperature == (0.4, 19) and first.taps == 4 and first.distance_names == ("r1", "r2") and not first.shares_kv
    assert fourth.shares_kv and fourth.taps == 2
    assert second.key_scale == 20 ** -0.5 and second.decay == (0.9, 0.99, 0.5) and second.position.rotary_dim == 12
    (left, left_scale, left_name), (right, right_scale, right_name) = third.branches
    assert (left_scale, left_name, right_scale, right_name) == (0.7, "left.", 1.4, "right.")
    assert left.value_name is None and left.softcap == 4.0 and left.position.factor == 4.0 and left.mask == "causal"
    assert (right.channels, right.states, right.dt_rank, right.taps) == (72, 13, 9, 3)
    assert spec.layers[2].feed_forward.activation == "relu_squared" and not spec.layers[2].feed_forward.bias
    routed = spec.layers[1].feed_forward
    assert not routed.normalize and routed.weight_on == "input" and routed.score == "sigmoid" and routed.num_groups == 1
    assert spec.layers[0].feed_forward is None and not spec.tie_word_embeddings and spec.embedding_scale == 3.0
    assert spec.final_norm.scalar and spec.final_norm.eps == 1e-5


def test_a_second_norm_that_lies_unused():
    config = config_from_dict(copy.deepcopy(MODELS["A"])).with_tensor_shapes({"l0.norm2": (), "l1.norm2": ()}.get)
    assert config.unused_tensors == (("l0.norm2", ()),)
    assert "l0.norm2" in {w.name for w in model_weight_specs(config.model_spec())}


@pytest.mark.parametrize("change, key", [
    (lambda r: r["layers"][0].update(type="mamba"), "mamba"),
    (lambda r: r["layers"][0]["mixer"].pop("heads"), "heads"),
    (lambda r: r["layers"][0]["mixer"].update(kv_heads=4), "kv_heads"),
    (lambda r: r["layers"][0]["mixer"].update(dim=300), "dim"),
    (lambda r: r["layers"][0]["mixer"]["q_temp"].pop("every"), "every"),
    (lambda r: r["layers"][0]["mixer"]["q_temp"].update(every=0), "every"),
    (lambda r: r["layers"][0]["mixer"].update(conv=0), "conv"),
    (lambda r: r["layers"][0]["mixer"].update(kv_from=0), "kv_from"),
    (lambda r: r["layers"][3]["mixer"].update(kv_from=1), "kv_from"),
    (lambda r: r["layers"][3]["mixer"].update(kv_from=3), "kv_from"),
    (lambda r: r["layers"][3]["mixer"].update(vdim=16), "kv_from"),
    (lambda r: r["layers"][1]["mixer"].update(decay=[0.5]), "decay"),
    (lambda r: r["layers"][1]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda r: r["layers"][1]["mixer"]["rot"].update(scaling={}), "scaling"),
    (lambda r: r["layers"][1]["mixer"].update(dim=320), "dim"),
    (lambda r: r["layers"][2]["mixer"].pop("left"), "left"),
    (lambda r: r["layers"][2]["mixer"]["left"].update(vdim=24), "vdim"),
    (lambda r: r["layers"][2]["mixer"]["left"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda r: r["layers"][2]["mixer"]["right"].pop("dt_rank"), "dt_rank"),
    (lambda r: r["layers"][2]["mixer"]["right"].update(state=200), "state"),
    (lambda r: r["layers"][1]["mlp"]["router"].update(top=6), "top"),
    (lambda r: r["layers"][2]["mlp"].update(kind="sparse"), "sparse"),
    (lambda r: r.pop("norm"), "norm"),
    (lambda r: r.pop("vocab"), "vocab"),
    (lambda r: r.update(layers=[]), "layers"),
])
def test_errors_name_the_key(change, key):
    raw = copy.deepcopy(MODELS["A"])
    change(raw)
    with pytest.raises(ConfigError, match=key):
        config_from_dict(raw)


def test_absent_keys_mean_absent_mechanisms():
    raw = model(64, 50, 1.0, [conv_attention(2, 1, 16, 16, 0.3, 3, (0.1, 4)),
                              parallel((2, 1, 16, 0.3, 5.0, None), (32, 4, 4, 2), 1.0, 1.0),
                              retention(2, 16, 16, [0.5, 0.9], None)])
    for key in ("q_temp", "conv", "vdim"):
        del raw["layers"][0]["mixer"][key]
    del raw["layers"][1]["mixer"]["left"]["softcap"], raw["embedding"]
    spec = config_from_dict(raw).model_spec()
    first = spec.layers[0].mixer
    assert first.temperature is None and first.taps is None and first.value_dim == 16
    assert "l0.mix.q.conv" not in {w.name for w in model_weight_specs(spec)}
    left = spec.layers[1].mixer.branches[0][0]
    assert left.softcap is None and left.position is None and spec.layers[2].mixer.position is None
    assert spec.embedding_scale == 1.0


def test_parts_refuse_what_they_cannot_do():
    spec = config_from_dict(copy.deepcopy(MODELS["A"])).model_spec()
    runtime = Runtime(device="cpu", dtype=torch.float32)
    left = spec.layers[2].mixer.branches[0][0]
    with pytest.raises(ValueError, match="paged cache"):               # two branches with keys and values
        part_class("mixer", "parallel").cache_request(ParallelMixerSpec(64, ((left, 1.0, "a."), (left, 1.0, "b."))))
    with pytest.raises(ValueError, match="BranchMixer"):
        part_class("mixer", "parallel")(ParallelMixerSpec(64, ((spec.layers[0].mixer, 1.0, "a."),)), runtime, "")
    routed = spec.layers[1].feed_forward
    with pytest.raises(ValueError, match="output"):
        RoutedExpertsSpec(**{**vars(routed), "weight_on": "both"})
    with pytest.raises(ValueError, match="matrices"):
        RoutedExpertsSpec(**{**vars(routed), "score": "softmax", "normalize": True, "num_identity": 1})


def test_frequency_table_is_the_plain_one():
    for dims, base, scaling in ((24, 5000.0, (4.0, 64.0, 8.0, 1.0)), (96, 300.0, (16.0, 32.0, 4.0, 1.0)),
                                (48, 500000.0, (8.0, 512.0, 16.0, 1.0)), (6, 90.0, None), (2, 10.0, (2.0, 10.0, 3.0, 3.0))):
        keys = ("factor", "original", "fast", "slow")
        named = dict(zip(keys, scaling)) if scaling else {}
        table, amplitude = interpolated_frequencies(InterpolatedRotarySpec(rotary_dim=dims, theta=base, **named))
        want, want_amplitude = plain.frequencies(dims, base, named or None)
        assert torch.allclose(table, want, rtol=1e-14) and amplitude == want_amplitude


# ---------------------------------------------------------------------- the plain model's own properties
def test_rotation_turns_by_the_distance_and_leaves_the_rest():
    gen = torch.Generator().manual_seed(1)
    q, k = torch.randn(1, 1, 12, generator=gen, dtype=F64), torch.randn(1, 1, 12, generator=gen, dtype=F64)
    for scaling in (None, (4.0, 64, 8.0, 1.0)):
        rot = turned(8, 100.0, scaling)
        score = lambda p, j: float((plain.rotate(q, torch.tensor([p]), rot) * plain.rotate(k, torch.tensor([j]), rot)).sum())
        assert abs(score(40, 33) - score(1007, 1000)) < 1e-9 and abs(score(40, 33) - score(40, 32)) > 1e-4
        moved = plain.rotate(q, torch.tensor([5]), rot)
        assert torch.equal(moved[..., 8:], q[..., 8:])
        longer = 1.0 if scaling is None else 0.1 * math.log(scaling[0]) + 1.0
        assert abs(float(moved[..., :8].norm() / q[..., :8].norm()) - longer) < 1e-12


def test_temperature_steps_at_whole_periods():
    t = plain.temperature(torch.arange(30), 0.5, 10)
    assert torch.equal(t[:9], torch.ones(9, dtype=F64))
    assert abs(float(t[9]) - (1 + 0.5 * math.log(2))) < 1e-12 and float(t[9]) == float(t[18]) < float(t[19])


def test_distance_bias_is_zero_at_home_and_grows_slowly():
    b = plain.distance_bias(50, torch.tensor([2.0, 0.5], dtype=F64), torch.tensor([0.3, 1.0], dtype=F64))
    assert float(b[:, torch.arange(50), torch.arange(50)].abs().max()) == 0.0
    assert abs(float(b[0, 20, 10]) - 2.0 * math.log(4.0)) < 1e-12 and abs(float(b[1, 49, 0]) - 0.5 * math.log(50.0)) < 1e-12


def test_convolution_looks_back_and_starts_from_zeros():
    u, w = torch.randn(9, 3, dtype=F64), torch.randn(3, 4, dtype=F64)
    y = plain.causal_conv(u, w)
    assert torch.allclose(y[0], w[:, 3] * u[0])
    assert torch.allclose(y[5], sum(w[:, j] * u[2 + j] for j in range(4)))


def test_both_recurrences_against_their_sums():
    gen = torch.Generator().manual_seed(2)
    T, H, D, V = 12, 2, 4, 3
    q, k, v = (torch.randn(T, H, n, generator=gen, dtype=F64) for n in (D, D, V))
    decay = torch.tensor([0.9, 0.3], dtype=F64)
    o = plain.linear_recurrence(q, k, v, decay)
    for t in (0, 7, 11):
        want = sum(decay[:, None] ** (t - j) * (q[t] * k[j]).sum(-1, keepdim=True) * v[j] for j in range(t + 1))
        assert torch.allclose(o[t], want)
    C, N = 5, 3
    x, dt, b, c = (torch.rand(T, n, generator=gen, dtype=F64) for n in (C, C, N, N))
    a, d = -torch.rand(C, N, generator=gen, dtype=F64), torch.randn(C, generator=gen, dtype=F64)
    y = plain.selective_scan(x, dt, b, c, a, d)
    want = d * x[7]
    for j in range(8):
        passed = dt[j + 1:8].sum(0)
        want = want + (torch.exp(passed[:, None] * a) * (dt[j] * x[j])[:, None] * b[j]) @ c[7]
    assert torch.allclose(y[7], want)


def test_the_weight_goes_on_the_experts_input():
    raw = single_layer(dict(retention(1, 8, 8, [0.5], None), mlp=moe(12, 4, 2)))
    w = doubles(draw(raw, seed=1))
    h = torch.randn(3, 64, dtype=F64)
    out = plain.feed_forward(h, w, "l0.mlp.", raw["layers"][0]["mlp"])
    chosen, score, _ = plain.route(h, w["l0.mlp.router"], 2)
    after = torch.zeros_like(out)
    for t in range(3):
        for slot in range(2):
            q = f"l0.mlp.e{int(chosen[t, slot])}."
            after[t] += score[t, slot] * plain.gated(h[t:t + 1], w[q + "gate"], w[q + "up"], w[q + "down"])[0]
    assert not torch.allclose(out, after, rtol=1e-2)
    full = torch.ones(4, 64, dtype=F64) * 1e3                           # scores of one: the two agree
    w["l0.mlp.router"] = full
    h = h.abs()
    out = plain.feed_forward(h, w, "l0.mlp.", raw["layers"][0]["mlp"], forced=chosen)
    want = sum(torch.stack([plain.gated(h[t:t + 1], w[f"l0.mlp.e{int(chosen[t, s])}.gate"], w[f"l0.mlp.e{int(chosen[t, s])}.up"],
                                        w[f"l0.mlp.e{int(chosen[t, s])}.down"])[0] for t in range(3)]) for s in range(2))
    assert torch.allclose(out, want)


def test_every_tensor_is_used_and_a_prefix_does_not_depend_on_what_follows():
    for name in ("A", "B", "C", "D"):
        raw = MODELS[name]
        weights = doubles(draw(raw, seed=5))
        tokens = ids(40, raw["vocab"], seed=2)
        full = plain.forward(raw, weights, tokens)
        assert torch.allclose(plain.forward(raw, weights, tokens[:30]), full[:30], atol=1e-9)
        moved_experts = 0
        for tensor in weights:
            changed = dict(weights)
            changed[tensor] = weights[tensor] * 1.5 + 0.01
            same = torch.allclose(plain.forward(raw, changed, tokens), full, atol=1e-9)
            if ".mlp.e" in tensor:
                moved_experts += not same                              # an expert that nobody drew changes nothing
            else:
                assert not same, tensor
        assert moved_experts > 0


def test_a_sharing_layer_reads_its_sources_keys_and_values():
    raw = MODELS["A"]
    weights = doubles(draw(raw, seed=5))
    tokens = ids(25, raw["vocab"], seed=3)
    taps = plain.forward(raw, weights, tokens, return_layers=True)[1]
    own = copy.deepcopy(raw)
    del own["layers"][3]["mixer"]["kv_from"]
    with pytest.raises(KeyError):                                       # it has no tensors for keys of its own
        plain.forward(own, weights, tokens)
    changed = dict(weights)
    changed["l0.mix.o"] = weights["l0.mix.o"] * 0.0                     # what layer 0 adds does not touch what it stores
    other = plain.forward(raw, changed, tokens, return_layers=True)[1]
    assert not torch.allclose(other[0], taps[0])
    k, v = plain.keys_values(plain.unit(weights["embed"][tokens] * 3.0, 1e-5) * weights["l0.norm1"], weights, "l0.mix.",
                             raw["layers"][0]["mixer"], 1e-5)
    assert k.shape == (25, 3, 24) and v.shape == (25, 3, 40)
    assert abs(float((k.reshape(25, -1) / weights["l0.mix.k.norm"]).pow(2).mean()) - 1.0) < 1e-3


def test_one_number_scales_every_coordinate_of_a_norm():
    raw = single_layer(dict(retention(1, 8, 8, [0.5], None), mlp=dense(16)))
    weights = doubles(draw(raw, seed=2))
    tokens = ids(9, raw["vocab"], seed=1)
    changed = dict(weights)
    changed["final.norm"] = weights["final.norm"] * 2.0
    assert torch.allclose(plain.forward(raw, changed, tokens), 2.0 * plain.forward(raw, weights, tokens))
