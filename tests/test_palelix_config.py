"""Palelix on the CPU: configuration, names, schedule, cache and state plan of the engine's description, and properties of the
plain implementation that the GPU tests measure against."""

import copy

import pytest
import torch

import plain_palelix as plain
from matricxon_b200.config import ConfigError, config_from_dict, resolve_architecture
from matricxon_b200.config.palelix import PalelixConfig
from matricxon_b200.models.decoder import model_weight_specs, plan_cache
from matricxon_b200.parts.base import Runtime, StateRequest, part_class
from matricxon_b200.parts.spec import DeltaRuleSpec, RetentionSpec, RoutedExpertsSpec
from palelix_configs import MODELS, RANKS, config_of, delta, dense, draw, ids, lightning, model, moe, parallel, single_layer

F64 = torch.float64


def doubles(tensors):
    return {name: value.double() for name, value in tensors.items()}


@pytest.mark.parametrize("name", list(MODELS))
def test_registry_and_round_trip(name):
    raw = MODELS[name]
    assert resolve_architecture(raw).config_class is PalelixConfig
    config = config_from_dict(copy.deepcopy(raw))
    assert config.to_dict() == raw
    assert config_from_dict(config.to_dict()) == config


def test_tensor_names_and_shapes():
    shapes = {w.name: tuple(w.shape) for w in model_weight_specs(config_of(MODELS["A"]).model_spec())}
    assert shapes["embed"] == (211, 96) and shapes["head"] == (211, 96) and shapes["final.norm"] == (96,)
    assert shapes["loop.step"] == (3, 96) and shapes["l0.norm1"] == (96,) and "l0.norm2" not in shapes
    p = "l0.mix.left."
    assert (shapes[p + "q"], shapes[p + "k"], shapes[p + "v"], shapes[p + "o"]) == ((144, 96), (72, 96), (120, 96), (96, 240))
    p = "l0.mix.right."
    assert (shapes[p + "q"], shapes[p + "k"], shapes[p + "v"], shapes[p + "o"]) == ((40, 96), (40, 96), (112, 96), (96, 112))
    assert (shapes[p + "q.conv"], shapes[p + "k.conv"], shapes[p + "v.conv"]) == ((40, 3), (40, 3), (112, 3))
    assert shapes[p + "b"] == (4, 96) and shapes[p + "A_log"] == (4,) and shapes[p + "norm"] == (28,)
    assert shapes[p + "a1"] == (RANKS["a1"], 96) and shapes[p + "a2"] == (80, RANKS["a1"]) and shapes[p + "dt_bias"] == (80,)
    assert shapes[p + "g1"] == (RANKS["g1"], 96) and shapes[p + "g2"] == (112, RANKS["g1"])
    assert shapes["l0.mlp.gate"] == (72, 96) and shapes["l0.mlp.up"] == (72, 96) and shapes["l0.mlp.down"] == (96, 72)
    assert shapes["l1.mix.q"] == (60, 96) and shapes["l1.mix.v"] == (84, 96) and shapes["l1.mix.g"] == (84, 96)
    assert shapes["l1.mix.norm"] == (84,) and shapes["l1.mix.o"] == (96, 84)
    assert not any(name.startswith("l1.mlp") for name in shapes)
    assert shapes["l2.mix.q"] == (24, 96) and shapes["l2.mix.v"] == (120, 96) and shapes["l2.mix.v.conv"] == (120, 5)
    assert shapes["l2.mix.a"] == (6, 96) and shapes["l2.mix.dt_bias"] == (6,) and shapes["l2.mix.norm"] == (20,)
    assert shapes["l2.mix.g"] == (120, 96) and "l2.mix.a1" not in shapes
    assert shapes["l2.mlp.router"] == (6, 96) and shapes["l2.mlp.e5.gate"] == (40, 96) and shapes["l2.mlp.e5.down"] == (96, 40)
    assert not any(name.endswith(".weight") for name in shapes)
    assert "loop.step" not in {w.name for w in model_weight_specs(config_of(MODELS["C"]).model_spec())}


def test_schedule_repeats_layers_with_caches_and_states_of_their_own():
    spec = config_of(MODELS["A"]).model_spec()
    assert [(e.layer, e.pass_index) for e in spec.schedule] == [(0, None), (1, None), (2, 0), (3, None), (2, 1), (3, None),
                                                                (2, 2), (3, None)]
    assert [(i, p) for i, p in plain.layer_runs(MODELS["A"])] == [(e.layer, e.pass_index) for e in spec.schedule]
    plan = plan_cache(spec)
    assert len(plan.groups) == 1 and plan.groups[0].entries == (0,) and plan.groups[0].request.head_dim == 48
    # five taps are run as eight, head sizes are filled up to multiples of four: [taps - 1][channels], then S
    deltas = StateRequest((7 * (2 * 2 * 12 + 6 * 20) + 6 * 20 * 12,))
    assert [plan.state_of_entry[i] for i in (2, 4, 6)] == [deltas] * 3
    assert plan.state_of_entry[0] == StateRequest((2 * (2 * 2 * 20 + 4 * 28) + 4 * 28 * 20,))
    assert plan.state_of_entry[1] == StateRequest((3, 20, 28)) and plan.state_of_entry[7] == StateRequest((2, 24, 16))
    b = plan_cache(config_of(MODELS["B"]).model_spec())
    assert sorted(len(g.entries) for g in b.groups) == [1, 2]             # the repeated attention layer twice
    d = plan_cache(config_of(MODELS["D"]).model_spec())
    assert d.groups == () and all(state is not None for state in d.state_of_entry) and len(d.state_of_entry) == 4


def test_what_the_description_says_of_the_mechanisms():
    spec = config_of(MODELS["A"]).model_spec()
    (left, left_scale, left_name), (right, right_scale, right_name) = spec.layers[0].mixer.branches
    assert (left_scale, left_name, right_scale, right_name) == (0.7, "left.", 1.4, "right.")
    assert left.query_norm_name is None and left.position.rotary_dim == 12 and left.mask == "causal" and left.gate is None
    assert right.decay == "channel" and right.gate == "sigmoid" and right.decay_rank == 7 and right.gate_rank == 10
    assert right.query_scale == 20 ** -0.5 and right.unit_eps == 1e-6 and right.taps == 3
    second, third = spec.layers[1].mixer, spec.layers[2].mixer
    assert second.activation == "silu" and second.norm == "all" and second.gate == "sigmoid" and second.key_scale == 1.0
    assert second.position is None and second.decay == (0.9, 0.99, 0.5)
    assert third.decay == "head" and third.gate == "silu" and third.num_kv_heads == 2 and third.decay_names == ("a",)
    routed = spec.layers[2].feed_forward
    assert routed.score == "softmax" and (routed.num_groups, routed.groups_kept, routed.group_best) == (3, 1, 1)
    assert (routed.expert.limit, routed.expert.slope, routed.expert.shift) == (0.8, 1.702, 1.0)
    assert spec.layers[0].feed_forward.activation == "silu" and spec.layers[1].feed_forward is None
    assert all(layer.block == "pre_norm_parallel" for layer in spec.layers) and not spec.tie_word_embeddings
    assert spec.pass_input.passes == 3 and config_of(MODELS["C"]).model_spec().pass_input is None
    assert config_of(MODELS["B"]).model_spec().layers[0].feed_forward.expert.limit is None


@pytest.mark.parametrize("change, key", [
    (lambda r: r["layers"][0].update(type="mamba"), "mamba"),
    (lambda r: r["layers"][0]["mixer"].pop("left"), "left"),
    (lambda r: r["layers"][0]["mixer"].pop("right"), "right"),
    (lambda r: r["layers"][0]["mixer"]["left"].update(kv_heads=4), "kv_heads"),
    (lambda r: r["layers"][0]["mixer"]["left"].update(vdim=300), "vdim"),
    (lambda r: r["layers"][0]["mixer"]["left"].pop("scale"), "scale"),
    (lambda r: r["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "dims"),
    (lambda r: r["layers"][0]["mixer"]["left"]["rot"].update(dims=26), "dims"),
    (lambda r: r["layers"][0]["mixer"]["right"].pop("conv"), "conv"),
    (lambda r: r["layers"][0]["mixer"]["right"].update(kv_heads=3), "kv_heads"),
    (lambda r: r["layers"][1]["mixer"].update(decay=[0.5]), "decay"),
    (lambda r: r["layers"][1]["mixer"].update(dim=320), "dim"),
    (lambda r: r["layers"][2]["mixer"].update(conv=17), "conv"),
    (lambda r: r["layers"][2]["mixer"].update(conv=0), "conv"),
    (lambda r: r["layers"][2]["mixer"].update(dim=257), "dim"),
    (lambda r: r["layers"][2]["mixer"].pop("heads"), "heads"),
    (lambda r: r["layers"][2]["mlp"]["router"].update(top=7), "top"),
    (lambda r: r["layers"][2]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda r: r["layers"][2]["mlp"]["router"]["groups"].update(keep=4), "groups"),
    (lambda r: r["layers"][2]["mlp"]["router"].update(top=3), "groups"),
    (lambda r: r["layers"][2]["mlp"]["expert"].update(limit=-1.0), "limit"),
    (lambda r: r["layers"][0]["mlp"].update(kind="sparse"), "sparse"),
    (lambda r: r["loop"].update(stop=5), "loop"),
    (lambda r: r["loop"].update(start=4), "loop"),
    (lambda r: r["loop"].pop("times"), "times"),
    (lambda r: r.pop("norm"), "norm"),
    (lambda r: r.pop("vocab"), "vocab"),
    (lambda r: r.update(layers=[]), "layers"),
])
def test_errors_name_the_key(change, key):
    raw = copy.deepcopy(MODELS["A"])
    change(raw)
    with pytest.raises(ConfigError, match=key):
        config_from_dict(raw)


def test_parts_refuse_what_they_cannot_do():
    runtime = Runtime(device="cpu", dtype=torch.float32)
    spec = config_of(MODELS["A"]).model_spec()
    routed = spec.layers[2].feed_forward
    with pytest.raises(ValueError, match="groups"):
        RoutedExpertsSpec(**{**vars(routed), "group_best": 2})
    with pytest.raises(ValueError, match="groups"):
        RoutedExpertsSpec(**{**vars(routed), "correction_name": "correction"})
    with pytest.raises(ValueError, match="fewer"):
        RoutedExpertsSpec(**{**vars(routed), "top": 3})
    third = spec.layers[2].mixer
    with pytest.raises(ValueError, match="two"):
        DeltaRuleSpec(**{**vars(third), "decay": "channel"})
    with pytest.raises(ValueError, match="taps"):
        DeltaRuleSpec(**{**vars(third), "taps": 17})
    second = spec.layers[1].mixer
    with pytest.raises(ValueError, match="weight"):
        RetentionSpec(**{**vars(second), "norm": "head"})
    with pytest.raises(ValueError, match="rotated"):
        position = spec.layers[0].mixer.branches[0][0].position
        part_class("mixer", "retention")(RetentionSpec(**{**vars(second), "position": position}), runtime, "")


# ---------------------------------------------------------------------- the plain model's own properties
def test_delta_rule_stores_replaces_and_forgets():
    key, other = torch.zeros(1, 4, dtype=F64), torch.zeros(1, 4, dtype=F64)
    key[0, 1], other[0, 2] = 1.0, 1.0
    v1, v2 = torch.tensor([[1.0, 2.0, 3.0]], dtype=F64), torch.tensor([[-4.0, 0.5, 1.0]], dtype=F64)
    ones = torch.ones(3, 1, 4, dtype=F64)
    # a full step replaces what is held under the key and leaves what is held under another
    o = plain.delta_rule(torch.stack([key, other, key]), torch.stack([key, other, key]), torch.stack([v1, v2, v2]), ones,
                         torch.ones(3, 1, dtype=F64))
    assert torch.allclose(o[0], v1) and torch.allclose(o[1], v2) and torch.allclose(o[2], v2)
    # a half step moves half way; the read-out sees the token's own write; a decay acts ahead of the correction
    g = ones * 0.5
    o = plain.delta_rule(torch.stack([key] * 2), torch.stack([key] * 2), torch.stack([v1, v2]), g[:2],
                         torch.full((2, 1), 0.5, dtype=F64))
    assert torch.allclose(o[0], v1 / 2) and torch.allclose(o[1], v1 / 4 + (v2 - v1 / 4) / 2)
    # a channel of its own: the decay of another row does not touch what is held under this key
    g = torch.ones(2, 1, 4, dtype=F64)
    g[:, :, 2] = 0.0
    o = plain.delta_rule(torch.stack([key] * 2), torch.stack([key, other]), torch.stack([v1, v2]), g, torch.ones(2, 1, dtype=F64))
    assert torch.allclose(o[1], v1)


def test_decaying_sum_against_its_closed_form():
    gen = torch.Generator().manual_seed(2)
    q, k, v = (torch.randn(12, 2, n, generator=gen, dtype=F64) for n in (4, 4, 3))
    decay = torch.tensor([0.9, 0.3], dtype=F64)
    o = plain.decaying_sum(q, k, v, decay)
    for t in (0, 7, 11):
        want = sum(decay[:, None] ** (t - j) * (q[t] * k[j]).sum(-1, keepdim=True) * v[j] for j in range(t + 1))
        assert torch.allclose(o[t], want)


def test_rotation_turns_by_the_distance_and_leaves_the_rest():
    gen = torch.Generator().manual_seed(1)
    q, k = torch.randn(1, 1, 12, generator=gen, dtype=F64), torch.randn(1, 1, 12, generator=gen, dtype=F64)
    rot = {"dims": 8, "base": 100.0}
    score = lambda p, j: float((plain.rotate(q, torch.tensor([p]), rot) * plain.rotate(k, torch.tensor([j]), rot)).sum())
    assert abs(score(40, 33) - score(1007, 1000)) < 1e-9 and abs(score(40, 33) - score(40, 32)) > 1e-4
    assert torch.equal(plain.rotate(q, torch.tensor([5]), rot)[..., 8:], q[..., 8:])


def test_convolution_looks_back_and_starts_from_zeros():
    u, w = torch.randn(9, 3, dtype=F64), torch.randn(3, 4, dtype=F64)
    y = plain.causal_conv(u, w)
    assert torch.allclose(y[0], w[:, 3] * u[0]) and torch.allclose(y[5], sum(w[:, j] * u[2 + j] for j in range(4)))


def test_groups_limit_the_choice_and_the_weights_are_shares():
    router = torch.eye(6, dtype=F64)
    h = torch.tensor([[5.0, 0.0, 4.0, 3.9, 1.0, 4.5]], dtype=F64)
    r = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}}
    assert plain.route(h, router, r)[0].tolist() == [[0, 1]]              # the group of the best expert alone
    r["groups"]["keep"] = 2
    assert plain.route(h, router, r)[0].tolist() == [[0, 5]]
    assert plain.route(h, router, {"experts": 6, "top": 3})[0].tolist() == [[0, 5, 2]]
    one = {k: torch.zeros(4, 3, dtype=F64) for k in ("gate", "up")}
    # with gate and up zero an expert gives nothing; clamps act on both sides
    assert float(plain.expert(torch.ones(1, 3, dtype=F64), one["gate"], one["up"], torch.ones(3, 4, dtype=F64), 1.0).abs().max()) == 0
    big = torch.full((1, 1), 50.0, dtype=F64)
    w = torch.ones(1, 1, dtype=F64)
    limited = plain.expert(big, w, w, w, 1.5)
    assert abs(float(limited) - 1.5 * float(torch.sigmoid(torch.tensor(1.702 * 1.5))) * 2.5) < 1e-6
    assert abs(float(plain.expert(-big, w, -w, w, 1.5))) < 1e-6           # the gate is not limited from below


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_every_tensor_is_used_and_a_prefix_does_not_depend_on_what_follows(name):
    raw = MODELS[name]
    weights = doubles(draw(raw, seed=5))
    tokens = ids(30, raw["vocab"], seed=2)
    full = plain.forward(raw, weights, tokens)
    assert torch.allclose(plain.forward(raw, weights, tokens[:20]), full[:20], atol=1e-9)
    moved_experts = 0
    for tensor in weights:
        changed = dict(weights)
        changed[tensor] = weights[tensor] * 1.5 + 0.01
        same = torch.allclose(plain.forward(raw, changed, tokens), full, atol=1e-9)
        if ".mlp.e" in tensor:
            moved_experts += not same                                  # an expert that nobody drew changes nothing
        elif not (tensor.endswith("router") and raw["layers"][int(tensor[1])]["mlp"]["router"]["experts"] == 1):
            assert not same, tensor
    assert moved_experts > 0


def test_both_sublayers_read_the_same_norm_and_every_pass_its_own_step():
    raw = model(32, 50, [dict(lightning(2, 8, 8, [0.5, 0.9]), mlp=dense(16)), delta(2, 1, 8, 8, 2)], loop=(0, 1, 2))
    w = doubles(draw(raw, seed=3))
    tokens = ids(6, 50, seed=1)
    taps = plain.forward(raw, w, tokens, return_layers=True)[1]
    assert taps.shape[0] == 3
    x = w["embed"][tokens] + w["loop.step"][0]
    h = plain.over_rms(x, 1e-5) * w["l0.norm1"]
    want = x + plain.lightning(h, w, "l0.mix.", raw["layers"][0]["mixer"], 1e-5) + plain.feed_forward(h, w, "l0.mlp.", dense(16))
    assert torch.allclose(taps[0], want)
    single = single_layer(parallel((2, 1, 8, 8, 0.3, None), (2, 1, 8, 8, 2), 0.0, 0.0), width=32)
    w = doubles(draw(single, seed=3))
    assert torch.allclose(plain.forward(single, w, tokens, return_layers=True)[1][0], w["embed"][tokens])
    assert moe(4, 2, 1)["expert"]["limit"] == 0.8
