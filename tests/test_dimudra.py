"""Dimudra on the CPU: configuration and its refusals, tensor names, the looped schedule, cache needs, the norm with a single
weight, and the plain functions against cases worked out by hand."""
import copy
import math

import pytest
import torch

from logssms_b200.config import ConfigError, make_model_config
from logssms_b200.models import build_model
from plain import dimudra_plain as P
from tiny_dimudra import DIMU, DIMU_A, DIMU_B, DIMU_D, DIMU_E

D = torch.float64


def test_config_round_trip_and_specs():
    cfg = make_model_config(DIMU_A)
    assert cfg.to_dict() == DIMU_A and cfg.architectures == ("Dimudra",)
    spec = cfg.model_spec()
    assert [b.mixer.spec.kind for b in spec.layers] == ["mixer_pair", "hgrn2", "gated_attention", "mixer_pair"]
    assert spec.embedding_multiplier == 3.0 and not spec.tie_word_embeddings and spec.final_norm.scalar
    pair = spec.layers[0].mixer.spec
    left, right = pair.left.spec, pair.right.spec
    assert (pair.left.out_scale, pair.right.out_scale) == (0.8, 1.3)
    assert (left.num_heads, left.num_kv_heads, left.head_dim, left.value_dim, left.window, left.softmax_scale) == (6, 2, 16, 24, 20, 0.3)
    assert left.proj_bias and left.qk_norm == "row" and left.position is None and not left.sink_zero
    assert (right.inner_size, right.state_size, right.dt_rank, right.conv_kernel) == (72, 12, 5, 4)
    rotary = spec.layers[2].mixer.spec
    assert rotary.sink_zero and rotary.qk_norm == "head_unit" and not rotary.proj_bias and rotary.window is None
    assert (rotary.position.rotary_dim, rotary.position.theta, rotary.value_dim) == (8, 500.0, 8)
    assert make_model_config(DIMU_E).model_spec().layers[1].mixer.spec.position is None
    moe = spec.layers[0].feed_forward
    assert (moe.num_experts, moe.top, moe.num_groups, moe.keep_groups, moe.expert_size, moe.shared_size) == (12, 3, 4, 2, 16, 24)
    assert moe.score == "sigmoid" and moe.normalize and moe.group_score == "pair" and moe.shared_gate and moe.correction
    assert spec.layers[3].feed_forward is None and spec.layers[3].feed_forward_norm is None
    assert all(b.input_conv == 3 for b in spec.layers)


def test_looped_schedule():
    runs = lambda raw: [(e.layer, e.cache, e.opens) for e in make_model_config(raw).model_spec().schedule]
    assert runs(DIMU_A) == [(0, 0, None), (1, 1, None), (2, 2, None), (1, 3, 0), (2, 4, None), (1, 5, 0), (2, 6, None), (3, 7, None)]
    assert runs(DIMU_B) == [(0, 0, None), (1, 1, None), (2, 2, None), (0, 3, 0), (1, 4, None), (2, 5, None)]
    assert runs(DIMU_D) == [(0, 0, None), (1, 1, None)]                       # an empty range
    assert runs(DIMU_E) == [(0, 0, None), (1, 1, None), (2, 2, None), (2, 3, 0), (2, 4, 0), (2, 5, 0), (3, 6, None)]
    none = copy.deepcopy(DIMU_A)
    del none["loop"]
    assert [e.layer for e in make_model_config(none).model_spec().schedule] == [0, 1, 2, 3]
    for raw in DIMU.values():                                                  # the plain model runs the layers in the same order
        assert P.layer_runs(raw) == make_model_config(raw).layer_runs()


@pytest.mark.parametrize("path, value, word", [
    (("layers", 0, "type"), "convolution", "not a mixer"),
    (("layers", 0, "mixer", "left", "heads"), 5, "multiple of kv_heads"),
    (("layers", 0, "mixer", "left", "mask", "size"), 0, "positive"),
    (("layers", 0, "mixer", "right", "conv"), 9, "taps"),
    (("layers", 0, "mixer", "right", "state"), 257, "at most"),
    (("layers", 0, "mixer", "right", "dt_rank"), 0, "positive"),
    (("layers", 1, "mixer", "vdim"), 0, "positive"),
    (("layers", 1, "mixer", "dim"), 513, "at most"),
    (("layers", 2, "mixer", "vdim"), 257, "at most"),
    (("layers", 0, "mlp", "router", "experts"), 260, "at most"),
    (("layers", 2, "mixer", "rot", "dims"), 7, "even"),
    (("layers", 2, "mixer", "rot", "dims"), 18, "at most"),
    (("layers", 2, "mixer", "rot", "base"), 0.0, "positive"),
    (("layers", 0, "mlp", "kind"), "dense", "not 'moe'"),
    (("layers", 0, "mlp", "router", "top"), 13, "top"),
    (("layers", 0, "mlp", "router", "groups", "count"), 5, "multiple of groups.count"),
    (("layers", 0, "mlp", "router", "groups", "keep"), 5, "keep"),
    (("layers", 2, "mlp", "router", "top"), 5, "keep"),
    (("canon", "taps"), 0, "taps"),
    (("loop", "stop"), 9, "loop"),
    (("norm", "eps"), 0.0, "positive"),
    (("vocab",), 0, "positive"),
])
def test_config_refusals(path, value, word):
    raw = copy.deepcopy(DIMU_A)
    at = raw
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=word):
        make_model_config(raw)


def test_missing_keys_are_refused():
    for drop in (("layers",), ("width",), ("norm",), ("canon",), ("embedding",), ("layers", 0, "mixer", "left", "scale"),
                 ("layers", 0, "mixer", "left_scale"), ("layers", 0, "mixer", "right", "inner"), ("layers", 1, "mixer", "dim"), ("layers", 0, "mlp", "router")):
        raw = copy.deepcopy(DIMU_A)
        at = raw
        for key in drop[:-1]:
            at = at[key]
        del at[drop[-1]]
        with pytest.raises(ConfigError):
            make_model_config(raw)


def test_tensor_names_and_shapes():
    model = build_model(make_model_config(DIMU_A))
    shapes = {n: tuple(s.shape) for n, s in model.named_param_specs()}
    assert shapes["embed"] == (211, 64) and shapes["head"] == (211, 64) and shapes["final.norm"] == ()
    assert shapes["l0.norm1"] == shapes["l0.norm2"] == () and shapes["l0.canon1"] == (64, 3)
    L = "l0.mix.left."
    assert shapes[L + "q"] == (96, 64) and shapes[L + "k"] == (32, 64) and shapes[L + "v"] == (48, 64) and shapes[L + "g"] == (144, 64)
    assert shapes[L + "o"] == (64, 144) and shapes[L + "q.b"] == shapes[L + "q.norm"] == (96,) and shapes[L + "k.b"] == shapes[L + "k.norm"] == (32,)
    assert shapes[L + "v.b"] == (48,) and L + "g.b" not in shapes
    R = "l0.mix.right."
    assert shapes[R + "in"] == (144, 64) and shapes[R + "conv"] == (72, 4) and shapes[R + "conv.b"] == (72,) and shapes[R + "x"] == (29, 72)
    assert shapes[R + "dt"] == (72, 5) and shapes[R + "dt.b"] == (72,) and shapes[R + "A_log"] == (72, 12) and shapes[R + "D"] == (72,)
    assert shapes[R + "o"] == (64, 72)
    assert shapes["l1.mix.q"] == shapes["l1.mix.f"] == (48, 64) and shapes["l1.mix.f.b"] == shapes["l1.mix.lower"] == (48,)
    assert shapes["l1.mix.v"] == (72, 64) and shapes["l1.mix.norm"] == (24,) and shapes["l1.mix.o"] == (64, 72)
    assert shapes["l2.mix.q"] == (64, 64) and shapes["l2.mix.v"] == (16, 64) and shapes["l2.mix.g"] == (32, 64)
    assert not any(n.startswith("l2.mix.") and (n.endswith(".b") or "norm" in n) for n in shapes)
    assert shapes["l0.mlp.router"] == (12, 64) and shapes["l0.mlp.correction"] == (12,) and shapes["l0.mlp.e11.down"] == (64, 16)
    assert shapes["l0.mlp.shared.sg"] == (1, 64) and shapes["l0.mlp.shared.up"] == (24, 64)
    assert "l3.norm2" not in shapes and "l3.mlp.router" not in shapes and shapes["l3.norm1"] == ()
    assert not any(n.startswith("loop") for n in shapes)


def test_cache_needs():
    needs = build_model(make_model_config(DIMU_A)).cache_needs()
    assert len(needs) == 8
    assert needs[0].kv.window == 20 and [t.shape for t in needs[0].kv.tensors] == [(2, 16), (2, 24)]
    assert [(s.name, s.shape, s.dtype) for s in needs[0].states] == [("conv", (72, 3), None), ("scan", (72, 12), torch.float32), ("input_conv", (64, 2), None)]
    assert needs[1].kv is None and [(s.name, s.shape, s.dtype) for s in needs[1].states] == [("hgrn2", (3, 16, 24), torch.float32), ("input_conv", (64, 2), None)]
    assert needs[2].kv.window is None and needs[1] == needs[3] == needs[5] and needs[2] == needs[4] == needs[6]
    one_tap = build_model(make_model_config(DIMU_B)).cache_needs()
    assert one_tap[0].states == () and [s.name for s in one_tap[2].states] == ["conv", "scan"]
    assert all(n.kv is None for n in build_model(make_model_config(DIMU_D)).cache_needs())


def test_every_tiny_configuration_builds():
    for name, raw in DIMU.items():
        model = build_model(make_model_config(raw))
        assert len(model.cache_needs()) == model.num_cache_layers, name


def test_norm_with_a_single_weight_spreads_it():
    from logssms_b200.config.specs import NormSpec
    from logssms_b200.parts import RMSNorm
    norm = RMSNorm(NormSpec(5, 1e-5, param_name="", scalar=True))
    assert tuple(norm.param_specs()[""].shape) == ()
    norm.bind({"": torch.tensor(0.25)})
    assert norm.weight.tolist() == [0.25] * 5 and norm.weight.is_contiguous()
    around = RMSNorm(NormSpec(3, 1e-5, param_name="", scalar=True, offset=1.0))
    around.bind({"": torch.tensor(0.25)})
    assert around.weight.tolist() == [1.25] * 3


def test_input_convolution_holds_its_input_on_the_last_tap():
    from logssms_b200.parts import InputConv
    conv = InputConv(2, 3)
    stored = torch.tensor([[1.0, 2.0, 3.0], [4.0, 5.0, 6.0]])
    conv.bind({"": stored})
    assert conv.weight.tolist() == [[1.0, 2.0, 4.0], [4.0, 5.0, 7.0]] and stored[0, 2] == 3.0
    assert InputConv(2, 1).state_needs() == ()
    with pytest.raises(ValueError, match="taps"):
        InputConv(2, 9)


def test_routed_feed_forward_refuses_a_gate_without_a_shared_expert():
    from logssms_b200.config.specs import RoutedMLPSpec
    from logssms_b200.parts import RoutedMLP
    base = dict(hidden_size=8, expert_size=4, num_experts=4, num_identity=0, top=2, num_groups=2, keep_groups=1, route_scale=1.0, limit=0.0,
                score="sigmoid", expert="silu")
    with pytest.raises(ValueError, match="shared expert"):
        RoutedMLP(RoutedMLPSpec(**base, shared_gate=True))
    with pytest.raises(ValueError, match="best member or pair"):
        RoutedMLP(RoutedMLPSpec(**base, group_score="sum"))


def test_plain_convolution_rotation_and_softmax_by_hand():
    # the last column is the current token's, zeros before the start; the mixer reads the input on top
    u = torch.tensor([[1.0], [2.0], [4.0]], dtype=D)
    w = torch.tensor([[100.0, 10.0, 1.0]], dtype=D)
    assert P.short_conv(u, w).flatten().tolist() == [1.0, 12.0, 124.0]
    assert P.input_conv(u, w).flatten().tolist() == [2.0, 14.0, 128.0]
    # halves: columns 0 and 2 of the first four turn together, column 4 stays
    q = torch.tensor([[[1.0, 0.0, 0.0, 2.0, 5.0]]], dtype=D).repeat(2, 1, 1)
    r = P.rotate_halves(q, torch.tensor([0, 3]), {"dims": 4, "base": 16.0})
    assert torch.allclose(r[0], q[0])
    c, s, c2, s2 = math.cos(3.0), math.sin(3.0), math.cos(0.75), math.sin(0.75)       # frequencies 1 and 16^(-1/2)
    assert torch.allclose(r[1, 0], torch.tensor([c, -2 * s2, s, 2 * c2, 5.0], dtype=D))
    # equal scores: one added to the denominator gives weights 1 / (n + 1), without it 1 / n; a window of 2
    k = torch.zeros(3, 1, 1, dtype=D)
    v = torch.tensor([[[1.0]], [[2.0]], [[4.0]]], dtype=D)
    assert torch.allclose(P.softmax_attention(k, k, v, 1.0, None, 1.0).flatten(), torch.tensor([1 / 2, 3 / 3, 7 / 4], dtype=D))
    assert torch.allclose(P.softmax_attention(k, k, v, 1.0, 2, 0.0).flatten(), torch.tensor([1.0, 3 / 2, 6 / 2], dtype=D))
    # grouped: query heads 0, 1 read key/value head 0, query heads 2, 3 head 1
    v2 = torch.tensor([[[1.0], [10.0]]], dtype=D)
    z = torch.zeros(1, 4, 1, dtype=D)
    assert P.softmax_attention(z, torch.zeros(1, 2, 1, dtype=D), v2, 1.0, None, 0.0).flatten().tolist() == [1.0, 1.0, 10.0, 10.0]


def test_plain_recurrences_by_hand():
    # forget gate 1/4 then 1/2, values 8 and 4, q = 1 and 3: S = 3/4 * 8 = 6, then 1/2 * 6 + 1/2 * 4 = 5
    f = torch.tensor([[[0.25]], [[0.5]]], dtype=D)
    v = torch.tensor([[[8.0]], [[4.0]]], dtype=D)
    q = torch.tensor([[[1.0]], [[3.0]]], dtype=D)
    assert P.gated_recurrence(q, f, v).flatten().tolist() == [6.0, 15.0]
    # one channel, two states: dt 1 and 2, A = -1 and -2, B = (1, 2), C = (1, 1) then (0, 3), D = 10
    x, dt = torch.tensor([[2.0], [3.0]], dtype=D), torch.tensor([[1.0], [2.0]], dtype=D)
    A = torch.tensor([[-1.0, -2.0]], dtype=D)
    B, C = torch.tensor([[1.0, 2.0], [1.0, 0.0]], dtype=D), torch.tensor([[1.0, 1.0], [0.0, 3.0]], dtype=D)
    y = P.selective_scan(x, dt, A, B, C, torch.tensor([10.0], dtype=D))
    assert torch.allclose(y.flatten(), torch.tensor([2.0 + 4.0 + 20.0, 3 * math.exp(-4.0) * 4.0 + 30.0], dtype=D))


def test_plain_router_by_hand():
    # six experts in three groups of two, two groups stay, three chosen.  Scores s = sigmoid(z); the correction moves the choice only.
    s = torch.tensor([0.9, 0.1, 0.6, 0.5, 0.2, 0.3], dtype=D)
    z = torch.log(s / (1 - s))[None]
    # without correction: group sums 1.0, 1.1, 0.5 -> groups 1 and 0 stay; experts 0, 2, 3
    w = P.route(z, torch.zeros(6, dtype=D), 3, 3, 2)[0]
    assert torch.allclose(w, torch.tensor([0.9, 0.0, 0.6, 0.5, 0.0, 0.0], dtype=D) / 2.0)
    # a correction that makes group 2 win although its members lose elsewhere, and negative choice scores that still beat the
    # experts of a group that left: group sums -0.9, 1.1, 1.1 -> groups 1, 2 stay, top 4 takes them all
    c = torch.tensor([-1.0, -1.0, 0.0, 0.0, 0.6, 0.0], dtype=D)
    w = P.route(z, c, 4, 3, 2)[0]
    assert torch.allclose(w, torch.tensor([0.0, 0.0, 0.6, 0.5, 0.2, 0.3], dtype=D) / 1.6)
    # all choice scores negative: the group that left (not zero, but out) is never chosen
    w = P.route(z, torch.full((6,), -2.0, dtype=D), 3, 3, 2)[0]
    assert float(w[4]) == 0.0 and float(w[5]) == 0.0 and int((w > 0).sum()) == 3
