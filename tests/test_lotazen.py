"""Lotazen without a GPU: configuration and refusals, tensor names and shapes, what each layer keeps per request, how the
sublayers' first products are joined, and the plain functions against closed forms."""
import copy
import math

import pytest
import torch

from qwen_inference_lab_b200.config import registry
from qwen_inference_lab_b200.config.model_config import ConfigError, LotazenConfig
from qwen_inference_lab_b200.parts import JointProjection, KVCacheSpec, RotaryFrequencies, StackedLinear, StateSpec
from tests import lotazen_cases as cases
from tests.plain import lotazen_plain as plain

F64 = torch.float64


def build(config, shapes=None):
    return registry.lookup(config).build(LotazenConfig.from_dict(config), tensor_shapes=shapes)


def test_the_registry_builds_the_model_with_the_design_names():
    entry = registry.lookup(cases.CASE_A)
    assert entry.config_class is LotazenConfig
    model = build(cases.CASE_A)
    params = model.all_named_params()
    expected = {"embed": (173, 96), "pos": (400, 96), "final.norm": (), "head": (173, 96), "l0.norm1": (),
                "l0.mix.left.q": (128, 96), "l0.mix.left.k": (64, 96), "l0.mix.left.v": (64, 96), "l0.mix.left.o": (96, 128),
                "l0.mix.right.q": (72, 96), "l0.mix.right.f": (72, 96), "l0.mix.right.f.b": (72,),
                "l0.mix.right.lower": (72,), "l0.mix.right.v": (48, 96), "l0.mix.right.norm": (16,),
                "l0.mix.right.o": (96, 48), "l0.mlp.router": (4, 96), "l0.mlp.e3.gate": (24, 96), "l0.mlp.e0.up": (24, 96),
                "l0.mlp.e0.down": (96, 24), "l0.mlp.shared.gate": (40, 96), "l0.mlp.shared.up": (40, 96),
                "l0.mlp.shared.down": (96, 40), "l1.mix.q": (60, 96), "l1.mix.k": (60, 96), "l1.mix.v": (84, 96),
                "l1.mix.g": (84, 96), "l1.mix.o": (96, 84), "l1.mix.norm": (84,), "l1.mix.i": (3, 96), "l1.mix.i.b": (3,),
                "l1.mix.f": (3, 96), "l1.mix.f.b": (3,), "l2.mix.q": (80, 96), "l3.mlp.e4.up": (32, 96)}
    for name, shape in expected.items():
        assert name in params and params[name].shape == shape, name
    absent = ("l0.mix.left.q.b", "l0.norm2", "l2.mlp.router", "l2.norm2", "l0.mlp.e4.gate", "l0.mix.right.k", "l1.mix.o.b")
    assert not any(name in params for name in absent)
    assert model.stream_dtype == torch.float32 and model.logit_softcap == 25.0 and model.max_positions == 400
    assert build(cases.CASE_B).logit_softcap == 0.0
    assert "l0.mlp.shared.gate" not in build(cases.CASE_B).all_named_params()


def test_the_table_of_positions_is_the_checkpoints():
    shorter = build(cases.CASE_A, {"pos": (123, 96)})
    assert shorter.all_named_params()["pos"].shape == (123, 96) and shorter.max_positions == 123
    longer = build(cases.CASE_A, {"pos": (1000, 96)})
    assert longer.all_named_params()["pos"].shape == (1000, 96) and longer.max_positions == 400


def test_what_a_layer_keeps_per_request():
    specs = build(cases.CASE_A).cache_specs()
    assert specs[0] == (KVCacheSpec(2, 32, 24), StateSpec((3, 24, 16)))       # pages behind the window go back
    assert specs[1] == (StateSpec((3, 20, 29)), StateSpec((3,)))              # the memory with its sum of keys, the maximum
    assert specs[2] == (StateSpec((2, 40, 17)), StateSpec((2,)))
    assert build(cases.CASE_C).cache_specs()[2][0] == KVCacheSpec(2, 24, 33, 40)


@pytest.mark.parametrize("change,message", [
    (lambda c: c.pop("max_positions"), "max_positions"),
    (lambda c: c["norm"].update(eps=0), "norm.eps"),
    (lambda c: c["layers"][0].update(type="attention"), "none of parallel"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "do not divide"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=34), "rot"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(factor=0), "scaling"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "mask"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][0]["mixer"].pop("right_scale"), "right_scale"),
    (lambda c: c["layers"][1]["mixer"].update(gate_cap=0.0), "gate_cap"),
    (lambda c: c["layers"][1]["mlp"].update(kind="dense"), "not moe"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=4), "top"),
    (lambda c: c["layers"][1]["mlp"]["shared"].pop("limit"), "shared"),
    (lambda c: c["layers"][1]["mlp"].pop("expert"), "expert"),
    (lambda c: c.update(logit_softcap=-1.0), "logit_softcap"),
])
def test_refused_configurations(change, message):
    config = copy.deepcopy(cases.CASE_A)
    change(config)
    with pytest.raises(ConfigError, match=message):
        LotazenConfig.from_dict(config)


def test_joined_projections_keep_every_part_in_reach():
    """The stacked weights lie one below the other from rows that are multiples of eight; every part's own weight is a
    view of them, and its columns in the joint rows are its own product."""
    a, b = StackedLinear(12, [("a.q", 5), ("a.k", 6)], suffixes=("", ".b")), StackedLinear(12, [("b.g", 9)], suffixes=("", ".b"))
    values = {}
    for part in (a, b):
        for name, param in part.named_params().items():
            values[name] = param.data = torch.randn(param.shape, generator=torch.Generator().manual_seed(len(name) + param.shape[0]))
        part.finalize("cpu", torch.float32)
    joint = JointProjection([a, b])
    joint.join()
    assert joint._weight().shape == (16 + 16, 12) and joint._first == {id(a): 0, id(b): 16}
    assert torch.equal(a._weight(), torch.cat([values["a.q"], values["a.k"]])) and torch.equal(b._weight(), values["b.g"])
    assert a._weight().data_ptr() == joint._weight().data_ptr()
    assert b._weight().data_ptr() == joint._weight()[16:].data_ptr() and not joint._weight()[11:16].any()
    single = JointProjection([a])
    single.join()
    assert single._weight() is None and single.forward_joint(None, None) is None


def test_stretched_frequencies_and_pairs_of_neighbours():
    part = RotaryFrequencies(8, 500.0, "interleaved", stretch=4.0)
    bare = RotaryFrequencies(8, 500.0, "interleaved")
    assert part.frequencies() == [f / 4.0 for f in bare.frequencies()]
    with pytest.raises(ValueError):
        RotaryFrequencies(8, 500.0, stretch=0.0)
    rot = dict(base=100.0, dims=4, scaling=dict(factor=2.0))
    x = torch.zeros(3, 1, 6, dtype=F64)
    x[:, 0, 0], x[:, 0, 2], x[:, 0, 5] = 1.0, 1.0, 7.0
    out = plain.rotate_neighbours(x, rot)
    for p in range(3):
        for first, f in ((0, 0.5), (2, 0.05)):
            assert abs(out[p, 0, first] - math.cos(p * f)) < 1e-12 and abs(out[p, 0, first + 1] - math.sin(p * f)) < 1e-12
        assert out[p, 0, 4] == 0 and out[p, 0, 5] == 7.0
    assert torch.equal(plain.rotate_neighbours(x[2:], rot, first=2), out[2:])


def test_a_weightless_norm_commutes_with_the_rotation():
    rot = dict(base=50.0, dims=6, scaling=dict(factor=3.0))
    x = torch.randn(9, 2, 10, dtype=F64, generator=torch.Generator().manual_seed(1))
    torch.testing.assert_close(plain.unit_rms(plain.rotate_neighbours(x, rot), 1e-3),
                               plain.rotate_neighbours(plain.unit_rms(x, 1e-3), rot))


def test_who_sees_whom():
    """Zero queries: every key scores zero, so position i gets the mean of the values it sees."""
    T, window = 9, 4
    v = torch.randn(T, 1, 3, dtype=F64, generator=torch.Generator().manual_seed(2))
    out = plain.window_attention(torch.zeros(T, 2, 5, dtype=F64), torch.randn(T, 1, 5, dtype=F64), v, 5.0, window)
    for i in range(T):
        torch.testing.assert_close(out[i, 1], v[max(0, i - 3):i + 1, 0].mean(0))


def test_the_tied_gate_blends_what_it_holds_with_what_comes():
    """A constant gate f: S_t = (1 - f) sum_j f^(t - j) v_j, a running average."""
    T, f = 7, 0.8
    v = torch.randn(T, 1, 2, dtype=F64, generator=torch.Generator().manual_seed(3))
    out, S = plain.tied_gate_scan(torch.ones(T, 1, 1, dtype=F64), torch.full((T, 1, 1), f, dtype=F64), v)
    for t in range(T):
        torch.testing.assert_close(out[t, 0], sum((1 - f) * f ** (t - j) * v[j, 0] for j in range(t + 1)))
    lower = torch.tensor([0.0, 0.25, 1.0], dtype=F64)
    gate = plain.forget_gate(torch.zeros(3, dtype=F64), torch.zeros(3, dtype=F64), lower)
    torch.testing.assert_close(gate, torch.tensor([0.5, 0.625, 1.0], dtype=F64))


def test_the_matrix_memory_does_not_depend_on_its_running_maximum():
    """The maximum scales memory and sum of keys alike; unscaled, S_t = sum_j exp(i_j + f_(j+1) + .. + f_t) k_j v_j^T and
    o_t = S^T q / max(|n . q|, 1): the floor exp(-m) stands for the one, since the maximum starts at zero."""
    g = torch.Generator().manual_seed(4)
    T, d, e = 12, 3, 2
    q, k, v = (torch.randn(T, 1, n, dtype=F64, generator=g) for n in (d, d, e))
    log_i, log_f = 3 * torch.randn(T, 1, dtype=F64, generator=g), -torch.rand(T, 1, dtype=F64, generator=g)
    out, (_, _, m) = plain.mlstm_scan(q, k, v, log_i, log_f)
    for t in range(T):
        weight = [math.exp(float(log_i[j] + log_f[j + 1:t + 1].sum())) for j in range(t + 1)]
        S = sum(a * k[j, 0][:, None] * v[j, 0][None, :] for j, a in enumerate(weight))
        n = sum(a * k[j, 0] for j, a in enumerate(weight))
        torch.testing.assert_close(out[t, 0], S.t() @ q[t, 0] / max(abs(float(n @ q[t, 0])), 1.0), atol=1e-5, rtol=1e-5)
    # gates that write next to nothing: the floor keeps the output small, m stays at the decayed zero
    faint, (_, _, m) = plain.mlstm_scan(q, k, v, torch.full((T, 1), -20.0, dtype=F64), torch.zeros(T, 1, dtype=F64))
    assert float(m[0]) == 0.0 and float(faint.abs().max()) < 1e-6


def test_an_expert_gets_its_score_times_the_input():
    m = cases.moe(4, 2, 5, 0.7, (6, 0.4))
    g = torch.Generator().manual_seed(5)
    width = 8
    w = {"f.router": torch.randn(4, width, generator=g, dtype=F64)}
    for prefix, ff in [(f"f.e{i}.", 5) for i in range(4)] + [("f.shared.", 6)]:
        w.update({prefix + "gate": torch.randn(ff, width, generator=g, dtype=F64), prefix + "up": torch.randn(ff, width, generator=g, dtype=F64),
                  prefix + "down": torch.randn(width, ff, generator=g, dtype=F64)})
    h = torch.randn(6, width, generator=g, dtype=F64)
    out = plain.routed_experts(h, w, "f.", m)
    scores = torch.sigmoid(h @ w["f.router"].t())
    for t in range(6):
        expected = plain.clamped_expert(h[t], w, "f.shared.", 0.4)
        for i in sorted(range(4), key=lambda e: -float(scores[t, e]))[:2]:
            expected = expected + plain.clamped_expert(scores[t, i] * h[t], w, f"f.e{i}.", 0.7)
        torch.testing.assert_close(out[t], expected)
    # both of the bounds hold: a huge positive input gives limit * sigmoid(1.702 limit) * (1 + limit)
    one = {"e.gate": torch.ones(1, 1, dtype=F64), "e.up": torch.ones(1, 1, dtype=F64), "e.down": torch.ones(1, 1, dtype=F64)}
    torch.testing.assert_close(plain.clamped_expert(torch.full((1, 1), 100.0, dtype=F64), one, "e.", 0.5),
                               torch.full((1, 1), 0.5 / (1 + math.exp(-1.702 * 0.5)) * 1.5, dtype=F64))


def test_positions_are_added_and_the_norm_has_one_number():
    config = dict(architecture="Lotazen", vocab=5, width=4, norm=dict(eps=0.1), max_positions=3, logit_softcap=2.0,
                  layers=[dict(cases.mlstm(1, 2, 2, 1.0), mlp=None)])
    weights = cases.make_weights(config, 1)
    for name in weights:
        if name.startswith("l0.mix.") and name != "l0.mix.norm":
            weights[name] = torch.zeros_like(weights[name])
    logits, after = plain.forward(config, weights, [4, 0, 4], return_layers=True)
    x = (weights["embed"][[4, 0, 4]] + weights["pos"]).double()
    torch.testing.assert_close(after[0], x)                                # a mixer that gives nothing
    h = x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + 0.1) * weights["final.norm"].double()
    torch.testing.assert_close(logits, 2.0 * torch.tanh(h @ weights["head"].double().t() / 2.0))
