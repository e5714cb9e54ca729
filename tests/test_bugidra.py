"""Bugidra without a GPU: configuration and refusals, tensor names and shapes, what each layer keeps per request, YaRN's ramp,
who mixes whose values, and the plain functions against closed forms."""
import copy
import math

import pytest
import torch

from qwen_inference_lab_b200.config import registry
from qwen_inference_lab_b200.config.model_config import BugidraConfig, ConfigError
from qwen_inference_lab_b200.parts import (DeferredPreNormBlock, GatedDeltaRule, GroupedQueryAttention, KVCacheSpec, ParallelMixers,
                                           Retention, RotaryFrequencies, StateSpec)
from tests import bugidra_cases as cases
from tests.plain import bugidra_plain as plain

F64 = torch.float64


def build(config):
    return registry.lookup(config).build(BugidraConfig.from_dict(config))


def rows(count, width, seed, scale=1.0):
    return torch.randn(count, width, generator=torch.Generator().manual_seed(seed), dtype=F64) * scale


def test_the_registry_builds_the_model_with_the_design_names():
    assert registry.lookup(cases.CASE_A).config_class is BugidraConfig
    model = build(cases.CASE_A)
    params = model.all_named_params()
    expected = {"embed": (173, 96), "head": (173, 96), "final.norm": (96,), "final.norm.b": (96,), "final.norm.alpha": (),
                "l0.norm1": (96,), "l0.norm1.b": (96,), "l0.norm1.alpha": (), "l0.norm2.alpha": (),
                "l0.mix.left.q": (128, 96), "l0.mix.left.k": (64, 96), "l0.mix.left.v": (32, 96), "l0.mix.left.o": (96, 64),
                "l0.mix.left.out": (96,), "l0.mix.right.out": (96,), "l0.mix.right.q": (72, 96), "l0.mix.right.k": (72, 96),
                "l0.mix.right.v": (48, 96), "l0.mix.right.g": (48, 96), "l0.mix.right.o": (96, 48), "l0.mlp.gate": (80, 96),
                "l0.mlp.up": (80, 96), "l0.mlp.down": (96, 80), "l1.mix.q": (128, 96), "l1.mix.k": (64, 96), "l1.mix.v": (64, 96),
                "l1.mix.q.norm": (128,), "l1.mix.k.norm": (64,), "l1.mix.vmix": (), "l1.mix.g": (128, 96), "l1.mix.o": (96, 128),
                "l2.mix.q": (32, 96), "l2.mix.q.conv": (32, 4), "l2.mix.k.conv": (32, 4), "l2.mix.v": (96, 96),
                "l2.mix.v.conv": (96, 4), "l2.mix.g": (96, 96), "l2.mix.b": (4, 96), "l2.mix.a": (4, 96), "l2.mix.A_log": (4,),
                "l2.mix.dt_bias": (4,), "l2.mix.norm": (24,), "l2.mix.o": (96, 96)}
    for name, shape in expected.items():
        assert name in params and params[name].shape == shape, name
    assert not any(name in params for name in ("l2.mlp.gate", "l4.mix.vmix", "l0.mix.left.q.norm", "l0.mix.right.norm", "l1.mix.q.b"))
    assert params["l2.norm2"].optional and not params["l0.norm2"].optional       # a layer without a feed-forward
    assert model.stream_dtype == torch.float32 and model.embedding.scale == 3.0
    assert all(isinstance(layer, DeferredPreNormBlock) for layer in model.layers)


def test_the_first_mixing_layer_hands_its_values_on():
    mixers = [layer.mixer for layer in build(cases.CASE_A).layers]
    assert [getattr(m, "first_values", None) for m in mixers] == [None, True, None, False, False, False]
    assert [getattr(m, "mixes_values", None) for m in mixers] == [None, True, None, True, False, True]
    params = build(cases.CASE_A).all_named_params()
    assert params["l1.mix.vmix"].optional and not params["l3.mix.vmix"].optional


def test_what_a_layer_keeps_per_request():
    specs = build(cases.CASE_A).cache_specs()
    assert specs[0] == (KVCacheSpec(2, 32, 0, 16), StateSpec((3, 24, 16)))
    assert specs[1] == KVCacheSpec(2, 32)
    assert specs[2] == (StateSpec((4, 16, 24)), StateSpec((3, 160)))          # the matrices, the convolution's earlier rows
    assert specs[3] == KVCacheSpec(1, 48, 0, 64)
    assert build(cases.CASE_B).cache_specs()[0] == StateSpec((1, 130, 40))    # one tap reaches back to nothing


@pytest.mark.parametrize("change,message", [
    (lambda c: c.update(width=0), "width"),
    (lambda c: c["norm"].update(eps=0), "norm.eps"),
    (lambda c: c.update(embedding=dict(scale="big")), "embedding.scale"),
    (lambda c: c["layers"][0].update(type="mamba"), "none of delta"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "do not divide"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=34), "rot"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("slow"), "scaling"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(base=1.0), "base above one"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5]), "decay"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5, 1.5, 0.1]), "decay"),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("rot"), "rot"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=-1.0), "softcap"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][3]["mixer"].update(vdim=32), "different widths"),
    (lambda c: c["layers"][2]["mixer"].update(kv_heads=3), "do not divide"),
    (lambda c: c["layers"][2]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][2]["mixer"].update(conv=40), "taps"),
    (lambda c: c["layers"][1]["mlp"].update(kind="moe"), "dense"),
])
def test_refused_configurations(change, message):
    config = copy.deepcopy(cases.CASE_A)
    change(config)
    with pytest.raises(ConfigError, match=message):
        BugidraConfig.from_dict(config)


def test_a_configuration_comes_back_as_it_was():
    config = BugidraConfig.from_dict(cases.CASE_D)
    assert config == BugidraConfig.from_dict(config.to_dict()) and config.to_dict()["layers"] == cases.CASE_D["layers"]
    bare = copy.deepcopy(cases.CASE_D)
    bare.pop("embedding")
    assert BugidraConfig.from_dict(bare).embedding_scale == 1.0


ROTATIONS = [cases.rot(20000.0, 48, (2.5, 900, 24.0, 1.5)), cases.rot(500.0, 8, (4.0, 64, 8.0, 1.0)), cases.rot(100.0, 2, (16.0, 500, 64.0, 3.0)),
             cases.rot(2.0, 16, (3.0, 10, 100.0, 50.0)), cases.rot(1e6, 32), cases.rot(1e6, 96, (1.0, 4096, 4.0, 4.0))]


@pytest.mark.parametrize("rot", ROTATIONS)
def test_yarns_ramp(rot):
    s = rot.get("scaling")
    ramp = None if s is None else tuple(s[k] for k in ("factor", "original", "fast", "slow"))
    part = RotaryFrequencies(rot["dims"], rot["base"], "halves", ramp=ramp)
    freq, gain = plain.rotary_frequencies(rot)
    torch.testing.assert_close(torch.tensor(part.frequencies(), dtype=F64), torch.tensor(freq, dtype=F64), rtol=1e-12, atol=0)
    assert part.gain == pytest.approx(gain)
    unscaled = [rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)]
    if s:
        # between the frequency itself and the slowed one, and never back up along the pairs
        share = [(u / f - 1.0) for u, f in zip(unscaled, freq)]
        assert all(-1e-12 <= v <= s["factor"] - 1.0 + 1e-9 for v in share) and all(b >= a - 1e-9 for a, b in zip(share, share[1:]))
    else:
        assert freq == unscaled and gain == 1.0


def test_a_ramp_that_ends_where_it_begins_is_a_step():
    freq, _ = plain.rotary_frequencies(cases.rot(2.0, 16, (3.0, 10, 100.0, 50.0)))       # both ends before the first pair
    assert freq[0] == 1.0 and all(abs(f - 2.0 ** (-i / 8) / 3.0) < 1e-12 for i, f in enumerate(freq) if i > 0)


def test_ramps_the_parts_refuse():
    for bad in ((0.0, 10, 2.0, 1.0), (2.0, 10, 2.0), (2.0, 10, -1.0, 1.0)):
        with pytest.raises(ValueError, match="ramp"):
            RotaryFrequencies(8, 100.0, ramp=bad)
    with pytest.raises(ValueError, match="no other scaling"):
        RotaryFrequencies(8, 100.0, stretch=2.0, ramp=(2.0, 10, 2.0, 1.0))


def test_parts_refuse_what_does_not_fit():
    names = dict(q="q", k="k", v="v", g="g", o="o", b="b", a="a", A_log="A", dt_bias="t", norm="n")
    position = RotaryFrequencies(8, 100.0)
    with pytest.raises(ValueError, match="one decay"):
        Retention(16, 2, 8, 4, [0.5], norm_eps=1e-5, names=names)
    with pytest.raises(ValueError, match="rotated dimensions"):
        Retention(16, 1, 4, 4, [0.5], norm_eps=1e-5, names=names, position=position)
    with pytest.raises(ValueError, match="divide"):
        GatedDeltaRule(16, 3, 2, 8, 4, 3, norm_eps=1e-5, names=names)
    with pytest.raises(ValueError, match="one kind of output gate"):
        GroupedQueryAttention(16, 2, 1, 8, names=names, position=position, head_gate="g", element_gate="h")
    with pytest.raises(ValueError, match="go with the rotation from frequencies"):
        GroupedQueryAttention(16, 2, 1, 8, names=names, value_mix=("m", True))


def test_a_pair_through_norms_gives_its_branches_with_their_weights():
    model = build(cases.CASE_A)
    mixer = model.layers[0].mixer
    assert isinstance(mixer, ParallelMixers) and mixer.share == 0.5 and mixer.norm_eps == 1e-5
    assert len(model.layers[0].input.projections) == 2        # the pair's first products run as one


# ------------------------------------------------------------------ the plain functions against closed forms
def test_plain_retention_is_a_decayed_sum():
    q, k, v = (rows(12, 2 * n, i).view(12, 2, n) for i, n in ((1, 5), (2, 5), (3, 4)))
    decay = (0.9, 0.3)
    out, state = plain.retention_scan(q, k, v, decay)
    for t in (0, 7, 11):
        for h in range(2):
            expected = sum(decay[h] ** (t - j) * (q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1))
            torch.testing.assert_close(out[t, h], expected, rtol=1e-6, atol=1e-7)


def test_plain_delta_rule_replaces_what_a_key_held():
    """One unit key written again with beta one and no decay: the value read back is the last one written; an orthogonal key's
    value stays; beta zero writes nothing; the decay acts before the correction."""
    e1, e2 = torch.tensor([1.0, 0, 0], dtype=F64), torch.tensor([0, 1.0, 0], dtype=F64)
    k = torch.stack([e1, e2, e1, e1])[:, None]
    v = rows(4, 2, 9)[:, None]
    ones = torch.ones(4, 1, dtype=F64)
    beta = torch.tensor([[1.0], [1.0], [1.0], [0.0]], dtype=F64)
    out, state = plain.delta_scan(k, k, v, ones, beta)
    torch.testing.assert_close(out[:, 0], torch.stack([v[0, 0], v[1, 0], v[2, 0], v[2, 0]]))
    torch.testing.assert_close(state[0], torch.stack([v[2, 0], v[1, 0], torch.zeros(2, dtype=F64)]))
    half, _ = plain.delta_scan(k[:1].expand(2, 1, 3), k[:1].expand(2, 1, 3), v[:2], ones[:2] * 0.5, ones[:2] * 0.25)
    first = 0.25 * v[0, 0]
    torch.testing.assert_close(half[1, 0], 0.5 * first + 0.25 * (v[1, 0] - 0.5 * first))


def test_plain_convolution_reaches_back_over_a_cut():
    u, taps = rows(9, 4, 1), rows(4, 3, 2)
    whole = plain.short_conv(u, taps)
    torch.testing.assert_close(whole[0], u[0] * taps[:, 2])
    torch.testing.assert_close(whole[5], u[3] * taps[:, 0] + u[4] * taps[:, 1] + u[5] * taps[:, 2])
    torch.testing.assert_close(plain.short_conv(u[4:], taps, u[2:4]), whole[4:])


def test_plain_decay_and_unit_vectors():
    a, a_log, dt = rows(3, 2, 4, 3.0), torch.tensor([0.5, -2.0], dtype=F64), torch.tensor([0.1, -0.3], dtype=F64)
    expected = [[math.exp(-math.exp(float(a_log[h])) * math.log1p(math.exp(float(a[t, h] + dt[h])))) for h in range(2)] for t in range(3)]
    torch.testing.assert_close(plain.delta_decay(a, a_log, dt), torch.tensor(expected, dtype=F64))
    torch.testing.assert_close(plain.unit_vector(torch.tensor([3e3, 4e3], dtype=F64)), torch.tensor([0.6, 0.8], dtype=F64))
    assert plain.unit_vector(torch.zeros(3, dtype=F64)).abs().max() == 0


@pytest.mark.parametrize("interleaved", [False, True])
def test_plain_rotation_keeps_relative_angles_and_grows_by_the_gain(interleaved):
    rot = cases.rot(1000.0, 6, (4.0, 40, 4.0, 1.0))
    _, gain = plain.rotary_frequencies(rot)
    x = rows(1, 9, 3).expand(40, 9).contiguous()
    turned = plain.rotate(x, rot, interleaved)
    torch.testing.assert_close(turned[:, 6:], x[:, 6:])
    torch.testing.assert_close(turned[:, :6].norm(dim=-1), gain * x[:, :6].norm(dim=-1))
    dots = lambda i, j: turned[i, :6] @ turned[j, :6]
    torch.testing.assert_close(dots(3, 10), dots(20, 27))
    torch.testing.assert_close(plain.rotate(x[5:], rot, interleaved, first=5), turned[5:])


def test_plain_attention_sees_the_past_alone_and_caps_scores():
    q, k, v = rows(6, 8, 1).view(6, 2, 4), rows(6, 4, 2).view(6, 1, 4), rows(6, 3, 3).view(6, 1, 3)
    out = plain.causal_attention(q, k, v, 0.7)
    torch.testing.assert_close(out[0], v[0].expand(2, 3))
    changed = v.clone(); changed[5] += 1.0
    assert torch.equal(plain.causal_attention(q, k, changed, 0.7)[:5], out[:5])
    flat = plain.causal_attention(q, k, v, 0.7, cap=1e-9)              # a cap next to nothing: every key alike
    torch.testing.assert_close(flat[5], v[:, 0].mean(dim=0).expand(2, 3))
    torch.testing.assert_close(plain.causal_attention(q, k, v, 0.7, cap=1e6), out, rtol=1e-6, atol=1e-6)


def test_plain_values_are_mixed_with_the_first_layers():
    v, first = rows(3, 4, 1), rows(3, 4, 2)
    torch.testing.assert_close(plain.mixed_values(v, first, torch.tensor(0.25)), 0.75 * v + 0.25 * first)
    w = cases.make_weights(cases.CASE_A, 5)
    tokens = cases.random_tokens(cases.CASE_A, 6, 1)
    base = plain.forward(cases.CASE_A, w, tokens)
    for name, matters in (("l1.mix.vmix", False), ("l3.mix.vmix", True), ("l5.mix.vmix", True)):
        other = dict(w); other[name] = w[name] + 0.5
        assert torch.equal(plain.forward(cases.CASE_A, other, tokens), base) != matters


def test_plain_tanh_norm_and_activation():
    w = {"n": torch.tensor([2.0, 3.0]), "n.b": torch.tensor([0.5, -0.5]), "n.alpha": torch.tensor(0.25)}
    x = torch.tensor([[1.0, -400.0]], dtype=F64)
    torch.testing.assert_close(plain.tanh_norm(x, w, "n"), torch.tensor([[2 * math.tanh(0.25) + 0.5, -3.5]], dtype=F64))
    z = rows(1, 50, 3, 3.0)
    torch.testing.assert_close(plain.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))
