"""Bugidra on the GPU: every mechanism alone against its plain function, keys made to stand out far back and at page borders,
tokens that only a state can remember, then whole models under four ways of cutting the work, long decoding, slots and
pages used again, generation through the engine, the replay program and the command line."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from tests import bugidra_cases as cases
from tests import harness
from tests.plain import bugidra_plain as plain
from tests.test_larolorn_gpu import (CUTS, Ctx, DTYPES, IDS, SCHEDULES, close, judge, low_of, peak_live_pages, rows,
                                     through_the_step_function)

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
F64 = torch.float64
SUFFIX = ("", ".b")


def fill(part, seed, dtype, values=None):
    """Random parameters (``cases.draw_weights``) or the given ones; returns name -> CPU float32."""
    drawn = cases.draw_weights(part.all_named_params(), seed)
    drawn.update(values or {})
    for name, param in part.all_named_params().items():
        drawn[name] = drawn[name].to(torch.bfloat16).float()
        param.data = drawn[name].to(dtype).cuda()
    part.finalize(torch.device("cuda"), dtype)
    return drawn


def int32(*values):
    return torch.tensor(values, dtype=torch.int32, device="cuda")


# ------------------------------------------------------------------ mechanisms without a cache
@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_the_norm_without_statistics(dtype):
    from qwen_inference_lab_b200.parts import TanhNorm
    part = TanhNorm(70, name="n", suffixes=("", ".b", ".alpha"))
    w = fill(part, 4, dtype)
    assert w["n.alpha"].shape == ()
    x = rows(6, 70, 5, 3.0)
    x[0] *= 1e4
    expected = plain.tanh_norm(x.double(), w, "n").float()
    picked = int32(4, 0, 4)
    bar = dict(atol=1e-6, rtol=1e-5) if dtype == torch.float32 else dict(atol=4e-3, rtol=8e-3)
    for stream in (x.cuda(), x.to(dtype).cuda()):
        torch.testing.assert_close(part.forward(Ctx(dtype), stream).float().cpu(), expected, **bar)
    torch.testing.assert_close(part.forward(Ctx(dtype), x.cuda(), rows=picked).float().cpu(), expected[[4, 0, 4]], **bar)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("width", [70, 96, 1536, 4096, 4100])
def test_branches_are_normed_on_their_way_into_the_stream(width, dtype):
    """Plain branches and branches with a weight (one, two, three of them, also one that is next to zero, where eps decides)
    join a float32 stream; what is handed on is the norm without statistics of the new stream, a norm of another kind, or
    the stream rounded."""
    from qwen_inference_lab_b200.kernels import ops
    n, eps = 5, 1e-3
    stream = rows(n, width, 1, 2.0)
    raw = [rows(n, width, 2 + i, s) for i, s in enumerate((3.0, 0.01, 1.0))]
    weights = [1 + 0.2 * rows(1, width, 6 + i)[0] for i in range(3)]
    w, b = (1 + 0.1 * rows(1, width, 10)[0]).to(dtype), (0.2 * rows(1, width, 11)[0]).to(dtype)
    for normed in ((0,), (0, 1), (1,), (0, 1, 2), ()):
        branches, expected = [], stream.double()
        for i, rows_ in enumerate(raw):
            scale = (0.5, 0.5, -1.25)[i]
            value = rows_.double()
            if i in normed:
                value = plain.unit_rms(value, eps) * weights[i].double()
                branches.append((rows_.cuda(), scale, weights[i].cuda()))
            else:
                branches.append((rows_.cuda(), scale))
            expected = expected + scale * value
        for kind in ("tanh", "rms", None):
            x = stream.clone().cuda()
            out = torch.full((n, width), float("nan"), dtype=dtype, device="cuda")
            how = {} if kind is None else dict(next_weight=w.cuda(), next_eps=0.3, next_kind=kind)
            if kind == "tanh":
                how.update(next_bias=b.cuda(), next_alpha=0.4)
            ops.branch_join(x, branches, rows=out, branch_eps=eps, **how)
            torch.testing.assert_close(x.cpu(), expected.float(), atol=2e-5, rtol=2e-6)
            now = x.cpu().double()
            handed = now if kind is None else torch.tanh(0.4 * now) * w.double() + b.double() if kind == "tanh" \
                else plain.unit_rms(now, 0.3) * w.double()
            bar = dict(atol=1e-5, rtol=1e-5) if dtype == torch.float32 else dict(atol=1e-2, rtol=8e-3)
            torch.testing.assert_close(out.float().cpu(), handed.float(), **bar)
            assert torch.equal(ops.branch_join(stream.clone().cuda(), branches, branch_eps=eps), x)


ROTATIONS = [(8, 8, 32, "halves"), (64, 48, 100, "halves"), (20, 6, 16, "halves"), (16, 16, 64, "interleaved"), (24, 2, 50, "interleaved"),
             (128, 128, 300, "halves"), (32, 16, 40, "halves")]


@pytest.mark.parametrize("head,dims,original,layout", ROTATIONS)
@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_rotation_with_a_gain_and_heads_of_unit_size_behind_it(head, dims, original, layout, dtype):
    """Both forms of the kernel: positions up to a million, YaRN's frequencies and gain; every head is divided by the root mean
    square of the turned head, whose rotated part the gain has grown (one head is made so small that eps decides)."""
    from qwen_inference_lab_b200.kernels import ops
    from qwen_inference_lab_b200.parts import RotaryFrequencies
    rot = cases.rot(5000.0, dims, (6.0, original, 8.0, 1.0))
    rotation = RotaryFrequencies(dims, 5000.0, layout, ramp=(6.0, original, 8.0, 1.0))
    rotation.finalize(torch.device("cuda"), torch.float32)
    assert rotation.gain > 1.1
    heads, positions, eps = 3, [0, 1, 17, 4095, 70001, 999999], 1e-4
    x = rows(len(positions), heads * head, 5)
    x[:, head:2 * head] = (x[:, head:2 * head] * 0.01).to(torch.bfloat16).float()
    args = (rotation.freq, dims, rotation.layout, int32(*positions))
    f, gain = plain.rotary_frequencies(rot)
    f = torch.tensor(f, dtype=F64).float()
    pairs = (slice(0, dims, 2), slice(1, dims, 2)) if layout == "interleaved" else (slice(0, dims // 2), slice(dims // 2, dims))
    turned = x.double().view(len(positions), heads, head).clone()
    for i, p in enumerate(positions):
        a = (torch.tensor(float(p), dtype=torch.float32) * f).double()
        u, v = turned[i][:, pairs[0]].clone(), turned[i][:, pairs[1]].clone()
        turned[i][:, pairs[0]], turned[i][:, pairs[1]] = gain * (u * a.cos() - v * a.sin()), gain * (v * a.cos() + u * a.sin())
    bar = dict(atol=3e-6, rtol=1e-5) if dtype == torch.float32 else dict(atol=1e-3, rtol=8e-3)
    q = torch.empty(len(positions), heads * head, device="cuda", dtype=dtype)
    ops.qk_rotate_store(x.to(dtype).cuda(), (0, heads * head, heads * head), q, None, None, None, eps, *args,
                        torch.arange(len(positions), dtype=torch.int32, device="cuda"), None, heads, 0, head, head, 4,
                        unit_heads=True, gain=rotation.gain)
    torch.testing.assert_close(q.float().cpu().view_as(turned), plain.unit_rms(turned, eps).float(), **bar)
    # the recurrence's rows: float32 whatever the projection is, from a column of a wider row, later heads scaled
    wide = torch.cat([rows(len(positions), 5, 7), x], dim=1)
    out = ops.rotate_rows(wide.to(dtype).cuda(), 5, heads, head, *args, gain=rotation.gain, scaled_from=1, scale=0.25)
    assert out.dtype == torch.float32
    turned[:, 1:] *= 0.25
    torch.testing.assert_close(out.cpu().view_as(turned), turned.float(), atol=3e-6, rtol=1e-5)


@pytest.mark.parametrize("layout,whole,head,dims", [("halves", True, 32, 32), ("halves", False, 32, 16), ("interleaved", True, 64, 8),
                                                    ("interleaved", True, 20, 10), ("halves", True, 256, 64)])
@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_norms_with_weights_before_the_rotation_in_both_layouts(layout, whole, head, dims, dtype):
    """The norm over the whole projection and the one per head, each with its weights, where lanes hold a head and where they
    cannot."""
    from qwen_inference_lab_b200.kernels import ops
    from qwen_inference_lab_b200.parts import RotaryFrequencies
    rotation = RotaryFrequencies(dims, 300.0, layout)
    rotation.finalize(torch.device("cuda"), torch.float32)
    heads, n, eps = 3, 7, 1e-4
    x = rows(n, heads * head, 5)
    weight = 1 + 0.3 * rows(1, heads * head if whole else head, 6)[0]
    q = torch.empty(n, heads * head, device="cuda", dtype=dtype)
    k_weight = weight[:head].to(dtype).cuda()
    ops.qk_rotate_store(x.to(dtype).cuda(), (0, heads * head, heads * head), q, None, weight.to(dtype).cuda(), k_weight, eps,
                        rotation.freq, dims, rotation.layout, torch.arange(n, dtype=torch.int32, device="cuda"),
                        torch.arange(n, dtype=torch.int32, device="cuda"), None, heads, 0, head, head, 4, per_head=not whole)
    low = weight.to(dtype).double()
    normed = plain.unit_rms(x.double(), eps) * low if whole else plain.unit_rms(x.double().view(n, heads, head), eps) * low
    expected = plain.rotate(normed.view(n, heads, head), cases.rot(300.0, dims), layout == "interleaved")
    bar = dict(atol=3e-6, rtol=1e-5) if dtype == torch.float32 else dict(atol=1e-2, rtol=8e-3)
    torch.testing.assert_close(q.float().cpu().view_as(expected), expected.float(), **bar)


# ------------------------------------------------------------------ the recurrence's kernels alone, in float32
def state_inputs(T, heads, kv_heads, d, e, seed, delta, decay):
    """(q, k, v, g, beta) in float32; decay "mixed" (of every size), "none", "strong" (a state is forgotten within a few tokens)
    or "gone" (e^-1e4 and less now and then)."""
    q, k = rows(T, kv_heads * d, seed).view(T, kv_heads, d), rows(T, kv_heads * d, seed + 1).view(T, kv_heads, d)
    k = plain.unit_vector(k) if delta else k * d ** -0.5
    v, z = rows(T, heads * e, seed + 2).view(T, heads, e), rows(T, heads, seed + 3)
    log_g = {"mixed": -torch.exp(2.0 * z - 2.0), "none": torch.zeros(T, heads), "strong": -torch.exp(z + 1.5),
             "gone": torch.where(z > 1.0, torch.full_like(z, -1e4), -0.01 * z.abs())}[decay]
    beta = torch.sigmoid(2.0 * rows(T, heads, seed + 4))
    return q, k, v, log_g, beta


def run_state(q, k, v, log_g, beta, cuts, form, start=None):
    """(outputs [T, heads, e], final state) through ``state_scan`` or ``state_chunks`` over portions of the given sizes."""
    from qwen_inference_lab_b200.kernels import ops
    T, kv_heads, d = q.shape
    heads, e = v.shape[1:]
    slots = torch.full((3, heads, d, e), float("nan"), device="cuda")
    slots[1] = 0.0 if start is None else start.cuda()
    qk = torch.cat([q.reshape(T, -1), k.reshape(T, -1)], dim=1).contiguous().cuda()
    values = torch.cat([torch.zeros(T, 3), v.reshape(T, -1)], dim=1).contiguous().cuda()
    outputs, first = [], 0
    for size in cuts:
        part = slice(first, first + size)
        inputs = ops.StateRows(qk[part].contiguous(), (values[part].contiguous(), 3), heads, kv_heads, d, e,
                               log_decay=log_g[part].contiguous().cuda(),
                               beta=None if beta is None else beta[part].contiguous().cuda())
        raw = torch.full((size, heads * e), float("nan"), device="cuda")
        if form == "scan":
            ops.state_scan(inputs, None, None, 0.0, slots, int32(0), int32(size), int32(1), 1, raw=raw)
        else:
            starts = list(range(0, size, 64))
            ops.state_chunks(inputs, slots, int32(*starts), int32(*(min(64, size - s) for s in starts)), len(starts),
                             int32(1, 0, len(starts)), 1, raw)
        outputs.append(raw.cpu().view(size, heads, e))
        first += size
    assert slots[0].isnan().all() and slots[2].isnan().all()
    return torch.cat(outputs), slots[1].cpu()


STATE_SIZES = [(3, 3, 16, 24), (4, 2, 40, 7), (2, 1, 128, 130), (2, 2, 33, 64), (1, 1, 256, 17), (6, 2, 5, 3), (2, 2, 64, 64)]


@pytest.mark.parametrize("delta", [True, False], ids=["delta", "plain"])
@pytest.mark.parametrize("heads,kv_heads,d,e", STATE_SIZES)
def test_the_recurrence_by_token_and_in_chunks(heads, kv_heads, d, e, delta):
    """Both forms against the plain recurrence in float64: whole, cut, and cut in the middle of a chunk; the state at the end;
    a chunk of one token; decays of every size, none at all, and ones that forget everything."""
    T = 200
    for decay in ("mixed", "none", "strong", "gone"):
        q, k, v, log_g, beta = state_inputs(T, heads, kv_heads, d, e, 3, delta, decay)
        start = rows(heads * d, e, 9).view(heads, d, e)
        spread = lambda x: x.double().repeat_interleave(heads // kv_heads, dim=1)
        g = torch.exp(log_g.double())
        if delta:
            expected, last = plain.delta_scan(spread(q), spread(k), v.double(), g, beta.double(), start.double())
        else:
            S, out = start.double().clone(), []
            for t in range(T):
                S = g[t][:, None, None] * S + spread(k)[t][:, :, None] * v[t].double()[:, None, :]
                out.append((S * spread(q)[t][:, :, None]).sum(dim=1))
            expected, last = torch.stack(out), S
        scale = float(expected.abs().max())
        for form, cuts in (("scan", [T]), ("scan", [1, 2, 9, 60, 128]), ("chunks", [T]), ("chunks", [129, 71]), ("chunks", [64, 1, 135])):
            got, state = run_state(q, k, v, log_g, beta if delta else None, cuts, form, start)
            torch.testing.assert_close(got, expected.float(), atol=3e-6 * scale, rtol=2e-5, msg=lambda m: f"{decay} {form} {cuts}: {m}")
            torch.testing.assert_close(state, last.float(), atol=3e-6 * float(last.abs().max()), rtol=2e-5)


def test_the_walk_by_token_does_not_depend_on_the_cut():
    q, k, v, log_g, beta = state_inputs(100, 2, 2, 48, 20, 5, True, "mixed")
    whole = run_state(q, k, v, log_g, beta, [100], "scan")
    for cuts in ([1] * 100, [2, 98], [7, 8, 9, 76]):
        cut = run_state(q, k, v, log_g, beta, cuts, "scan")
        assert torch.equal(whole[0], cut[0]) and torch.equal(whole[1], cut[1])


def test_keys_that_all_point_one_way_do_not_grow():
    """The triangular system at its worst: the same unit key at every token, step sizes next to one, no decay.  What is read
    back is the running replacement of one value, of the values' size."""
    T, d, e = 256, 64, 32
    q, k, v, log_g, beta = state_inputs(T, 1, 1, d, e, 8, True, "none")
    k = k[:1].expand(T, 1, d).contiguous()
    q = k.clone()
    beta = torch.full((T, 1), 0.999)
    expected, _ = plain.delta_scan(q.double(), k.double(), v.double(), torch.exp(log_g.double()), beta.double())
    for form in ("scan", "chunks"):
        got, _ = run_state(q, k, v, log_g, beta, [T], form)
        torch.testing.assert_close(got, expected.float(), atol=1e-5, rtol=1e-5)


# ------------------------------------------------------------------ the mixers alone, through the step function
def left_part(hidden, m, eps=1e-5, prefix="m."):
    from qwen_inference_lab_b200.models.bugidra import _rotation
    from qwen_inference_lab_b200.parts import GroupedQueryAttention
    return GroupedQueryAttention(hidden, m["heads"], m["kv_heads"], m["dim"], names={k: prefix + k for k in ("q", "k", "v", "o")},
                                 scale=m["scale"], v_head_dim=m["vdim"], suffixes=SUFFIX, position=_rotation(m["rot"], "halves"),
                                 unit_qk_norm_eps=eps)


def right_part(hidden, m, eps=1e-5, prefix="m."):
    from qwen_inference_lab_b200.models.bugidra import _rotation
    from qwen_inference_lab_b200.parts import Retention
    return Retention(hidden, m["heads"], m["dim"], m["vdim"], m["decay"], norm_eps=eps, suffixes=SUFFIX,
                     position=_rotation(m["rot"], "halves"), names={k: prefix + k for k in ("q", "k", "v", "g", "o")})


def gated_part(hidden, m, eps=1e-5, prefix="m.", first=False):
    from qwen_inference_lab_b200.models.bugidra import _attention
    return _attention(hidden, m, prefix, eps, first)


def delta_part(hidden, m, eps=1e-5, prefix="m."):
    from qwen_inference_lab_b200.models.bugidra import _delta
    return _delta(hidden, m, prefix, eps, False)


LEFTS = [cases.left(4, 2, 32, 32, 0.3, cases.rot(300000.0, 16)),                              # the tensor-core kernels in bfloat16
         cases.left(6, 3, 32, 16, 0.3, cases.rot(1000.0, 32, (8.0, 50, 8.0, 1.0))),           # values smaller than keys
         cases.left(3, 3, 20, 12, 0.22, cases.rot(50.0, 4, (2.0, 16, 32.0, 1.0))),            # sizes only the float32 kernel takes
         cases.left(2, 1, 80, 80, 0.11, cases.rot(500.0, 80, (4.0, 100, 4.0, 0.5))),
         cases.left(6, 1, 48, 64, 0.25, cases.rot(10000.0, 2, (3.0, 7, 2.0, 1.0))),           # values larger than keys, one pair
         cases.left(8, 2, 128, 64, 0.08, cases.rot(500000.0, 64, (2.0, 512, 32.0, 1.0)))]


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("m", LEFTS, ids=[f"d{m['dim']}e{m['vdim']}" for m in LEFTS])
def test_attention_with_unit_heads_whole_cut_and_side_by_side(dtype, m):
    part = left_part(72, m)
    w = fill(part, 21, dtype)
    inputs = {"a": rows(75, 72, 22), "b": rows(41, 72, 23)}
    expected = {rid: plain.unit_attention_mixer(x.double(), w, "m.", m, 1e-5, low_of(dtype)) for rid, x in inputs.items()}
    for cuts in CUTS:
        got = through_the_step_function(part, 72, dtype, inputs, cuts, num_pages=48)
        for rid in inputs:
            close(got[rid], expected[rid], dtype)


GATED = [(dict(cases.left(4, 2, 32, 32, 0.3, cases.rot(3000.0, 16)), softcap=4.0), (4, 1, 16, 64)),
         (dict(cases.left(6, 1, 48, 64, 0.2, cases.rot(1000.0, 48))), (2, 2, 32, 32)),
         (dict(cases.left(3, 3, 20, 12, 0.4, cases.rot(50.0, 4)), softcap=2.0), (4, 2, 24, 18)),
         (dict(cases.left(2, 1, 14, 9, 0.3, cases.rot(77.0, 14)), softcap=30.0), (3, 1, 10, 9)),
         (dict(cases.left(8, 2, 128, 64, 0.1, cases.rot(500000.0, 64)), softcap=10.0), (8, 2, 32, 64))]


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("first,second", GATED, ids=[f"d{m['dim']}e{m['vdim']}" for m, _ in GATED])
def test_gated_attention_and_mixed_values(dtype, first, second):
    """Two such layers of the same rows, the second one's values mixed with the first one's of the same token, which a decoded
    token and every portion carry along; with the first alone, and with a share of none and of all."""
    from qwen_inference_lab_b200.parts.base import Mixer
    second = dict(cases.left(*second, 0.25, cases.rot(900.0, 6)), v_mix=True)
    first = dict(first, v_mix=True)

    class Two(Mixer):
        def __init__(self):
            self.parts = (gated_part(72, first, prefix="a.", first=True), gated_part(72, second, prefix="b."))

        def children(self):
            return list(self.parts)

        def cache_spec(self):
            return tuple(part.cache_spec() for part in self.parts)

    inputs = {"a": rows(75, 72, 22), "b": rows(41, 72, 23)}
    for share in (0.375, 0.0, 1.0):
        part = Two()
        w = fill(part, 31, dtype, {"b.vmix": torch.tensor(share)})
        expected = {}
        for rid, x in inputs.items():
            kept = []
            one = plain.gated_attention_mixer(x.double(), w, "a.", first, 1e-5, low_of(dtype), kept)
            expected[rid] = torch.cat([one, plain.gated_attention_mixer(x.double(), w, "b.", second, 1e-5, low_of(dtype), kept)], dim=1)
        body = lambda ctx, x, view: torch.cat([p.forward(ctx, x, v, out_float32=True) for p, v in zip(part.parts, view)], dim=1)
        for cuts in CUTS:
            got = harness.run_part(part, 72, dtype, body, inputs, cuts, page_size=4, num_pages=48)
            for rid in inputs:
                for half in (slice(0, 72), slice(72, 144)):
                    close(got[rid][:, half], expected[rid][:, half], dtype)


@pytest.mark.parametrize("dim,vdim", [(128, 128), (128, 64), (64, 64), (48, 80), (32, 16), (16, 128), (112, 96)])
def test_whole_tiles_take_the_tensor_memory_kernel(monkeypatch, dim, vdim):
    """Whole 128-token tiles of a prompt go to the tcgen05 kernel whatever the sizes of keys and values: one slab of 64 columns
    and two, whole and in part; leftovers and single tokens take the tiled kernels."""
    from qwen_inference_lab_b200.kernels import attention_tc
    calls = []
    original = attention_tc.prefill
    monkeypatch.setattr(attention_tc, "prefill", lambda *a, **k: (calls.append(k.get("softcap")), original(*a, **k))[1])
    gated = dict(cases.left(4, 2, dim, vdim, 2.2 * dim ** -0.5, cases.rot(10000.0, dim)), softcap=6.0)
    unit = cases.left(4, 1, dim, vdim, 2.2 * dim ** -0.5, cases.rot(10000.0, dim // 2, (4.0, 128, 16.0, 1.0)))
    inputs = {"a": rows(460, 64, 32), "b": rows(140, 64, 33)}
    for m, part, mixer in ((gated, gated_part(64, gated), plain.gated_attention_mixer), (unit, left_part(64, unit), plain.unit_attention_mixer)):
        w = fill(part, 31, torch.bfloat16)
        expected = {rid: mixer(x.double(), w, "m.", m, 1e-5, torch.bfloat16) for rid, x in inputs.items()}
        calls.clear()
        for cuts in ({"a": [460], "b": [140]}, {"a": [129, 1, 330], "b": [7, 133]}):
            got = through_the_step_function(part, 64, torch.bfloat16, inputs, cuts, page_size=16, num_pages=48)
            for rid in inputs:
                close(got[rid], expected[rid], torch.bfloat16)
        assert calls and all(call == m.get("softcap", 0.0) for call in calls)


SCAN_CUTS = ({"a": [300], "b": [41]}, {"a": [2, 129, 1, 1, 64, 3, 100], "b": [1] * 9 + [2] * 6 + [20]},
             {"a": [150, 150], "b": [17, 24]}, {"a": [1] * 40 + [260], "b": [41]})

RIGHTS = [cases.right(16, 24, cases.rot(100.0, 8), (0.9, 0.999)), cases.right(40, 8, cases.rot(1e4, 40, (2.0, 64, 8.0, 1.0)), (1.0, 0.5, 0.0)),
          cases.right(64, 64, cases.rot(1e6, 64), (0.995,)), cases.right(10, 6, cases.rot(10.0, 2), (0.1, 0.8, 0.97, 0.99, 1.0)),
          cases.right(128, 80, cases.rot(5000.0, 64), (0.98, 0.9995)), cases.right(96, 140, cases.rot(300.0, 96), (0.99,))]


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("m", RIGHTS, ids=[f"h{m['heads']}d{m['dim']}e{m['vdim']}" for m in RIGHTS])
def test_retention_whole_cut_and_side_by_side(dtype, m):
    """Short portions run token by token, portions of more than 128 tokens as chunks."""
    part = right_part(56, m)
    w = fill(part, 31, dtype)
    inputs = {"a": rows(300, 56, 32), "b": rows(41, 56, 33)}
    expected = {rid: plain.retention_mixer(x.double(), w, "m.", m, 1e-5, low_of(dtype)) for rid, x in inputs.items()}
    for cuts in SCAN_CUTS:
        got = through_the_step_function(part, 56, dtype, inputs, cuts, page_size=16, num_pages=24)
        for rid in inputs:
            close(got[rid], expected[rid], dtype, scale=float(expected[rid].abs().max()))


DELTAS = [cases.delta_sizes(2, 2, 16, 24, 4), cases.delta_sizes(6, 2, 40, 8, 3), cases.delta_sizes(1, 1, 64, 64, 1),
          cases.delta_sizes(5, 1, 10, 6, 2), cases.delta_sizes(4, 2, 128, 96, 4), cases.delta_sizes(2, 1, 130, 33, 16),
          cases.delta_sizes(1, 1, 270, 12, 3), cases.delta_sizes(2, 2, 96, 140, 5)]


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("m", DELTAS, ids=[f"h{m['heads']}d{m['dim']}e{m['vdim']}t{m['conv']}" for m in DELTAS])
def test_gated_delta_rule_whole_cut_and_side_by_side(dtype, m):
    """Portions shorter than the convolution reaches, single tokens, chunks, heads too wide for chunks; the q/k heads shared by
    several value heads.  A head whose decay is next to none and one that forgets at once."""
    part = delta_part(56, m)
    drawn = cases.draw_weights(part.all_named_params(), 41)
    drawn["m.A_log"][0] = -7.0
    drawn["m.A_log"][-1] = drawn["m.A_log"][-1] if m["heads"] == 1 else 3.0
    w = fill(part, 41, dtype, drawn)
    inputs = {"a": rows(300, 56, 42), "b": rows(41, 56, 43)}
    expected = {rid: plain.delta_mixer(x.double(), w, "m.", m, 1e-5, low_of(dtype)) for rid, x in inputs.items()}
    for cuts in SCAN_CUTS:
        got = through_the_step_function(part, 56, dtype, inputs, cuts, page_size=16, num_pages=24)
        for rid in inputs:
            close(got[rid], expected[rid], dtype, scale=float(expected[rid].abs().max()))


@pytest.mark.parametrize("layer", [0, 1, 2, 3])
@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_a_block_alone(layer, dtype):
    """A block whose sums and norms are deferred, over portions and single tokens: the plain layer; in float32 the same bits
    with the pair's first products joined and apart."""
    from qwen_inference_lab_b200.config import registry
    from qwen_inference_lab_b200.parts.block import settle_stream
    entry = registry.lookup(cases.CASE_A)
    block = entry.build(entry.config_class.from_dict(cases.CASE_A)).layers[layer]
    w = fill(block, 51, dtype)
    spec, p = cases.CASE_A["layers"][layer], f"l{layer}."
    if layer == 3:                                     # on its own there is no first layer's values to mix in
        block.mixer.mixes_values, spec = False, dict(spec, mixer=dict(spec["mixer"], v_mix=False))

    def body(ctx, x, view):
        out = block.forward(ctx, x.float(), view)
        settle_stream(ctx)
        return out

    inputs = {"a": rows(75, 96, 52), "b": rows(41, 96, 53)}
    joint = block.input._w
    assert (joint is None) == (layer != 0)
    low = low_of(dtype)
    for cuts in CUTS:
        got = harness.run_part(block, 96, dtype, body, inputs, cuts, page_size=4, num_pages=48)
        block.input._w = None
        apart = harness.run_part(block, 96, dtype, body, inputs, cuts, page_size=4, num_pages=48)
        block.input._w = joint
        for rid, x in inputs.items():
            assert dtype == torch.bfloat16 or torch.equal(got[rid], apart[rid])
            h = plain._round(plain.tanh_norm(x.double(), w, p + "norm1"), low)
            more = ([],) if spec["type"] == "attention" else ()
            expected = x.double() + plain.MIXERS[spec["type"]](h, w, p + "mix.", spec["mixer"], 1e-5, low, *more)
            if spec["mlp"]:
                expected = expected + plain.feed_forward(plain._round(plain.tanh_norm(expected, w, p + "norm2"), low), w, p + "mlp.", low)
            close(got[rid], expected, dtype, scale=float(expected.abs().max()))


# ------------------------------------------------------------------ one key made to stand out
FAR = [(127, 0), (128, 63), (130, 64), (19, 16), (64, 15), (200, 127), (200, 128), (650, 1), (1000, 0), (1000, 999)]


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("single", [False, True], ids=["prompt", "decoded"])
@pytest.mark.parametrize("query,far", FAR)
def test_a_key_far_back_that_stands_out(dtype, single, query, far):
    """Heads are of unit size, so a key stands out by its direction only: the query's input is solved for so that every
    head's query, turned at its position, points along the far token's turned key, and the far token's input is drawn
    again until it leads every other key by 30 in every head.  The output is then that token's value.  A wrong angle,
    frequency, gain or position loses the key, a wrong page or slot its value."""
    from qwen_inference_lab_b200.models.bugidra import _rotation
    hidden = 160
    m = cases.left(4, 2, 32, 16, 3.0, cases.rot(10000.0, 24, (4.0, 64, 8.0, 1.0)))
    H, G, d, e, r = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["rot"]["dims"]
    part = left_part(hidden, m)
    w = fill(part, 61, dtype)
    W = {k: v.double() for k, v in w.items()}
    x = rows(query + 1, hidden, 62 + query, 0.5)
    freq, gain = plain.rotary_frequencies(m["rot"])
    freq = torch.tensor(freq, dtype=F64)
    for attempt in range(80):
        x[far] = rows(1, hidden, 1000 + attempt, 0.5)[0]
        k_far = (x[far].double() @ W["m.k"].t()).view(G, d)
        wanted = k_far.clone()                         # such that turned at the query's position it is k_far turned at its own
        pairs = torch.complex(k_far[:, :r // 2], k_far[:, r // 2:r]) * torch.exp(1j * (far - query) * freq)
        wanted[:, :r] = torch.cat([pairs.real, pairs.imag], dim=1)
        target = torch.stack([wanted[a // (H // G)] for a in range(H)]).flatten()
        x[query] = (torch.linalg.pinv(W["m.q"]) @ target).to(torch.bfloat16).float()
        q = plain.unit_rms(plain.rotate((x.double() @ W["m.q"].t()).view(-1, H, d), m["rot"]), 1e-5)[query]
        k = plain.unit_rms(plain.rotate((x.double() @ W["m.k"].t()).view(-1, G, d), m["rot"]), 1e-5)
        scores = torch.stack([k[:, a // (H // G)] @ q[a] for a in range(H)]) * m["scale"]      # [H, T]
        others = torch.cat([scores[:, :far], scores[:, far + 1:]], dim=1)
        if float((scores[:, far] - others.max(dim=1).values).min()) > 30.0:
            break
    else:
        raise AssertionError("no input found whose key stands out")
    v_far = (x[far].double() @ W["m.v"].t()).view(G, e)
    alone = torch.stack([v_far[a // (H // G)] for a in range(H)]).flatten() @ W["m.o"].t()
    tail = 1 if single else min(5, query + 1)
    head = query + 1 - tail
    cuts = ([head - 2, 2] if head > 3 else [head] if head else []) + [tail]
    got = through_the_step_function(part, hidden, dtype, {"a": x}, {"a": cuts}, page_size=8, num_pages=(query + 1) // 8 + 3)["a"]
    close(got[-1], alone, dtype)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("single", [False, True], ids=["prompt", "decoded"])
@pytest.mark.parametrize("query,far", [(64, 15), (200, 128), (650, 1), (1000, 0)])
def test_a_capped_key_far_back_whose_value_is_mixed(dtype, single, query, far):
    """The same through the gated attention: the far key scores 60 before the cap of 40 and 36 behind it, every other key less
    than half as much and 25, and the value that comes back is the mixture of the far token's own and the first layer's."""
    hidden = 200
    m = dict(cases.left(2, 1, 32, 16, 1.0, cases.rot(5000.0, 32)), softcap=40.0, v_mix=True)
    H, d, e = m["heads"], m["dim"], m["vdim"]
    part = gated_part(hidden, m)
    w = fill(part, 61, dtype)
    W = {k: v.double() for k, v in w.items()}
    x = rows(query + 1, hidden, 62 + query, 0.5)
    first_values = rows(query + 1, e, 63)
    freq = torch.tensor(plain.rotary_frequencies(m["rot"])[0], dtype=F64)
    normed = lambda name: plain.unit_rms(x.double() @ W["m." + name].t(), 1e-5) * W[f"m.{name}.norm"]
    for attempt in range(80):
        x[far] = rows(1, hidden, 1000 + attempt, 0.5)[0]
        k_far = normed("k")[far]
        pairs = torch.complex(k_far[0::2], k_far[1::2]) * torch.exp(1j * (far - query) * freq)
        wanted = torch.view_as_real(pairs).flatten().repeat(H) / W["m.q.norm"]
        x[query] = (torch.linalg.pinv(W["m.q"]) @ wanted).to(torch.bfloat16).float()
        q = plain.rotate(normed("q").view(-1, H, d), m["rot"], True)[query]
        k = plain.rotate(normed("k").view(-1, 1, d), m["rot"], True)[:, 0]
        scores = k @ q.t()                                                                     # [T, H]
        scale = 60.0 / float(scores[far].min())
        others = torch.cat([scores[:far], scores[far + 1:]]) * scale
        if float(others.max()) < 30.0 and float(scores[far].max() * scale) < 90.0:
            break
    else:
        raise AssertionError("no input found whose key stands out")
    m["scale"] = part.scale = scale
    exact = plain.gated_attention_mixer(x.double(), w, "m.", m, 1e-5, None, [first_values.double()])
    share = float(w["m.vmix"])
    value = (1.0 - share) * (x[far].double() @ W["m.v"].t()) + share * first_values[far].double()
    gate = torch.sigmoid(x[query].double() @ W["m.g"].t())
    alone = (value.repeat(H) * gate) @ W["m.o"].t()
    assert float((exact[query] - alone).abs().max()) < 0.05 * float(alone.abs().max())
    tail = 1 if single else min(5, query + 1)
    head = query + 1 - tail
    cuts = ([head - 2, 2] if head > 3 else [head] if head else []) + [tail]
    kept = first_values.to(dtype).cuda()
    seen = {"at": 0}

    def body(ctx, inputs, view):
        n = inputs.shape[0]
        ctx.shared["first_values"] = (kept[seen["at"]:seen["at"] + n].contiguous(), 0)
        seen["at"] += n
        return part.forward(ctx, inputs, view, out_float32=True)

    got = harness.run_part(part, hidden, dtype, body, {"a": x}, {"a": cuts}, page_size=8, num_pages=(query + 1) // 8 + 3)["a"]
    close(got[-1], exact[query], dtype)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("single", [False, True], ids=["prompt", "decoded"])
@pytest.mark.parametrize("kind", ["retention", "delta"])
def test_the_state_remembers_a_token_from_far_back(dtype, single, kind):
    """Token 2 alone writes much: every other token is faint (and, with the delta rule, its step size next to nothing), and
    nothing is forgotten to speak of.  The query 600 positions later is solved for: its q points along what token 2 wrote.
    Without token 2 the query's row is another one, so a lost state shows."""
    hidden, query, heads, d, e = 120, 602, 2, 16, 8
    x = rows(query + 1, hidden, 72, 0.02)
    pull = lambda system, target: (torch.linalg.pinv(torch.cat(system)) @ torch.cat(target)).to(torch.bfloat16).float()
    key = rows(1, heads * d, 74)[0]
    if kind == "retention":
        m = cases.right(d, e, cases.rot(1e7, 2), (0.9990234375, 1.0))
        part, mixer = right_part(hidden, m), plain.retention_mixer
        w = cases.draw_weights(part.all_named_params(), 71)
        x[2] = pull([w["m.k"], w["m.v"]], [3.0 * key, rows(1, heads * e, 73, 8.0)[0]])
        x[query] = pull([w["m.q"], w["m.g"], w["m.k"]], [key, torch.full((heads * e,), 3.0), torch.zeros(heads * d)])
    else:
        m = cases.delta_sizes(heads, heads, d, e, 3)
        part, mixer = delta_part(hidden, m), plain.delta_mixer
        w = cases.draw_weights(part.all_named_params(), 71)
        w["m.A_log"], w["m.dt_bias"] = torch.full((heads,), -7.0), torch.full((heads,), -3.0)
        for name in ("q", "k", "v"):
            w[f"m.{name}.conv"] = torch.zeros_like(w[f"m.{name}.conv"])
            w[f"m.{name}.conv"][:, 2] = 1.0
        shut = pull([w["m.b"]], [torch.full((heads,), -12.0)])
        x += shut                                            # every token's step size is next to nothing
        x[2] = pull([w["m.k"], w["m.v"], w["m.b"]], [3.0 * key, rows(1, heads * e, 73, 8.0)[0], torch.full((heads,), 4.0)])
        x[query] = pull([w["m.q"], w["m.g"], w["m.b"]], [3.0 * key, torch.full((heads * e,), 3.0), torch.full((heads,), -12.0)])
        x = x.to(torch.bfloat16).float()
    w = fill(part, 71, dtype, w)
    expected = mixer(x.double(), w, "m.", m, 1e-5, low_of(dtype))
    lost = x.clone(); lost[2] = x[3]
    without = mixer(lost.double(), w, "m.", m, 1e-5)
    assert (expected[query].double() - without[query]).abs().max() > 0.3 * expected[query].abs().max()
    tail = 1 if single else 5
    cuts = [130, 2, 200, 1, query + 1 - 333 - tail, tail]
    got = through_the_step_function(part, hidden, dtype, {"a": x}, {"a": cuts}, page_size=16, num_pages=40)["a"]
    close(got[-1:], expected[-1:], dtype, scale=float(expected.abs().max()))


# ------------------------------------------------------------------ whole models
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    result = {}
    for name, case in cases.CASES.items():
        folder = tmp_path_factory.mktemp(f"bugidra{name}")
        weights = cases.write_folder(case["config"], case["seed"], folder)
        requests = {f"r{i}": cases.random_tokens(case["config"], n, 60 + i) for i, n in enumerate(case["lengths"])}
        result[name] = (folder, weights, requests)
    return result


@pytest.fixture(scope="module")
def truth(folders):
    """The plain rows of every case, in float64 and with bfloat16 roundings."""
    return {name: (cases.plain_rows(requests, weights, cases.CASES[name]["config"]),
                   cases.plain_rows(requests, weights, cases.CASES[name]["config"], torch.bfloat16))
            for name, (folder, weights, requests) in folders.items()}


def replay(folders, case, schedule_name, dtype):
    folder, weights, requests = folders[case]
    page_size = cases.CASES[case]["page_size"]
    schedule = SCHEDULES[schedule_name](requests)
    from qwen_inference_lab_b200.config import registry
    entry = registry.lookup(cases.CASES[case]["config"])
    shell = entry.build(entry.config_class.from_dict(cases.CASES[case]["config"]))
    num_pages = peak_live_pages(schedule, shell, page_size) + 1
    _, cache, runner = harness.build_engine_parts(folder, dtype, num_pages=num_pages, page_size=page_size)
    for _, _, tensor in cache.state_groups:
        tensor.fill_(float("nan"))             # a slot that is not zeroed at admission shows
    ledger = harness.PageLedger(cache)
    actual = harness.run_schedule(runner, cache, schedule, ledger)
    assert cache.free_pages() == num_pages and not cache.owners()
    assert ledger.handovers > 0, "no page was used again by another request: the pool is too large"
    return actual


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("schedule", list(SCHEDULES))
@pytest.mark.parametrize("case", list(cases.CASES))
def test_replay_matches_plain(folders, truth, case, schedule, dtype):
    actual = replay(folders, case, schedule, dtype)
    expected, low = truth[case]
    judge(actual, expected, low, dtype, f"bugidra {case} {schedule} {dtype}")


@pytest.mark.parametrize("case", list(cases.CASES))
def test_float32_rows_agree_under_every_schedule(folders, case):
    """Portions of up to 128 tokens and single tokens walk the states token by token, attention walks key tiles aligned
    to positions and float32 products sum in ascending order: such schedules give the same bits.  A longer portion's
    states come in chunks, which round differently in the last bits."""
    runs = {name: replay(folders, case, name, torch.float32) for name in SCHEDULES}
    longest = max(cases.CASES[case]["lengths"])
    for name, got in runs.items():
        if longest <= 128:
            different = [key for key in sorted(got) if not torch.equal(got[key], runs["chunks"][key])]
        else:
            different = [key for key in sorted(got) if not torch.allclose(got[key], runs["chunks"][key], atol=5e-5, rtol=1e-5)]
        assert not different, \
            f"bugidra {case}: {len(different)} rows of schedule {name} differ from the run in portions, first {different[0]}"
    for name in ("tail_decode", "mixed"):
        short = [key for key in sorted(runs[name]) if len(folders[case][2][key[0]]) <= 128]
        assert all(torch.equal(runs[name][key], runs["chunks"][key]) for key in short)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("case", ["A", "C"])
def test_long_decoding_and_the_first_tokens(folders, dtype, case):
    """Three tokens as a prompt, then 300 single tokens (recorded graphs), every position judged."""
    folder, weights, _ = folders[case]
    config, page_size = cases.CASES[case]["config"], cases.CASES[case]["page_size"]
    tokens = cases.random_tokens(config, 303, 99)
    schedule = [([("r", tokens[:3], [0, 1, 2])], [])]
    schedule += [([("r", [tokens[i]], [0])], ["r"] if i == 302 else []) for i in range(3, 303)]
    _, cache, runner = harness.build_engine_parts(folder, dtype, num_pages=303 // page_size + 1, page_size=page_size)
    actual = harness.run_schedule(runner, cache, schedule)
    assert runner._graphs, "single-token steps should have been recorded"
    expected = cases.plain_rows({"r": tokens}, weights, config)
    low = cases.plain_rows({"r": tokens}, weights, config, torch.bfloat16) if dtype == torch.bfloat16 else None
    judge(actual, expected, low, dtype, f"bugidra {case} long decoding {dtype}")


def test_a_state_slot_and_pages_that_another_request_used_before(folders):
    """"x" runs and ends; "y" takes its slots and its pages: its logits are those of "y" in a fresh cache, bit for bit."""
    folder, weights, _ = folders["A"]
    config = cases.CASE_A
    x, y = cases.random_tokens(config, 37, 1), cases.random_tokens(config, 29, 2)
    def run(first):
        _, cache, runner = harness.build_engine_parts(folder, torch.float32, num_pages=12, page_size=4, max_requests=1)
        schedule = []
        if first:
            schedule += [([("x", x[:30], [])], [])] + [([("x", [t], [0])], []) for t in x[30:]]
            schedule[-1] = (schedule[-1][0], ["x"])
        schedule += [([("y", y[:11], list(range(11)))], []), ([("y", y[11:13], [0, 1])], [])]
        schedule += [([("y", [t], [0])], []) for t in y[13:]]
        schedule[-1] = (schedule[-1][0], ["y"])
        got = harness.run_schedule(runner, cache, schedule)
        return torch.stack([got[("y", p)] for p in range(len(y))])
    assert torch.equal(run(first=True), run(first=False))


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_greedy_generation_through_the_engine(folders, dtype):
    """Prompts of unequal length through ``Engine.generate`` (scheduler, chunked prompts, sampler): every token is
    the plain implementation's best one, or in bfloat16 inside what bfloat16 costs the plain implementation."""
    from qwen_inference_lab_b200 import Engine, load_model
    folder, weights, _ = folders["A"]
    config = cases.CASE_A
    model = load_model(folder, device="cuda", dtype=dtype)
    engine = Engine(model, num_pages=48, page_size=4, token_budget=24, prefill_chunk=10, max_active=3)
    prompts = [cases.random_tokens(config, n, 40 + n) for n in (2, 31, 17, 5)]
    results = engine.generate(prompts, max_new_tokens=12, ignore_eos=True)
    assert engine.idle and engine.cache.free_pages() == 48
    for prompt, row in zip(prompts, results):
        assert len(row["token_ids"]) == 12
        sequence = list(prompt)
        for token in row["token_ids"]:
            logits = plain.forward(config, weights, sequence, torch.float32)[-1]
            best = int(logits.argmax())
            if token != best:
                assert dtype == torch.bfloat16, f"token {token} instead of {best} after {len(sequence)} tokens"
                noise = (plain.forward(config, weights, sequence, torch.float32, torch.bfloat16)[-1] - logits).abs().max().item()
                assert float(logits[best] - logits[token]) < 4 * noise
            sequence.append(token)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_a_model_that_keeps_no_pages(tmp_path, dtype):
    """Delta layers alone, one of them with a convolution of one tap: state slots and no key or value anywhere."""
    config = cases.config(61, 48, 1e-5, 1.5, cases.delta(2, 1, 12, 16, 4, ff=40), cases.delta(3, 3, 16, 8, 1))
    weights = cases.write_folder(config, 9, tmp_path)
    requests = {"a": cases.random_tokens(config, 150, 1), "b": cases.random_tokens(config, 20, 2)}
    _, cache, runner = harness.build_engine_parts(tmp_path, dtype, num_pages=4, page_size=64)
    for schedule in (harness.whole_schedule(requests), harness.mixed_schedule(requests)):
        got = harness.run_schedule(runner, cache, schedule)
        judge(got, cases.plain_rows(requests, weights, config), cases.plain_rows(requests, weights, config, torch.bfloat16), dtype,
              f"bugidra without pages {dtype}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_replay_program_runs_a_mixed_schedule(folders, truth, tmp_path, dtype):
    folder, weights, requests = folders["A"]
    schedule = harness.mixed_schedule(requests)
    peak = harness.peak_pages(schedule, 64, round_to=64) * 64
    process = subprocess.Popen([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype,
                                "--out", str(tmp_path / "out"), "--max-tokens", str(peak)],
                               stdin=subprocess.PIPE, stdout=subprocess.PIPE, text=True)
    got, position = {}, {}
    for number, (entries, ended) in enumerate(schedule):
        step = dict(step=number, entries=[dict(id=rid, tokens=tokens, want=want) for rid, tokens, want in entries], end=ended)
        process.stdin.write(json.dumps(step) + "\n")
        process.stdin.flush()
        assert process.stdout.readline().strip() == f"done {number}"
        wanted = [(rid, position.get(rid, 0) + w) for rid, tokens, want in entries for w in want]
        data = np.fromfile(tmp_path / "out" / f"{number}.f32", dtype="<f4").reshape(len(wanted), cases.CASE_A["vocab"])
        for key, row in zip(wanted, data):
            got[key] = torch.from_numpy(row.copy())
        for rid, tokens, _ in entries:
            position[rid] = position.get(rid, 0) + len(tokens)
    process.stdin.close()
    assert process.wait(timeout=60) == 0
    expected, low = truth["A"]
    judge(got, expected, low, torch.float32 if dtype == "float32" else torch.bfloat16, f"bugidra replay program {dtype}")


def test_command_line_generates_with_written_and_with_random_weights(folders, tmp_path):
    folder, weights, _ = folders["C"]
    prompt = cases.random_tokens(cases.CASE_C, 9, 77)          # ids that every case's vocabulary holds
    run = lambda model, *extra: subprocess.run(
        [sys.executable, "-m", "qwen_inference_lab_b200", "--model", str(model), "--token-ids", json.dumps(prompt),
         "--dtype", "float32", "--max-new-tokens", "4", "--pages", "24", "--page-size", "4", "--chunk-size", "5",
         "--ignore-eos", *extra], capture_output=True, text=True, cwd=str(ROOT))
    done = run(folder)
    assert done.returncode == 0, done.stderr
    tokens = json.loads(done.stdout)["token_ids"]
    sequence = list(prompt)
    for token in tokens:
        assert token == int(plain.forward(cases.CASE_C, weights, sequence, torch.float32)[-1].argmax())
        sequence.append(token)
    bare = tmp_path / "bare"
    bare.mkdir()
    (bare / "config.json").write_text(json.dumps(cases.CASE_A))
    done = run(bare, "--random-weights", "3")
    assert done.returncode == 0, done.stderr
    assert len(json.loads(done.stdout)["token_ids"]) == 4 and (bare / "model.safetensors").is_file()
