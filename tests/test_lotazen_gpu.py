"""Lotazen on the GPU: every mechanism alone against its plain function, keys made to stand out at window edges and page
borders, tokens that only a state can remember, then whole models under four ways of cutting the work, long decoding,
slots and pages used again, generation through the engine, the replay program and the command line."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from tests import harness
from tests import lotazen_cases as cases
from tests.plain import lotazen_plain as plain
from tests.test_larolorn_gpu import (CUTS, Ctx, DTYPES, IDS, SCHEDULES, close, low_of, peak_live_pages, rows,
                                     through_the_step_function)
from tests.test_larolorn_gpu import judge as judge_rows

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


# ------------------------------------------------------------------ mechanisms without a cache
@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("width", [70, 96, 1536, 4096, 4100])
def test_branches_join_the_stream_and_the_next_norm_rides_along(width, dtype):
    """x += sum of scale * branch + routed rows on a float32 stream; the rows handed on are the norm of the new stream
    (of either kind), or the new stream rounded."""
    from qwen_inference_lab_b200.kernels import ops
    n, top = 5, 3
    stream = rows(n, width, 1, 4.0)
    branches = [(rows(n, width, 2 + i), scale) for i, scale in enumerate((0.7, -1.3, 1.0))]
    routed = rows(n * top, width, 9).view(n, top, width)
    weight = (1 + 0.1 * rows(1, width, 8)[0]).to(dtype)
    for many in range(4):
        for experts in (None, routed):
            expected = stream.double() + sum(scale * b.double() for b, scale in branches[:many])
            if experts is not None:
                expected = expected + routed.double().sum(dim=1)
            for kind in ("rms", "layer", None):
                x = stream.clone().cuda()
                out = torch.full((n, width), float("nan"), dtype=dtype, device="cuda")
                ops.branch_join(x, [(b.cuda(), scale) for b, scale in branches[:many]],
                                routed=None if experts is None else experts.cuda(), rows=out,
                                **({} if kind is None else dict(next_weight=weight.cuda(), next_eps=0.3, next_kind=kind)))
                torch.testing.assert_close(x.cpu(), expected.float(), atol=1e-5, rtol=1e-6)
                centred = x.cpu().double()
                if kind == "layer":
                    centred = centred - centred.mean(dim=-1, keepdim=True)
                normed = centred if kind is None else plain.unit_rms(centred, 0.3) * weight.double()
                bar = dict(atol=1e-5, rtol=1e-5) if dtype == torch.float32 else dict(atol=1e-2, rtol=8e-3)
                torch.testing.assert_close(out.float().cpu(), normed.float(), **bar)
                alone = ops.branch_join(stream.clone().cuda(), [(b.cuda(), scale) for b, scale in branches[:many]],
                                        routed=None if experts is None else experts.cuda())
                assert torch.equal(alone, x)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_the_norm_with_one_number(dtype):
    from qwen_inference_lab_b200.parts import ScalarRMSNorm
    part = ScalarRMSNorm(70, 0.2, name="n", suffix="")
    w = fill(part, 4, dtype)
    assert w["n"].shape == ()
    x = rows(6, 70, 5, 3.0)
    expected = plain.scalar_norm(x.double(), w["n"], 0.2).float()
    picked = torch.tensor([4, 0, 4], dtype=torch.int32, device="cuda")
    bar = dict(atol=1e-6, rtol=1e-5) if dtype == torch.float32 else dict(atol=1e-2, rtol=8e-3)
    torch.testing.assert_close(part.forward(Ctx(dtype), x.cuda()).float().cpu(), expected, **bar)
    torch.testing.assert_close(part.forward(Ctx(dtype), x.cuda(), rows=picked).float().cpu(), expected[[4, 0, 4]], **bar)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_a_learned_vector_per_position_joins_the_embedding(dtype):
    from qwen_inference_lab_b200.parts import TokenEmbedding
    part = TokenEmbedding(11, 70, name="e", suffix="", scale=1.5, positions=("p", 40))
    w = fill(part, 6, dtype)
    ids, positions = [3, 10, 0, 3], [0, 39, 17, 1]
    ctx = Ctx(dtype)
    ctx.positions = torch.tensor(positions, dtype=torch.int32, device="cuda")
    out = part.forward(ctx, torch.tensor(ids, dtype=torch.int32, device="cuda"))
    assert out.dtype == torch.float32
    torch.testing.assert_close(out.cpu(), 1.5 * w["e"][ids] + w["p"][positions], atol=1e-6, rtol=1e-6)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("n,width,mlp", [(1, 96, cases.moe(5, 2, 24, 1.2, (40, 0.6))), (9, 70, cases.moe(7, 7, 11, 0.5)),
                                         (300, 64, cases.moe(3, 1, 48, 2.0, (16, 0.3))), (70, 64, cases.moe(40, 6, 16, 1.0))])
def test_experts_whose_input_is_weighed(dtype, n, width, mlp):
    """Inputs large enough that the gate passes its upper bound and the other branch both of its bounds; scores from
    close to nothing to close to one.  A token's result is the same bits alone and in the batch in float32."""
    from qwen_inference_lab_b200.kernels import ops
    from qwen_inference_lab_b200.models.lotazen import _feed_forward
    part = _feed_forward(width, mlp, "f.")
    w = fill(part, 3, dtype)
    x = rows(n, width, 4, 2.0)
    margins = []
    plain.routed_experts(x.double(), w, "f.", mlp, margins=margins)
    if margins:                     # leave out tokens whose choice of experts bfloat16 could flip
        x = x[(margins[0] > 0.05).nonzero().flatten()].contiguous()
        assert len(x) > n // 2
    chosen, weights = ops.moe_route(x.to(dtype).cuda(), part._router, None, mlp["router"]["top"], sigmoid=True)
    order, scores = plain.route(x.double(), w["f.router"], mlp["router"]["top"])
    assert torch.equal(chosen.cpu().long(), order)
    torch.testing.assert_close(weights.cpu(), scores.float(), atol=1e-6, rtol=1e-5)
    expected = plain.routed_experts(x.double(), w, "f.", mlp, low_of(dtype))

    def run(inputs):
        shared, routed = part.branches(Ctx(dtype), inputs)
        assert len(shared) == (1 if mlp["shared"] else 0) and routed.dtype == torch.float32
        out = torch.zeros(inputs.shape, device="cuda")
        return ops.branch_join(out, shared, routed=routed)

    out = run(x.to(dtype).cuda())
    close(out, expected, dtype, scale=float(expected.abs().max()))
    summed = part.forward(Ctx(dtype), x.to(dtype).cuda(), out_float32=True)          # the same through the combine kernel
    torch.testing.assert_close(summed, out, atol=1e-5 * float(expected.abs().max()), rtol=1e-5)
    if dtype == torch.float32:
        for t in (0, len(x) - 1):
            assert torch.equal(run(x[t:t + 1].cuda())[0], out[t])


def test_sigmoid_scores_choose_by_the_logits_even_where_they_round_to_one():
    from qwen_inference_lab_b200.kernels import ops
    router = torch.eye(6, 8)
    x = torch.tensor([[40.0, 60.0, 50.0, -90.0, -80.0, -100.0, 0, 0], [-90.0, -80.0, -100.0, -200.0, -300.0, -85.0, 0, 0]])
    for n in (2, 128):                                                   # both forms of the kernel
        chosen, weights = ops.moe_route(x.repeat(n // 2, 1).cuda(), router.cuda(), None, 3, sigmoid=True)
        assert chosen[0].tolist() == [1, 2, 0] and chosen[1].tolist() == [1, 5, 0] and chosen[n - 1].tolist() == [1, 5, 0]
        assert weights[0].tolist() == [1.0, 1.0, 1.0]
        torch.testing.assert_close(weights[1].cpu().double(), torch.sigmoid(torch.tensor([-80.0, -85.0, -90.0], dtype=F64)), rtol=1e-5, atol=0)


@pytest.mark.parametrize("dims,head,factor", [(16, 16, 1.0), (4, 20, 8.0), (2, 6, 0.5), (80, 80, 3.0)])
def test_rotation_by_neighbours_with_stretched_frequencies_and_heads_of_unit_size(dims, head, factor):
    """The kernel alone in float32: positions up to a million, angles as the design computes them, every head divided by
    its own root mean square (one head is made so small that eps decides)."""
    from qwen_inference_lab_b200.kernels import ops
    from qwen_inference_lab_b200.parts import RotaryFrequencies
    rotation = RotaryFrequencies(dims, 5000.0, "interleaved", stretch=factor)
    rotation.finalize(torch.device("cuda"), torch.float32)
    heads, positions, eps = 3, [0, 1, 17, 4095, 70001, 999999], 1e-4
    x = rows(len(positions), heads * head, 5)
    x[:, head:2 * head] *= 0.01
    q = torch.empty(len(positions), heads * head, device="cuda")
    ops.qk_rotate_store(x.cuda(), (0, heads * head, heads * head), q, None, None, None, eps, rotation.freq, dims, rotation.layout,
                        torch.tensor(positions, dtype=torch.int32, device="cuda"),
                        torch.arange(len(positions), dtype=torch.int32, device="cuda"), None, heads, 0, head, head, 4, unit_heads=True)
    f = torch.tensor([5000.0 ** (-2.0 * i / dims) / factor for i in range(dims // 2)], dtype=F64).float()
    for i, p in enumerate(positions):
        a = (torch.tensor(float(p), dtype=torch.float32) * f).double()
        turned = x[i].view(heads, head).double().clone()
        u, v = turned[:, 0:dims:2].clone(), turned[:, 1:dims:2].clone()
        turned[:, 0:dims:2], turned[:, 1:dims:2] = u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin()
        torch.testing.assert_close(q[i].cpu().view(heads, head), plain.unit_rms(turned, eps).float(), atol=3e-6, rtol=1e-5)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("width,stride", [(24, 64), (37, 81), (64, 128), (16, 40)])
def test_activation_over_a_column_range(dtype, width, stride):
    from qwen_inference_lab_b200.kernels import ops
    buffer = rows(7, stride, 3, 3.0)
    for column in (0, stride - 2 * width):
        out = ops.gated_activation(buffer.to(dtype).cuda(), "clamped_swish", limit=1.1, alpha=1.702, column=column, width=width)
        g = torch.clamp(buffer[:, column:column + width].double(), max=1.1)
        u = torch.clamp(buffer[:, column + width:column + 2 * width].double(), min=-1.1, max=1.1)
        expected = (g * torch.sigmoid(1.702 * g) * (u + 1)).float()
        torch.testing.assert_close(out.float().cpu(), expected, **(dict(atol=1e-6, rtol=1e-5) if dtype == torch.float32 else dict(atol=4e-3, rtol=8e-3)))


# ------------------------------------------------------------------ the mixers alone, through the step function
def left_part(hidden, m, eps=1e-5, prefix="m."):
    from qwen_inference_lab_b200.parts import GroupedQueryAttention, RotaryFrequencies
    rot = m["rot"]
    position = RotaryFrequencies(rot["dims"], rot["base"], "interleaved", stretch=(rot.get("scaling") or {}).get("factor", 1.0))
    return GroupedQueryAttention(hidden, m["heads"], m["kv_heads"], m["dim"], names={k: prefix + k for k in ("q", "k", "v", "o")},
                                 scale=m["scale"], v_head_dim=m["vdim"], suffixes=SUFFIX, position=position,
                                 window=m["mask"]["size"], unit_qk_norm_eps=eps)


def right_part(hidden, m, eps=1e-5, prefix="m."):
    from qwen_inference_lab_b200.parts import TiedGateLinearAttention
    return TiedGateLinearAttention(hidden, m["heads"], m["dim"], m["vdim"], norm_eps=eps, suffixes=SUFFIX, norm_suffix="",
                                   names={k: prefix + k for k in ("q", "f", "v", "o", "lower", "norm")})


def memory_part(hidden, m, eps=1e-5, prefix="m."):
    from qwen_inference_lab_b200.parts import MatrixMemory
    return MatrixMemory(hidden, m["heads"], m["dim"], m["vdim"], m["gate_cap"], norm_eps=eps, suffixes=SUFFIX, norm_suffix="",
                        names={k: prefix + k for k in ("q", "k", "v", "g", "i", "f", "o", "norm")})


LEFTS = [cases.left(4, 2, 32, 32, 0.2, 300000.0, 16, 24, 4.0),     # the tensor-core kernels in bfloat16; half a head rotated
         cases.left(6, 3, 16, 8, 0.3, 1000.0, 16, 7),              # values smaller than keys: the float32 kernel
         cases.left(3, 3, 20, 12, 0.22, 50.0, 4, 1, 2.0),          # a window of one position: a token sees itself
         cases.left(2, 1, 80, 80, 0.11, 500.0, 80, 4096),          # one key/value head, no window's edge in reach
         cases.left(6, 1, 16, 16, 0.25, 10000.0, 2, 33, 0.5),      # six query heads on one key/value head, one rotated pair
         cases.left(8, 2, 128, 128, 0.08, 500000.0, 64, 50),       # heads of 128, half of each rotated
         cases.left(2, 2, 24, 56, 0.2, 1e4, 24, 19, 3.0)]          # values larger than keys


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("m", LEFTS, ids=[f"d{m['dim']}w{m['mask']['size']}" for m in LEFTS])
def test_windowed_attention_whole_cut_and_side_by_side(dtype, m):
    part = left_part(72, m)
    w = fill(part, 21, dtype)
    inputs = {"a": rows(75, 72, 22), "b": rows(41, 72, 23)}
    expected = {rid: plain.window_attention_mixer(x.double(), w, "m.", m, 1e-5, low_of(dtype)) for rid, x in inputs.items()}
    for cuts in CUTS:
        got = through_the_step_function(part, 72, dtype, inputs, cuts, num_pages=48)
        for rid in inputs:
            close(got[rid], expected[rid], dtype)


@pytest.mark.parametrize("window", [1, 50, 64, 128, 200, 4096])
def test_whole_tiles_of_heads_of_128_take_the_tensor_memory_kernel_with_a_window(monkeypatch, window):
    """Whole 128-token tiles of a prompt go to the tcgen05 kernel, which starts at the first key that a tile's first row
    sees and masks, row by row, what lies before a later row's window; leftovers and single tokens take the tiled
    kernels.  Pages behind the window are gone by the second portion."""
    from qwen_inference_lab_b200.kernels import attention_tc
    calls = []
    original = attention_tc.prefill
    monkeypatch.setattr(attention_tc, "prefill", lambda *a, **k: (calls.append(k.get("window")), original(*a, **k))[1])
    m = cases.left(4, 2, 128, 128, 0.09, 10000.0, 128, window)
    part = left_part(64, m)
    w = fill(part, 31, torch.bfloat16)
    inputs = {"a": rows(460, 64, 32), "b": rows(140, 64, 33)}
    expected = {rid: plain.window_attention_mixer(x.double(), w, "m.", m, 1e-5, torch.bfloat16) for rid, x in inputs.items()}
    for cuts in ({"a": [460], "b": [140]}, {"a": [129, 1, 330], "b": [7, 133]}):
        got = through_the_step_function(part, 64, torch.bfloat16, inputs, cuts, page_size=16, num_pages=48)
        for rid in inputs:
            close(got[rid], expected[rid], torch.bfloat16)
    assert calls and all(call == window for call in calls)


RIGHTS = [cases.right(2, 16, 24), cases.right(3, 40, 8), cases.right(1, 64, 64), cases.right(5, 10, 6), cases.right(2, 128, 80),
          cases.right(1, 12, 300)]


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("m", RIGHTS, ids=[f"h{m['heads']}d{m['dim']}e{m['vdim']}" for m in RIGHTS])
def test_tied_gate_attention_whole_cut_and_side_by_side(dtype, m):
    """Short portions run token by token, portions of more than 128 tokens as chunks with a carry.  Lower bounds of exactly
    zero, of one (a channel that is never written) and next to one (a channel that forgets nothing)."""
    part = right_part(56, m)
    drawn = cases.draw_weights(part.all_named_params(), 31)
    drawn["m.lower"][:4] = torch.tensor([0.0, 1.0, 0.99609375, 0.5])
    w = fill(part, 31, dtype, drawn)
    inputs = {"a": rows(300, 56, 32), "b": rows(41, 56, 33)}
    expected = {rid: plain.hgrn2_mixer(x.double(), w, "m.", m, 1e-5, low_of(dtype)) for rid, x in inputs.items()}
    for cuts in SCAN_CUTS:
        got = through_the_step_function(part, 56, dtype, inputs, cuts, page_size=16, num_pages=24)
        for rid in inputs:
            close(got[rid], expected[rid], dtype, scale=float(expected[rid].abs().max()))


SCAN_CUTS = ({"a": [300], "b": [41]}, {"a": [2, 129, 1, 1, 64, 3, 100], "b": [1] * 9 + [2] * 6 + [20]},
             {"a": [150, 150], "b": [17, 24]}, {"a": [1] * 40 + [260], "b": [41]})

MEMORIES = [cases.memory(2, 16, 24, 15.0), cases.memory(3, 40, 8, 2.0), cases.memory(1, 64, 64, 30.0), cases.memory(5, 10, 6, 0.5),
            cases.memory(2, 128, 96, 12.0), cases.memory(1, 130, 33, 8.0)]


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("m", MEMORIES, ids=[f"h{m['heads']}d{m['dim']}e{m['vdim']}" for m in MEMORIES])
def test_matrix_memory_whole_cut_and_side_by_side(dtype, m):
    """Input gates of both signs and up to the cap, so that the running maximum rises, decays and rises again; one token
    far above the others in the middle; portions of every size carry memory, sum of keys and maximum on."""
    part = memory_part(56, m)
    drawn = cases.draw_weights(part.all_named_params(), 41)
    drawn["m.i"] = drawn["m.i"] * 2.0
    w = fill(part, 41, dtype, drawn)
    inputs = {"a": rows(300, 56, 42), "b": rows(41, 56, 43)}
    inputs["a"][140] *= 3.0
    expected = {rid: plain.mlstm_mixer(x.double(), w, "m.", m, 1e-5, low_of(dtype)) for rid, x in inputs.items()}
    for cuts in SCAN_CUTS:
        got = through_the_step_function(part, 56, dtype, inputs, cuts, page_size=16, num_pages=24)
        for rid in inputs:
            close(got[rid], expected[rid], dtype, scale=float(expected[rid].abs().max()))


@pytest.mark.parametrize("bias", [-20.0, -3.0, 0.0, 12.0])
def test_the_running_maximum_starts_at_zero_and_the_gates_walk_it(bias):
    """The gate kernel alone in float32, one long segment and the same in portions: the same maximum in the slot to the bit,
    decays, gains and floors as the recurrence has them."""
    from qwen_inference_lab_b200.kernels import ops
    heads, T, cap = 5, 210, 9.0
    gates = rows(T, 2 * heads + 3, 7, 5.0)
    bi, bf = torch.full((heads,), bias), torch.full((heads,), 1.5)
    log_i = plain.capped(gates[:, 3:3 + heads].double() + bi, cap)
    log_f = torch.nn.functional.logsigmoid(plain.capped(gates[:, 3 + heads:].double() + bf, cap))
    m, expected = torch.zeros(heads, dtype=F64), []
    for t in range(T):
        now = torch.maximum(log_f[t] + m, log_i[t])
        expected.append((torch.exp(log_f[t] + m - now), torch.exp(log_i[t] - now), torch.exp(-now)))
        m = now
    slots = {}
    for name, sizes in (("whole", [T]), ("cut", [1, 2, 31, 32, 33, 64, 1, 46])):
        slot = torch.full((3, heads), float("nan"), device="cuda")
        slot[1] = 0.0
        collected, first = [], 0
        for size in sizes:
            one = lambda v: torch.tensor([v], dtype=torch.int32, device="cuda")
            out = ops.mlstm_gates(gates[first:first + size].contiguous().cuda(), (3, 3 + heads), (bi.cuda(), bf.cuda()), cap, slot,
                                  one(0), one(size), one(1), 1)
            collected.append(torch.stack(out, dim=1).cpu())
            first += size
        slots[name] = (slot[1].cpu(), torch.cat(collected))
        assert slot[0].isnan().all() and slot[2].isnan().all()
    assert torch.equal(slots["whole"][0], slots["cut"][0]) and torch.equal(slots["whole"][1], slots["cut"][1])
    torch.testing.assert_close(slots["whole"][0], m.float(), atol=2e-5, rtol=1e-5)
    torch.testing.assert_close(slots["whole"][1], torch.stack([torch.stack(row) for row in expected]).float(), atol=1e-6, rtol=1e-4)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("scales", [(0.7, 1.3), (1.0, -0.25)])
def test_two_mixers_summed_by_scales(dtype, scales):
    from qwen_inference_lab_b200.parts import ParallelMixers
    ml, mr = cases.left(4, 2, 32, 32, 0.2, 300000.0, 16, 24, 2.0), cases.right(3, 24, 8)
    part = ParallelMixers(80, left_part(80, ml, prefix="m.left."), right_part(80, mr, prefix="m.right."), scales=scales)
    w = fill(part, 41, dtype)
    inputs = {"a": rows(75, 80, 42), "b": rows(41, 80, 43)}
    m = dict(left=ml, right=mr, left_scale=scales[0], right_scale=scales[1])
    expected = {rid: plain.parallel_mixer(x.double(), w, "m.", m, 1e-5, low_of(dtype)) for rid, x in inputs.items()}
    body = lambda ctx, x, view: part.forward(ctx, x, view)
    for cuts in CUTS:
        got = harness.run_part(part, 80, dtype, body, inputs, cuts, page_size=4, num_pages=48)
        for rid in inputs:
            close(got[rid], expected[rid], dtype)


@pytest.mark.parametrize("layer", [0, 1, 2, 3])
def test_a_block_with_its_first_products_joined_and_apart(layer):
    """Sublayers that read the same row run their first projections as one product: in float32 the block gives the same
    bits as with every part's own product, over portions and single tokens, and both are the plain layer."""
    from qwen_inference_lab_b200.config import registry
    from qwen_inference_lab_b200.parts.block import settle_stream
    entry = registry.lookup(cases.CASE_A)
    block = entry.build(entry.config_class.from_dict(cases.CASE_A)).layers[layer]
    w = fill(block, 51, torch.float32)
    spec, p = cases.CASE_A["layers"][layer], f"l{layer}."

    def body(ctx, x, view):
        out = block.forward(ctx, x.clone(), view)
        settle_stream(ctx)
        return out

    inputs = {"a": rows(75, 96, 52), "b": rows(41, 96, 53)}
    joint = block.input._w
    assert (joint is None) == (layer == 2)             # a memory without a feed-forward has one product anyway
    for cuts in CUTS:
        got = harness.run_part(block, 96, torch.float32, body, inputs, cuts, page_size=4, num_pages=48)
        block.input._w = None
        apart = harness.run_part(block, 96, torch.float32, body, inputs, cuts, page_size=4, num_pages=48)
        block.input._w = joint
        for rid, x in inputs.items():
            assert torch.equal(got[rid], apart[rid])
            h = plain.scalar_norm(x.double(), w[p + "norm1"], 1e-5)
            expected = x.double() + plain.MIXERS[spec["type"]](h, w, p + "mix.", spec["mixer"], 1e-5)
            if spec["mlp"]:
                expected = expected + plain.routed_experts(h, w, p + "mlp.", spec["mlp"])
            close(got[rid], expected, torch.float32, scale=float(expected.abs().max()))


# ------------------------------------------------------------------ one key made to stand out
WINDOW_EDGES = [(64, 127, 64, True), (64, 128, 64, False), (20, 19, 0, True), (20, 20, 0, False), (100, 200, 101, True),
                (100, 200, 100, False), (600, 650, 51, True), (600, 651, 51, False), (1, 9, 9, None), (1, 9, 8, False),
                (33, 64, 32, True), (33, 65, 32, False), (2, 8, 7, True), (2, 8, 6, False), (4096, 500, 0, True)]


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("single", [False, True], ids=["prompt", "decoded"])
@pytest.mark.parametrize("window,query,far,inside", WINDOW_EDGES)
def test_a_key_just_inside_and_just_outside_the_window(dtype, single, window, query, far, inside):
    """Heads are of unit size, so a key stands out by its direction only: the query's input is solved for so that every
    head's query, turned at its position, points along the far token's turned key (its score is then the largest a pair
    can have), and the far token's input is drawn again until it leads every other key by 30 in every head.  Just inside
    the window the output is that token's value; one position further it is not seen at all.  Pages behind the window
    have been given back by then.  A wrong angle, position or frequency loses the key."""
    hidden = 160
    m = cases.left(4, 2, 32, 32, 3.0, 10000.0, 8, window, 2.0)
    H, G, d, e, r = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["rot"]["dims"]
    part = left_part(hidden, m)
    w = fill(part, 61, dtype)
    W = {k: v.double() for k, v in w.items()}
    x = rows(query + 1, hidden, 62 + query, 0.5)
    freq = torch.tensor([m["rot"]["base"] ** (-2.0 * i / r) / 2.0 for i in range(r // 2)], dtype=F64)
    for attempt in range(60):
        if far == query:
            break
        x[far] = rows(1, hidden, 1000 + attempt, 0.5)[0]
        k_far = plain.unit_rms((x[far].double() @ W["m.k"].t()).view(G, d), 1e-5)
        turned = k_far.clone()                         # such that turned at the query's position it is k_far turned at its own
        pairs = torch.view_as_complex(k_far[:, :r].reshape(G, r // 2, 2).contiguous()) * torch.exp(1j * (far - query) * freq)
        turned[:, :r] = torch.view_as_real(pairs).reshape(G, r)
        target = torch.stack([turned[a // (H // G)] for a in range(H)]).flatten()
        x[query] = (torch.linalg.pinv(W["m.q"]) @ target).to(torch.bfloat16).float()
        q = plain.unit_rms(plain.rotate_neighbours((x.double() @ W["m.q"].t()).view(-1, H, d), m["rot"]), 1e-5)[query]
        k = plain.unit_rms(plain.rotate_neighbours((x.double() @ W["m.k"].t()).view(-1, G, d), m["rot"]), 1e-5)
        scores = torch.stack([k[:, a // (H // G)] @ q[a] for a in range(H)]) * m["scale"]      # [H, T]
        others = torch.cat([scores[:, :far], scores[:, far + 1:]], dim=1)
        if float((scores[:, far] - others.max(dim=1).values).min()) > 30.0:
            break
    else:
        raise AssertionError("no input found whose key stands out")
    expected = plain.window_attention_mixer(x.double(), w, "m.", m, 1e-5, low_of(dtype))
    exact = plain.window_attention_mixer(x.double(), w, "m.", m, 1e-5)
    v_far = (x[far].double() @ W["m.v"].t()).view(G, e)
    alone = torch.stack([v_far[a // (H // G)] for a in range(H)]).flatten() @ W["m.o"].t()
    tail = 1 if single else min(5, query + 1)
    head = query + 1 - tail
    cuts = ([head - 2, 2] if head > 3 else [head] if head else []) + [tail]
    got = through_the_step_function(part, hidden, dtype, {"a": x}, {"a": cuts}, page_size=8, num_pages=(query + 1) // 8 + 3)["a"]
    assert inside is None or ((exact[query] - alone).abs().max() < 1e-6 * alone.abs().max()) == inside
    if dtype == torch.float32:                          # under this scale bfloat16 moves the other rows' softmax about
        close(got[-min(5, query + 1):], expected[-min(5, query + 1):], dtype)
    if inside:
        close(got[-1], alone, dtype)
    elif inside is False:
        assert (got[-1].double() - alone).abs().max() > 0.02 * alone.abs().max()
    else:
        close(got[-1], expected[query], dtype)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("single", [False, True], ids=["prompt", "decoded"])
@pytest.mark.parametrize("kind", ["tied gate", "memory"])
def test_the_state_remembers_a_token_from_far_back(dtype, single, kind):
    """Token 2 alone writes much: its input is solved for so that its gate opens, every other token is faint and its gate
    shut; nothing is forgotten to speak of.  The query 600 positions later is solved for as well: its q points along what
    token 2 wrote and its own gate stays shut.  Without token 2 the query's row is another one, so a lost state, a lost
    maximum or a lost sum of keys shows."""
    hidden, query, heads, d, e = 96, 602, 2, 16, 8
    x = rows(query + 1, hidden, 72, 0.05)
    pull = lambda system, target: (torch.linalg.pinv(torch.cat(system)) @ torch.cat(target)).to(torch.bfloat16).float()
    if kind == "tied gate":
        m = cases.right(heads, d, e)
        part, mixer = right_part(hidden, m), plain.hgrn2_mixer
        w = cases.draw_weights(part.all_named_params(), 71)
        w["m.f.b"], w["m.lower"] = torch.full((heads * d,), 9.0), torch.zeros(heads * d)
        x[2] = pull([w["m.f"], w["m.v"]], [torch.full((heads * d,), -10.0), rows(1, heads * e, 73, 5.0)[0]])
        x[query] = pull([w["m.f"], w["m.q"]], [torch.zeros(heads * d), torch.full((heads * d,), 2.0)])
    else:
        m = cases.memory(heads, d, e, 15.0)
        part, mixer = memory_part(hidden, m), plain.mlstm_mixer
        w = cases.draw_weights(part.all_named_params(), 71)
        w["m.f.b"], w["m.i.b"] = torch.full((heads,), 9.0), torch.full((heads,), -6.0)
        key = rows(1, heads * d, 74)[0]
        x[2] = pull([w["m.i"], w["m.f"], w["m.k"], w["m.v"]], [torch.full((heads,), 12.0), torch.zeros(heads), key, rows(1, heads * e, 73, 5.0)[0]])
        x[query] = pull([w["m.i"], w["m.f"], w["m.q"]], [torch.zeros(2 * heads), key])
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
        folder = tmp_path_factory.mktemp(f"lotazen{name}")
        weights = cases.write_folder(case["config"], case["seed"], folder)
        requests = {f"r{i}": cases.random_tokens(case["config"], n, 60 + i) for i, n in enumerate(case["lengths"])}
        result[name] = (folder, weights, requests)
    return result


@pytest.fixture(scope="module")
def truth(folders):
    """The plain rows of every case, in float64 and with bfloat16 roundings, and the rows whose routing is a close call."""
    return {name: (cases.plain_rows(requests, weights, cases.CASES[name]["config"]),
                   cases.plain_rows(requests, weights, cases.CASES[name]["config"], torch.bfloat16),
                   cases.close_calls(requests, weights, cases.CASES[name]["config"]))
            for name, (folder, weights, requests) in folders.items()}


def judge(actual, expected, low, skip, dtype, what):
    """``tests.test_larolorn_gpu.judge``; bfloat16 rows whose choice of experts is a close call are not judged."""
    assert set(actual) == set(expected), f"{what}: different (request, position) sets"
    if dtype == torch.bfloat16:
        actual, expected, low = ({k: v for k, v in rows_.items() if k not in skip} for rows_ in (actual, expected, low))
    judge_rows(actual, expected, low, dtype, what)


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
    expected, low, skip = truth[case]
    judge(actual, expected, low, skip, dtype, f"lotazen {case} {schedule} {dtype}")


@pytest.mark.parametrize("case", list(cases.CASES))
def test_float32_rows_agree_under_every_schedule(folders, case):
    """Portions of up to 128 tokens and single tokens walk the states token by token, attention walks key tiles aligned
    to positions and float32 products sum in ascending order: such schedules give the same bits.  A longer portion's
    states come through the chunked scan's carry, which rounds differently in the last bits."""
    runs = {name: replay(folders, case, name, torch.float32) for name in SCHEDULES}
    longest = max(cases.CASES[case]["lengths"])
    for name, got in runs.items():
        if longest <= 128:
            different = [key for key in sorted(got) if not torch.equal(got[key], runs["chunks"][key])]
        else:
            different = [key for key in sorted(got) if not torch.allclose(got[key], runs["chunks"][key], atol=5e-5, rtol=1e-5)]
        assert not different, \
            f"lotazen {case}: {len(different)} rows of schedule {name} differ from the run in portions, first {different[0]}"
    for name in ("tail_decode", "mixed"):
        short = [key for key in sorted(runs[name]) if len(folders[case][2][key[0]]) <= 128]
        assert all(torch.equal(runs[name][key], runs["chunks"][key]) for key in short)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("case", ["A", "C"])
def test_long_decoding_and_the_first_tokens(folders, dtype, case):
    """Three tokens as a prompt, then 300 single tokens (recorded graphs) across many window edges, every position judged;
    the pool holds fewer pages than the positions need, because windows that have passed give theirs back."""
    folder, weights, _ = folders[case]
    config, page_size = cases.CASES[case]["config"], cases.CASES[case]["page_size"]
    tokens = cases.random_tokens(config, 303, 99)
    schedule = [([("r", tokens[:3], [0, 1, 2])], [])]
    schedule += [([("r", [tokens[i]], [0])], ["r"] if i == 302 else []) for i in range(3, 303)]
    _, cache, runner = harness.build_engine_parts(folder, dtype, num_pages={"A": 10, "C": 20}[case], page_size=page_size)
    actual = harness.run_schedule(runner, cache, schedule)
    assert runner._graphs, "single-token steps should have been recorded"
    expected = cases.plain_rows({"r": tokens}, weights, config)
    low = cases.plain_rows({"r": tokens}, weights, config, torch.bfloat16) if dtype == torch.bfloat16 else None
    judge(actual, expected, low, set(), dtype, f"lotazen {case} long decoding {dtype}")


def test_a_request_longer_than_the_table_of_positions_is_refused(folders):
    from qwen_inference_lab_b200.engine import StepEntry
    from qwen_inference_lab_b200.engine.step import StepError
    folder, _, _ = folders["C"]
    _, cache, runner = harness.build_engine_parts(folder, torch.float32, num_pages=200, page_size=2)
    assert cache.admit("r")
    runner.run([StepEntry("r", [1] * 310, [])])
    with pytest.raises(StepError, match="310 positions"):
        runner.run([StepEntry("r", [1], [0])])


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
    expected, low, skip = truth["A"]
    judge(got, expected, low, skip, torch.float32 if dtype == "float32" else torch.bfloat16, f"lotazen replay program {dtype}")


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
