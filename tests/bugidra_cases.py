"""Small Bugidra configurations and random weights for the tests.

The sizes differ from layer to layer and between the cases: head sizes the tensor-core attention takes and ones it does
not, values larger than, smaller than and as large as keys, one to six query heads per key/value head, rotations over all
and over two of a head's dimensions with and without YaRN's ramp (whose ends lie inside, before and behind the rotated pairs),
states whose columns one thread, two, four, eight and sixteen threads hold and whose values take one block or several,
decays of one and next to one, convolutions of one tap and of several, q/k heads shared by several value heads, value
mixing in three layers, in one and in none, caps present and absent, layers without a feed-forward.
"""
import json
from pathlib import Path

import torch

import qwen_inference_lab_b200.models  # noqa: F401  (registers the architectures)
from qwen_inference_lab_b200.config import registry
from qwen_inference_lab_b200.weights import write_safetensors
from tests.plain import bugidra_plain as plain


def rot(base, dims, scaling=None):
    result = dict(base=base, dims=dims)
    if scaling is not None:
        result["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return result


def left(heads, kv_heads, dim, vdim, scale, rotation):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, rot=rotation)


def right(dim, vdim, rotation, decay):
    return dict(heads=len(decay), dim=dim, vdim=vdim, rot=rotation, decay=list(decay))


def pair(left_mixer, right_mixer, ff=None):
    return dict(type="parallel", mixer=dict(left=left_mixer, right=right_mixer), mlp=dense(ff))


def attention(*sizes, cap=None, v_mix=False, ff=None):
    mixer = dict(left(*sizes), v_mix=v_mix)
    if cap is not None:
        mixer["softcap"] = cap
    return dict(type="attention", mixer=mixer, mlp=dense(ff))


def delta_sizes(heads, kv_heads, dim, vdim, taps):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=taps)


def delta(*sizes, ff=None):
    return dict(type="delta", mixer=delta_sizes(*sizes), mlp=dense(ff))


def dense(ff):
    return None if ff is None else dict(kind="dense", ff=ff)


def config(vocab, width, eps, scale, *layers):
    return dict(architecture="Bugidra", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=scale), layers=list(layers))


# requests of up to 128 tokens; tensor-core heads with values of their own size; three layers that mix values
CASE_A = config(173, 96, 1e-5, 3.0,
                pair(left(4, 2, 32, 16, 0.3, rot(10000.0, 16, (4.0, 64, 8.0, 1.0))), right(24, 16, rot(500.0, 8), (0.97, 1.0, 0.5)), 80),
                attention(4, 2, 32, 32, 0.25, rot(5000.0, 32), cap=20.0, v_mix=True, ff=64),
                delta(4, 2, 16, 24, 4),
                attention(6, 1, 48, 64, 0.15, rot(300.0, 10), v_mix=True),
                attention(2, 2, 16, 16, 0.4, rot(1e6, 16), cap=5.0, ff=40),
                attention(2, 2, 32, 32, 0.2, rot(5e4, 2), v_mix=True, ff=48))
# no convolution over time, a column spread over eight threads and one over sixteen (too wide for the chunks), a head's values
# over two blocks, a first layer that mixes but has no one to mix with
CASE_B = config(97, 64, 1e-6, 1.0,
                delta(1, 1, 130, 40, 1, ff=72),
                pair(left(2, 1, 80, 80, 0.11, rot(500.0, 80)), right(96, 140, rot(2000.0, 96, (8.0, 30, 2.0, 0.5)), (0.999,)), 40),
                attention(3, 3, 48, 48, 0.15, rot(20000.0, 2, (16.0, 500, 64.0, 3.0)), cap=30.0, v_mix=True),
                delta(2, 1, 260, 10, 3),
                pair(left(2, 2, 16, 32, 0.2, rot(100.0, 4)), right(10, 24, rot(10.0, 2), (0.8, 0.95, 0.99, 0.999)), 24))
# awkward sizes: a width that is a multiple of nothing, heads of 20 and 7 with values of 12 and 9, five heads on one q/k head
CASE_C = config(53, 70, 1e-5, 0.7,
                pair(left(3, 3, 20, 12, 0.22, rot(50.0, 4, (2.0, 16, 32.0, 1.0))), right(7, 11, rot(30.0, 6), (0.9, 0.99)), 37),
                delta(5, 1, 6, 9, 2, ff=31),
                attention(4, 2, 24, 40, 0.3, rot(1e6, 10), cap=8.0, v_mix=True),
                delta(3, 3, 33, 17, 5),
                attention(2, 1, 14, 80, 0.25, rot(77.0, 14), v_mix=True, ff=29))
# longer requests over pages of 16: heads of 128 whose whole 128-token tiles take the tensor-memory kernel, capped; several
# chunks of the recurrences in one portion
CASE_D = config(301, 256, 1e-5, 2.0,
                delta(4, 2, 64, 72, 4, ff=160),
                pair(left(4, 2, 128, 128, 0.09, rot(100000.0, 48, (2.0, 256, 32.0, 1.0))), right(32, 40, rot(1e5, 32), (0.98, 0.995, 0.9995, 0.6)), 128),
                attention(4, 2, 128, 128, 0.08, rot(10000.0, 64), cap=25.0, v_mix=True, ff=96),
                attention(4, 4, 128, 64, 0.1, rot(3000.0, 128), v_mix=True),
                delta(2, 2, 128, 130, 3, ff=64))
CASES = {"A": dict(config=CASE_A, seed=5, page_size=4, lengths=(70, 9, 33, 120, 1, 50)),
         "B": dict(config=CASE_B, seed=6, page_size=16, lengths=(40, 3, 300, 64, 25)),
         "C": dict(config=CASE_C, seed=7, page_size=2, lengths=(31, 2, 77, 20, 145)),
         "D": dict(config=CASE_D, seed=8, page_size=16, lengths=(400, 130, 17, 260))}


def draw_weights(params: dict, seed: int) -> dict:
    """name -> CPU float32 tensor of bfloat16-representable values for ``params`` (name -> Param): weights of norms around
    one, alphas around a half, decays of every kind, the embedding of order a half, matrices scaled by their input size."""
    generator = torch.Generator().manual_seed(seed)
    weights = {}
    for name, param in params.items():
        draw = torch.randn(param.shape, generator=generator)
        leaf = name.split(".")[-1]
        if leaf == "alpha":
            value = 0.5 + 0.1 * draw
        elif leaf == "vmix":
            value = 0.4 + 0.2 * draw
        elif leaf == "A_log":
            value = draw - 1.0
        elif leaf == "dt_bias":
            value = draw - 1.5
        elif leaf == "b" and len(param.shape) == 1:
            value = draw * 0.1
        elif leaf == "conv":
            value = draw * 0.7
        elif len(param.shape) < 2:
            value = 1.0 + draw * 0.1
        elif leaf == "embed":
            value = draw * 0.5
        else:
            value = draw * (param.shape[-1] ** -0.5)
        weights[name] = value.to(torch.bfloat16).float()
    return weights


def make_weights(config: dict, seed: int) -> dict:
    entry = registry.lookup(config)
    model = entry.build(entry.config_class.from_dict(config))
    return draw_weights(model.all_named_params(), seed)


def write_folder(config: dict, seed: int, folder) -> dict:
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    weights = make_weights(config, seed)
    (folder / "config.json").write_text(json.dumps(config))
    write_safetensors(folder / "model.safetensors", {k: v.to(torch.bfloat16) for k, v in weights.items()})
    return weights


def random_tokens(config, count, seed):
    return torch.randint(0, config["vocab"], (count,), generator=torch.Generator().manual_seed(seed)).tolist()


def plain_rows(requests, weights, config, low=None):
    """{(id, position): logits row} of the plain implementation (float64 arithmetic; with ``low`` float32
    arithmetic that rounds what the design allows in bfloat16)."""
    rows = {}
    for rid, tokens in requests.items():
        logits = plain.forward(config, weights, tokens, torch.float64 if low is None else torch.float32, low)
        for position in range(len(tokens)):
            rows[(rid, position)] = logits[position].float()
    return rows
