"""Small Lotazen configurations and random weights for the tests.

The sizes differ from layer to layer and between the cases: head sizes the tensor-core attention takes and ones it
does not, one to six query heads per key/value head, values larger than, smaller than and as large as keys, rotations
over all and over two of a head's dimensions with and without stretched frequencies, windows of one position, of a few
and longer than every request, states whose columns one thread, two, four and eight threads hold and whose values take
one block or several, memories of one head and of five, experts of which a token uses one, a few and all, with and
without a shared expert whose limit is another, layers without a feed-forward, scales and caps of one and absent.
"""
import json
from pathlib import Path

import torch

import qwen_inference_lab_b200.models  # noqa: F401  (registers the architectures)
from qwen_inference_lab_b200.config import registry
from qwen_inference_lab_b200.weights import write_safetensors
from tests.plain import lotazen_plain as plain


def left(heads, kv_heads, dim, vdim, scale, base, dims, window, factor=None):
    rot = dict(base=base, dims=dims)
    if factor is not None:
        rot["scaling"] = dict(factor=factor)
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, rot=rot, mask=dict(size=window))


def right(heads, dim, vdim):
    return dict(heads=heads, dim=dim, vdim=vdim)


def pair(left_mixer, right_mixer, left_scale, right_scale):
    return dict(type="parallel", mixer=dict(left=left_mixer, right=right_mixer, left_scale=left_scale, right_scale=right_scale))


def memory(heads, dim, vdim, gate_cap):
    return dict(heads=heads, dim=dim, vdim=vdim, gate_cap=gate_cap)


def mlstm(*sizes, kind="mlstm"):
    return dict(type=kind, mixer=memory(*sizes))


def moe(experts, top, ff, limit, shared=None):
    return dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=experts, top=top),
                shared=None if shared is None else dict(ff=shared[0], limit=shared[1]))


# every expert for every token (no close calls: bfloat16 is judged everywhere)
CASE_A = dict(architecture="Lotazen", vocab=173, width=96, norm=dict(eps=1e-5), max_positions=400, logit_softcap=25.0, layers=[
    dict(pair(left(4, 2, 32, 32, 0.2, 10000.0, 16, 24, 4.0), right(3, 24, 16), 0.7, 1.3), mlp=moe(4, 4, 24, 1.2, (40, 0.6))),
    dict(mlstm(3, 20, 28, 6.0), mlp=moe(3, 3, 16, 2.0, (24, 5.0))),
    dict(mlstm(2, 40, 16, 16.0, kind="mlstm_2"), mlp=None),
    dict(pair(left(6, 1, 16, 16, 0.3, 300.0, 16, 7), right(2, 64, 80), 1.0, 0.4), mlp=moe(5, 5, 32, 0.9, (16, 3.0))),
])
# one expert a token and two of five, no shared expert, no cap; windows of one position and longer than every request; one
# key/value head under two query heads of 80; a state of 300 values (two blocks), a memory of one head with 130 channels (a
# channel's column spread over eight threads); no scaling of the frequencies
CASE_B = dict(architecture="Lotazen", vocab=97, width=64, norm=dict(eps=1e-6), max_positions=320, layers=[
    dict(mlstm(1, 130, 40, 3.0), mlp=moe(3, 1, 48, 7.0)),
    dict(pair(left(2, 1, 80, 80, 0.11, 500.0, 80, 4096), right(1, 16, 300), 1.0, 1.0), mlp=moe(5, 2, 40, 1.0, (48, 1.5))),
    dict(pair(left(3, 3, 48, 48, 0.15, 20000.0, 2, 1, 16.0), right(4, 8, 8), 0.5, 0.25), mlp=None),
])
# awkward sizes: a width that is a multiple of nothing, heads of 20 with values of 12 (the float32 attention kernel), seven
# experts of eleven for every token, five heads of six channels and nine values
CASE_C = dict(architecture="Lotazen", vocab=53, width=70, norm=dict(eps=1e-5), max_positions=310, logit_softcap=35.0, layers=[
    dict(pair(left(3, 3, 20, 12, 0.22, 50.0, 4, 5, 2.0), right(5, 7, 11), 0.9, 1.1), mlp=None),
    dict(mlstm(5, 6, 9, 2.0, kind="mlstm_2"), mlp=moe(7, 7, 11, 0.5, (13, 0.8))),
    dict(pair(left(4, 2, 24, 40, 0.3, 1e6, 10, 33, 1.0), right(1, 33, 5), -0.6, 0.8), mlp=moe(2, 2, 37, 1.5, (9, 2.5))),
    dict(mlstm(2, 17, 70, 30.0), mlp=moe(3, 3, 8, 4.0)),
])
# longer requests over pages of 16: heads of 128 whose whole 128-token tiles take the tensor-memory kernel with a window that is
# a multiple of neither a page nor a key tile; requests beyond the chunked scan's length
CASE_D = dict(architecture="Lotazen", vocab=301, width=256, norm=dict(eps=1e-5), max_positions=512, logit_softcap=20.0, layers=[
    dict(pair(left(4, 2, 128, 128, 0.09, 100000.0, 48, 100, 4.0), right(4, 32, 40), 0.85, 0.95), mlp=moe(4, 4, 40, 1.0, (64, 2.0))),
    dict(mlstm(4, 32, 72, 14.0), mlp=moe(2, 2, 72, 1.4, (40, 0.9))),
    dict(pair(left(2, 2, 64, 64, 0.125, 10000.0, 64, 300), right(2, 128, 64), 1.1, 0.6), mlp=None),
    dict(mlstm(2, 64, 130, 8.0, kind="mlstm_2"), mlp=moe(3, 3, 48, 3.0, (24, 0.7))),
])
CASES = {"A": dict(config=CASE_A, seed=5, page_size=4, lengths=(70, 9, 33, 150, 1, 50)),
         "B": dict(config=CASE_B, seed=6, page_size=16, lengths=(40, 3, 300, 64, 25)),
         "C": dict(config=CASE_C, seed=7, page_size=2, lengths=(31, 2, 77, 20, 45)),
         "D": dict(config=CASE_D, seed=8, page_size=16, lengths=(400, 130, 17, 260))}


def draw_weights(params: dict, seed: int) -> dict:
    """name -> CPU float32 tensor of bfloat16-representable values for ``params`` (name -> Param): weights of norms
    around one, forget gates that keep most of what they hold, lower bounds between zero and one, the embedding of order
    a half, matrices scaled by their input size (the router's less, so that its scores are spread)."""
    generator = torch.Generator().manual_seed(seed)
    weights = {}
    for name, param in params.items():
        draw = torch.randn(param.shape, generator=generator)
        parts = name.split(".")
        leaf = parts[-1]
        if leaf == "b":
            value = draw + (2.0 if parts[-2] == "f" else 0.0)
        elif leaf == "lower":
            value = torch.sigmoid(draw)
        elif len(param.shape) < 2:
            value = 1.0 + draw * 0.1
        elif leaf == "embed":
            value = draw * 0.5
        elif leaf == "pos":
            value = draw * 0.3
        elif leaf == "router":
            value = draw * 2.0 * (param.shape[-1] ** -0.5)
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


CLOSE_CALL = 0.06      # a router margin (of outputs of order two) below which bfloat16 rounding can flip the choice


def close_calls(requests, weights, config):
    """The (id, position) that a close call in the choice of experts can reach: the position of the close call itself
    (in any layer) and, since later tokens attend to it and the states keep it, every later position of its request.
    bfloat16 runs are not judged there (another expert is another function; the float32 runs are judged everywhere)."""
    found = set()
    for rid, tokens in requests.items():
        margins = []
        plain.forward(config, weights, tokens, torch.float64, margins=margins)
        if margins:
            close = (torch.stack(margins).min(dim=0).values < CLOSE_CALL).nonzero().flatten()
            if len(close):
                found |= {(rid, p) for p in range(int(close[0]), len(tokens))}
    return found
