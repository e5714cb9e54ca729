"""Lotazen as an arrangement of parts, with the checkpoint's tensor names.

Layer i (tensors ``l<i>.*``) has one norm, a root-mean-square norm with a single learned number (``norm1``), and both
sublayers read its output: x <- x + mixer(h) + ff(h), h = norm1(x).  The stream starts as the token's row of ``embed``
plus the position's row of ``pos``; after ``final.norm`` (the same kind of norm) and ``head`` the logits are capped:
cap * tanh(logits / cap).  The residual stream, the norms, the angles of the rotation, attention scores, the gates and
states of the recurrences and the routers are float32 whatever the activation dtype is.

``parallel``          two mixers side by side: left_scale * left + right_scale * right.  ``left`` a grouped attention with a
                      sliding window, q and k rotated (interleaved, all frequencies divided by ``rot.scaling.factor``)
                      and divided by their own root mean square per head; ``right`` HGRN2, a linear attention whose
                      forget gate also decides what is written (``parts.linear_attention.TiedGateLinearAttention``).
``mlstm``, ``mlstm_2``  the matrix memory of xLSTM (``parts.linear_attention.MatrixMemory``).
``moe``               sigmoid scores, the ``top`` largest multiply their experts' inputs; an expert is
                      down(g * sigmoid(1.702 g) * (u + 1)), g = min(gate x, limit), u = clamp(up x, -limit, limit); a
                      shared expert of the same form runs for every token.
"""
from __future__ import annotations

import torch

from ..config.model_config import LotazenConfig
from ..config.registry import register
from ..parts import (DecoderModel, GatedMLP, GroupedQueryAttention, LayerCall, Linear, MatrixMemory, ParallelBlock,
                     ParallelMixers, RotaryFrequencies, RoutedExperts, ScalarRMSNorm, TiedGateLinearAttention,
                     TokenEmbedding)

BARE = ("", ".b")          # this design's tensors carry the projection's own name; biases add ".b"
SWISH_ALPHA = 1.702        # the experts' activation: g * sigmoid(1.702 g)


def _parallel(width, m, prefix, eps):
    left, right = m["left"], m["right"]
    rot = left["rot"]
    position = RotaryFrequencies(rot["dims"], rot["base"], "interleaved", stretch=(rot.get("scaling") or {}).get("factor", 1.0))
    attention = GroupedQueryAttention(
        width, left["heads"], left["kv_heads"], left["dim"], names={k: f"{prefix}left.{k}" for k in ("q", "k", "v", "o")},
        scale=left["scale"], v_head_dim=left["vdim"], suffixes=BARE, position=position,
        window=(left.get("mask") or {}).get("size", 0), unit_qk_norm_eps=eps)
    recurrent = TiedGateLinearAttention(
        width, right["heads"], right["dim"], right["vdim"], norm_eps=eps, suffixes=BARE, norm_suffix="",
        names={k: f"{prefix}right.{k}" for k in ("q", "f", "v", "o", "lower", "norm")})
    return ParallelMixers(width, attention, recurrent, scales=(m["left_scale"], m["right_scale"]))


def _matrix_memory(width, m, prefix, eps):
    return MatrixMemory(width, m["heads"], m["dim"], m["vdim"], m["gate_cap"], norm_eps=eps, suffixes=BARE, norm_suffix="",
                        names={k: prefix + k for k in ("q", "k", "v", "g", "i", "f", "o", "norm")})


_MIXERS = {"parallel": _parallel, "mlstm": _matrix_memory, "mlstm_2": _matrix_memory}


def _feed_forward(width, mlp, prefix):
    if mlp is None:
        return None
    shared = None
    if mlp.get("shared"):
        shared = GatedMLP(width, mlp["shared"]["ff"], names={k: f"{prefix}shared.{k}" for k in ("gate", "up", "down")},
                          activation="clamped_swish", limit=mlp["shared"]["limit"], alpha=SWISH_ALPHA, suffixes=BARE)
    names = dict(router=prefix + "router", expert=lambda index, which: f"{prefix}e{index}.{which}")
    return RoutedExperts(width, mlp["expert"]["ff"], mlp["router"]["experts"], mlp["router"]["top"], names=names,
                         activation="clamped_swish", limit=mlp["expert"]["limit"], alpha=SWISH_ALPHA, shared=shared,
                         routing="sigmoid", weigh_input=True)


def build_lotazen(config: LotazenConfig, tensor_shapes=None) -> DecoderModel:
    width, eps = config.width, config.eps
    norm = lambda name: ScalarRMSNorm(width, eps, name=name, suffix="")
    layers = [ParallelBlock(norm(f"l{i}.norm1"), _MIXERS[layer["type"]](width, layer["mixer"], f"l{i}.mix.", eps),
                            _feed_forward(width, layer.get("mlp"), f"l{i}.mlp.")) for i, layer in enumerate(config.layers)]
    # the table of positions is as long as the checkpoint's, which bounds a request as max_positions does
    rows = tensor_shapes["pos"][0] if tensor_shapes and len(tensor_shapes.get("pos", ())) == 2 else config.max_positions
    return DecoderModel(config=config,
                        embedding=TokenEmbedding(config.vocab_size, width, name="embed", suffix="", positions=("pos", rows)),
                        layers=layers, order=[LayerCall(i) for i in range(len(layers))], final_norm=norm("final.norm"),
                        head=Linear(width, config.vocab_size, name="head", suffixes=BARE),
                        max_positions=min(rows, config.max_positions), stream_dtype=torch.float32,
                        logit_softcap=config.logit_softcap)


ARCHITECTURE = register(LotazenConfig.architecture, LotazenConfig.model_type, LotazenConfig, build_lotazen, shape_aware=True)
