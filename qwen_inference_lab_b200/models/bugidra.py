"""Bugidra as an arrangement of parts, with the checkpoint's tensor names.

Layer i (tensors ``l<i>.*``) is pre-norm, x <- x + mixer(norm1 x), x <- x + ff(norm2 x), and its norms are Dynamic Tanh:
tanh(alpha x) w + b, with alpha (``norm1.alpha``) and b (``norm1.b``) beside the weight.  A token's row of ``embed`` enters the
stream times ``embedding.scale``; after ``final.norm`` comes ``head``.  The residual stream, the norms, the angles of the
rotations, attention scores and everything that enters a recurrence, with its state, are float32 whatever the activation
dtype is.

``parallel``   two mixers side by side (``parts.parallel``), each output normed over the width, half their sum: ``left`` a
               grouped attention whose q and k are turned by halves (``rot.scaling``: YaRN's ramp) and divided by their own
               root mean square per head; ``right`` a retention (``parts.matrix_state.Retention``).
``attention``  a grouped attention with q and k normed over the whole projection, turned by neighbours, capped scores, a
               sigmoid gate per output element; with ``v_mix`` its values are mixed with the first such layer's.
``delta``      the gated delta rule behind short convolutions (``parts.matrix_state.GatedDeltaRule``).
``dense``      down(gelu_tanh(gate x) * up x).
"""
from __future__ import annotations

import torch

from ..config.model_config import BugidraConfig
from ..config.registry import register
from ..parts import (DecoderModel, DeferredPreNormBlock, GatedDeltaRule, GatedMLP, GroupedQueryAttention, LayerCall, Linear,
                     ParallelMixers, Retention, RotaryFrequencies, TanhNorm, TokenEmbedding)

BARE = ("", ".b")          # this design's tensors carry the projection's own name


def _rotation(rot, layout):
    scaling = rot.get("scaling")
    ramp = None if scaling is None else tuple(scaling[k] for k in ("factor", "original", "fast", "slow"))
    return RotaryFrequencies(rot["dims"], rot["base"], layout, ramp=ramp)


def _parallel(width, m, prefix, eps, first_values):
    left, right = m["left"], m["right"]
    attention = GroupedQueryAttention(
        width, left["heads"], left["kv_heads"], left["dim"], names={k: f"{prefix}left.{k}" for k in ("q", "k", "v", "o")},
        scale=left["scale"], v_head_dim=left["vdim"], suffixes=BARE, position=_rotation(left["rot"], "halves"),
        unit_qk_norm_eps=eps)
    recurrent = Retention(width, right["heads"], right["dim"], right["vdim"], right["decay"], norm_eps=eps, suffixes=BARE,
                          position=_rotation(right["rot"], "halves"),
                          names={k: f"{prefix}right.{k}" for k in ("q", "k", "v", "g", "o")})
    return ParallelMixers(width, attention, recurrent, norm_eps=eps, share=0.5, norm_suffix="",
                          names=dict(left_out=prefix + "left.out", right_out=prefix + "right.out"))


def _attention(width, m, prefix, eps, first_values):
    names = {k: prefix + k for k in ("q", "k", "v", "o")}
    names.update(q_norm=prefix + "q.norm", k_norm=prefix + "k.norm")
    return GroupedQueryAttention(
        width, m["heads"], m["kv_heads"], m["dim"], names=names, scale=m["scale"], v_head_dim=m["vdim"], suffixes=BARE,
        position=_rotation(m["rot"], "interleaved"), whole_qk_norm_eps=eps, norm_suffix="", softcap=m.get("softcap") or 0.0,
        element_gate=prefix + "g", value_mix=(prefix + "vmix", first_values) if m.get("v_mix") else None)


def _delta(width, m, prefix, eps, first_values):
    return GatedDeltaRule(width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], norm_eps=eps, suffixes=BARE,
                          norm_suffix="", conv_suffix=".conv",
                          names={k: prefix + k for k in ("q", "k", "v", "g", "b", "a", "o", "A_log", "dt_bias", "norm")})


_MIXERS = {"parallel": _parallel, "attention": _attention, "delta": _delta}


def build_bugidra(config: BugidraConfig) -> DecoderModel:
    width, eps = config.width, config.eps
    norm = lambda name, optional=False: TanhNorm(width, name=name, suffixes=("", ".b", ".alpha"), optional=optional)
    first = next((i for i, layer in enumerate(config.layers) if layer["type"] == "attention" and layer["mixer"].get("v_mix")), None)
    layers = []
    for i, layer in enumerate(config.layers):
        prefix, mlp = f"l{i}.", layer.get("mlp")
        feed_forward = None if mlp is None else GatedMLP(
            width, mlp["ff"], names={k: f"{prefix}mlp.{k}" for k in ("gate", "up", "down")}, activation="gelu_tanh", suffixes=BARE)
        layers.append(DeferredPreNormBlock(norm(prefix + "norm1"),
                                           _MIXERS[layer["type"]](width, layer["mixer"], prefix + "mix.", eps, i == first),
                                           norm(prefix + "norm2", optional=mlp is None), feed_forward))
    return DecoderModel(config=config,
                        embedding=TokenEmbedding(config.vocab_size, width, name="embed", suffix="", scale=config.embedding_scale),
                        layers=layers, order=[LayerCall(i) for i in range(len(layers))], final_norm=norm("final.norm"),
                        head=Linear(width, config.vocab_size, name="head", suffixes=BARE),
                        max_positions=config.max_positions, stream_dtype=torch.float32)


ARCHITECTURE = register(BugidraConfig.architecture, BugidraConfig.model_type, BugidraConfig, build_bugidra)
