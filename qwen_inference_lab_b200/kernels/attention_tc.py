"""The tcgen05/TMA attention for whole 128-token query tiles (bfloat16, head and value sizes up to 128), compiled per pair of
sizes on first use.

``prefill`` takes tiles of exactly 128 tokens; :func:`attention_mma.prefill` takes what is left.
The kernel's mbarrier waits are bounded and report through an error word that ``check()`` reads.
"""
from __future__ import annotations

from ctypes import c_float, c_int

import torch

from . import build
from . import ops
from .ops import KernelError, _check, _need, _p, _stream

MOST_DIM = 128
TILE = 128
_libs: dict = {}
_fault = ops.ErrorWord(lambda code: f"attention_tc: a wait inside the kernel ran out (code {code}: 1x producer, "
                                    f"13-17 MMA issuer, 2x softmax warps)")


def library_name(head_dim=MOST_DIM, v_dim=None):
    """(name, defines) of the library for queries and keys of ``head_dim`` and values of ``v_dim`` (None: the same)."""
    v_dim = head_dim if v_dim is None else v_dim
    if head_dim == v_dim == MOST_DIM:
        return "qil_attn_tc", {}
    return f"qil_attn_tc_d{head_dim}_v{v_dim}", {"QIL_HEAD_DIM": head_dim, "QIL_V_DIM": v_dim}


def library(head_dim=MOST_DIM, v_dim=None):
    v_dim = head_dim if v_dim is None else v_dim
    lib = _libs.get((head_dim, v_dim))
    if lib is None:
        name, defines = library_name(head_dim, v_dim)
        lib = build.load(name, ["attention_tc.cu"], defines)
        ops.register_post_step_check(check)
        if lib.qil_attn_tc_head_dim() != head_dim or lib.qil_attn_tc_v_dim() != v_dim:
            raise KernelError("attention_tc was built for other head sizes")
        _libs[(head_dim, v_dim)] = lib
    return lib


def supports(head_dim, page_size, window, v_dim=None) -> bool:
    fits = lambda size: size % 16 == 0 and 16 <= size <= MOST_DIM
    return fits(head_dim) and fits(head_dim if v_dim is None else v_dim) and window >= 0 and page_size in (8, 16, 32, 64)


def takes(options) -> bool:
    """Of the score options (``attention_mma.ScoreOptions``) this kernel has the cap, chunks and a learned sink."""
    return options.distance_bias is None and (not options.sink or options.sink_logits is not None)


def prefill(q, pages, out, tile_info, n_tiles, block_table, n_q_heads, n_kv_heads, page_size, scale, trace=None,
            lib=None, slopes_log2=None, chunk=0, sink_log2=None, softcap=0.0, window=0, head_dim=MOST_DIM, v_dim=None):
    """q bfloat16 [N, Hq*head_dim], out [N, Hq*v_dim] (``v_dim`` None: head_dim); pages [num_pages, 2, Hkv, page_size, head_dim],
    or with a value size of its own [num_pages, Hkv * page_size * (head_dim + v_dim)];
    tile_info int32 [n_tiles * 4] = (first token, its position, 128, block-table row).
    ``slopes_log2`` float32 [Hq] on the device: slope_h * log2(e) of a bias slope_h * (query position - key
    position) taken off the scaled score.  ``chunk`` > 0: a query sees the keys of its own chunk of that many
    positions only.  ``sink_log2`` float32 [Hq] on the device: learned scores times log2(e) whose exponentials join
    the softmax's denominator.  ``softcap`` > 0: score <- cap * tanh(score / cap) on the scaled product.
    ``window`` > 0: a query sees the last ``window`` positions, its own included."""
    if sink_log2 is not None:
        _need(sink_log2, "sink_log2", torch.float32, 1)
        if sink_log2.shape[0] != n_q_heads:
            raise KernelError("attention_tc: one sink score per query head")
    if slopes_log2 is not None:
        _need(slopes_log2, "slopes_log2", torch.float32, 1)
        if slopes_log2.shape[0] != n_q_heads:
            raise KernelError("attention_tc: one slope per query head")
    v_dim = head_dim if v_dim is None else v_dim
    _need(q, "q", torch.bfloat16, 2); _need(out, "out", torch.bfloat16, 2)
    ops.check_pages(pages, torch.bfloat16, n_kv_heads, page_size, head_dim, v_dim, "attention_tc")
    if q.shape[1] != n_q_heads * head_dim or out.shape != (q.shape[0], n_q_heads * v_dim):
        raise KernelError("attention_tc: shapes do not match the head counts")
    lib = lib or library(head_dim, v_dim)
    word = _fault.tensor(q.device)
    _fault.mark()
    _check(lib, lib.qil_attn_tc_prefill_capped(
        _p(q), _p(pages), _p(out), _p(tile_info), c_int(n_tiles), c_int(q.shape[0]), _p(block_table),
        c_int(block_table.shape[1]), c_int(n_q_heads), c_int(n_kv_heads), c_int(page_size), c_int(pages.shape[0]),
        c_float(scale), _p(slopes_log2), c_int(int(chunk or 0)), _p(sink_log2), c_float(float(softcap or 0.0)),
        c_int(int(window or 0)), _p(word), _p(trace), _stream()),
        "attention (128-token tiles)")


def check(wait=True) -> None:
    """Raise if a bounded wait inside a launch ran out (see ``ops.ErrorWord.check``)."""
    _fault.check(wait)
