"""Gated linear attention: a recurrent mixer whose state is a matrix per head, decayed per key channel.

Per head, with d key channels and e value channels, for the tokens of a sequence in order:

    a_t = sigmoid(A2 (A1 x_t) + b)^(1/tau)          decay per key channel, float32
    S_t = diag(a_t) S_(t-1) + k_t v_t^T              S_0 = 0, float32, one per request and layer call
    o_t = S_t^T (q_t * q_scale)
    y_t = W_o ( rmsnorm_e(o_t; w) * silu(W_g x_t) )  the norm is over a head's e values, w shared by heads

q, k, v, the gate and the low-rank input of the decay are one stacked product; the decays are a small kernel
of their own (``kernels.ops.gla_decay``); the recurrence, the norm and the gate are one kernel that walks a segment of the step from the request's state slot
(``kernels.ops.gla_scan``): single decoded tokens and prompt portions of up to ``LONG_SEGMENT`` tokens take it
token by token, and their result does not depend on the cut to the last bit.  Longer portions are cut into
chunks of ``CHUNK`` tokens that run side by side: every chunk's own state from zero, a carry over the chunks
in order, then every chunk again from its incoming state (twice the arithmetic, all chunks at once; the
carry rounds differently from the token-by-token scan, in the last bits).
"""
from __future__ import annotations

import torch

import numpy as np

from ..kernels import ops
from .base import Mixer, Param, StateSpec, StepPlanner
from .linear import Linear, StackedLinear

CHUNK = 64              # tokens of a chunk of a long segment
LONG_SEGMENT = 128      # segments longer than this are cut into chunks


class ScanPlanner(StepPlanner):
    """A step's segments as the scan wants them: the short ones as they are (first token, tokens, state slot),
    the long ones as chunks (first token, tokens, index among the step's chunks) and one carry entry per long
    segment (state slot, first chunk, chunks).  All recurrent layers of a model share the plan."""
    key = "state_scan"

    def plan(self, segments):
        lens = np.asarray(segments.lens)
        short = np.nonzero(lens <= LONG_SEGMENT)[0]
        chunks, carry = [], []
        for i in np.nonzero(lens > LONG_SEGMENT)[0]:
            first, count = int(segments.first[i]), int(lens[i])
            carry.append((int(segments.rows[i]), len(chunks), -(-count // CHUNK)))
            chunks += [(first + off, min(CHUNK, count - off), len(chunks) + off // CHUNK) for off in range(0, count, CHUNK)]
        chunks = np.array(chunks, dtype=np.int64).reshape(-1, 3)
        return dict(short_start=segments.first[short], short_len=lens[short], short_row=np.asarray(segments.rows)[short],
                    chunk_start=chunks[:, 0], chunk_len=chunks[:, 1], chunk_index=chunks[:, 2],
                    carry=np.array(carry, dtype=np.int64).reshape(-1))

    def refresh_single_tokens(self, arrays, segments):
        return True         # single tokens in the same rows: nothing here depends on their positions


_PLANNER = ScanPlanner()


def _scratch_needs(d, e, ones=False):
    """(short segments, chunks): does the scan of each need the scratch buffer, since no block holds a whole head's row?"""
    return tuple(ops.gla_scan_needs_scratch(d, e, ones, mode) for mode in (ops.GLA_WHOLE, ops.GLA_FROM_STATE))


def _step_needs_scratch(plan, needs):
    """Of a step: the kernel that finishes the scratch buffer runs over all its tokens, so all scans use it or none."""
    return (plan.count["short_start"] > 0 and needs[0]) or (plan.count["chunk_start"] > 0 and needs[1])


class GatedLinearAttention(Mixer):
    """names: dict with keys q, k, v, g, o, a1, a2 (projection names) and norm (the output norm's weight).
    ``suffixes``: what the checkpoint appends to a projection's name for weight and bias."""
    graph_safe = True

    def __init__(self, hidden_size, n_heads, key_dim, value_dim, decay_rank, *, tau, norm_eps, names,
                 q_scale=None, suffixes=(".weight", ".bias"), norm_suffix=".weight"):
        self.hidden_size, self.n_heads = int(hidden_size), int(n_heads)
        self.key_dim, self.value_dim, self.decay_rank = int(key_dim), int(value_dim), int(decay_rank)
        self.tau, self.norm_eps = float(tau), float(norm_eps)
        if not self.tau > 0:
            raise ValueError("tau must be positive")
        self.q_scale = float(q_scale) if q_scale is not None else self.key_dim ** -0.5
        kw, vw = self.n_heads * self.key_dim, self.n_heads * self.value_dim
        self.projection = StackedLinear(hidden_size, [(names["q"], kw), (names["k"], kw), (names["v"], vw),
                                                      (names["g"], vw), (names["a1"], self.decay_rank)],
                                        suffixes=suffixes)
        self.columns = (0, kw, 2 * kw, 2 * kw + vw, 2 * kw + 2 * vw)
        self.decay_up = Param((kw, self.decay_rank), std=0.2)
        self.decay_bias = Param((kw,), init="zeros")
        self.norm_weight = Param((self.value_dim,), init="norm", std=0.05)
        self._names = {names["a2"] + suffixes[0]: self.decay_up, names["a2"] + suffixes[1]: self.decay_bias,
                       names["norm"] + norm_suffix: self.norm_weight}
        self.out = Linear(vw, hidden_size, name=names["o"], suffixes=suffixes)
        self._needs_scratch = False

    def named_params(self):
        return dict(self._names)

    def children(self):
        return [self.projection, self.out]

    def finalize(self, device, dtype):
        super().finalize(device, dtype)
        common = self.projection._weight().dtype
        for param in (self.decay_up, self.decay_bias, self.norm_weight):
            param.data = param.data.to(common).contiguous()
        self._needs_scratch = _scratch_needs(self.key_dim, self.value_dim)

    def cache_spec(self):
        return StateSpec((self.n_heads, self.key_dim, self.value_dim), torch.float32)

    def step_planners(self):
        return {**super().step_planners(), _PLANNER.key: _PLANNER}

    takes_norm = True

    def forward(self, ctx, x, cache, residual=None, norm=None):
        """x [N, hidden] -> [N, hidden] (+ residual); ``cache`` is a StateView with one slot per request row."""
        projected = self.projection.forward(ctx, x, norm=norm)
        mixed = ctx.empty((x.shape[0], self.n_heads * self.value_dim))
        self.scan(ctx, projected, cache, mixed)
        return self.out.forward(ctx, mixed, residual=residual)

    def scan(self, ctx, projected, cache, mixed):
        """The recurrence, the norm and the gate over the step's segments: ``projected`` -> ``mixed``."""
        n = projected.shape[0]
        plan = ctx.plans[_PLANNER.key]
        scratch = ctx.empty((n, self.n_heads * self.value_dim), dtype=torch.float32) \
            if _step_needs_scratch(plan, self._needs_scratch) else None
        alpha = ops.gla_decay(projected, self.columns[4], self.decay_up.data, self.decay_bias.data, self.tau)
        common = (projected, self.columns, alpha, self.q_scale, self.norm_weight.data, self.norm_eps)
        sizes = (self.n_heads, self.key_dim, self.value_dim, mixed)
        n_short, n_chunks = plan.count["short_start"], plan.count["chunk_start"]
        if n_short:
            ops.gla_scan(*common, cache.slots, plan.array["short_start"], plan.array["short_len"],
                         plan.array["short_row"], n_short, *sizes, scratch=scratch)
        if n_chunks:
            chunk = (plan.array["chunk_start"], plan.array["chunk_len"], plan.array["chunk_index"], n_chunks)
            states = ctx.empty((n_chunks, self.n_heads, self.key_dim, self.value_dim), dtype=torch.float32)
            decays = ctx.empty((n_chunks, self.n_heads, self.key_dim), dtype=torch.float32)
            ops.gla_scan(*common, states, *chunk, *sizes, mode=ops.GLA_OWN_STATE, decay_product=decays)
            ops.gla_carry(states, decays, cache.slots, plan.array["carry"], plan.count["carry"] // 3)
            ops.gla_scan(*common, states, *chunk, *sizes, scratch=scratch, mode=ops.GLA_FROM_STATE)
        if scratch is not None:
            ops.gla_norm_gate(scratch, projected, self.columns[3], self.norm_weight.data, self.norm_eps, self.n_heads,
                              self.value_dim, mixed)
        return mixed


class DecayLinearAttention(Mixer):
    """Linear attention with one fixed decay per head (a state matrix per head and request, float32):

        q_t = silu(Wq x_t), k_t = silu(Wk x_t)  [H][d];   v_t = silu(Wv x_t)  [H][e]
        S_t = decay_h S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t                   S_0 = 0
        y_t = Wo ( o_t / sqrt(mean(o_t^2) + eps) * w  *  sigmoid(Wg x_t) )     one norm over all heads' H * e values

    q, k, v and the gate are one stacked product.  The recurrence is the scan of :class:`GatedLinearAttention`
    (``kernels.ops.gla_scan``) with a decay per head in place of decays per token and the activation applied as
    q, k and v are read; it shares that mixer's step plan, so short segments run token by token and long ones as
    chunks with a carry.  The scan leaves the un-normed outputs in float32; ``kernels.ops.lin_norm_gate_whole``
    norms a token's whole row and gates it.

    names: dict with keys q, k, v, g, o (projection names) and norm (the output norm's weight)."""
    graph_safe = True

    def __init__(self, hidden_size, n_heads, key_dim, value_dim, decay, *, norm_eps, names,
                 suffixes=(".weight", ".bias"), norm_suffix=".weight"):
        self.hidden_size, self.n_heads = int(hidden_size), int(n_heads)
        self.key_dim, self.value_dim, self.norm_eps = int(key_dim), int(value_dim), float(norm_eps)
        self.decay = [float(v) for v in decay]
        if len(self.decay) != self.n_heads or any(not 0.0 <= v <= 1.0 for v in self.decay):
            raise ValueError("one decay in [0, 1] per head")
        kw, vw = self.n_heads * self.key_dim, self.n_heads * self.value_dim
        self.projection = StackedLinear(hidden_size, [(names["q"], kw), (names["k"], kw), (names["v"], vw), (names["g"], vw)],
                                        suffixes=suffixes)
        self.columns = (0, kw, 2 * kw, 2 * kw + vw)
        self.norm_weight = Param((vw,), init="norm", std=0.05)
        self._names = {names["norm"] + norm_suffix: self.norm_weight}
        self.out = Linear(vw, hidden_size, name=names["o"], suffixes=suffixes)
        self._decay = None

    def named_params(self):
        return dict(self._names)

    def children(self):
        return [self.projection, self.out]

    def finalize(self, device, dtype):
        super().finalize(device, dtype)
        self.norm_weight.data = self.norm_weight.data.to(self.projection._weight().dtype).contiguous()
        self._decay = torch.tensor(self.decay, dtype=torch.float64).to(torch.float32).to(device)
        ops.gla_scan_needs_scratch(self.key_dim, self.value_dim)       # refuses key sizes the scan cannot hold

    def cache_spec(self):
        return StateSpec((self.n_heads, self.key_dim, self.value_dim), torch.float32)

    def step_planners(self):
        return {**super().step_planners(), _PLANNER.key: _PLANNER}

    def forward(self, ctx, x, cache, residual=None, out_float32=False):
        """x [N, hidden] -> [N, hidden] (+ residual); ``cache`` is a StateView with one slot per request row."""
        projected = self.projection.forward(ctx, x)
        raw = self.scan(ctx, projected, cache)
        mixed = ctx.empty((x.shape[0], self.n_heads * self.value_dim))
        ops.lin_norm_gate_whole(raw, projected, self.columns[3], self.norm_weight.data, self.norm_eps, mixed)
        return self.out.forward(ctx, mixed, residual=residual, out_float32=out_float32)

    def scan(self, ctx, projected, cache):
        """The recurrence over the step's segments: ``projected`` -> the un-normed outputs, float32 [N, heads * e]."""
        n, heads, d, e = projected.shape[0], self.n_heads, self.key_dim, self.value_dim
        plan = ctx.plans[_PLANNER.key]
        raw = ctx.empty((n, heads * e), dtype=torch.float32)
        common = (projected, self.columns, None, 1.0, None, self.norm_eps)
        options = dict(head_decay=self._decay, silu_inputs="qkv", raw_only=True)
        n_short, n_chunks = plan.count["short_start"], plan.count["chunk_start"]
        if n_short:
            ops.gla_scan(*common, cache.slots, plan.array["short_start"], plan.array["short_len"], plan.array["short_row"],
                         n_short, heads, d, e, None, scratch=raw, **options)
        if n_chunks:
            chunk = (plan.array["chunk_start"], plan.array["chunk_len"], plan.array["chunk_index"], n_chunks)
            states = ctx.empty((n_chunks, heads, d, e), dtype=torch.float32)
            decays = ctx.empty((n_chunks, heads, d), dtype=torch.float32)
            ops.gla_scan(*common, states, *chunk, heads, d, e, None, mode=ops.GLA_OWN_STATE, decay_product=decays, **options)
            ops.gla_carry(states, decays, cache.slots, plan.array["carry"], plan.count["carry"] // 3)
            ops.gla_scan(*common, states, *chunk, heads, d, e, None, scratch=raw, mode=ops.GLA_FROM_STATE, **options)
        return raw


def _scan_step(ctx, slots, run, sizes):
    """The recurrence over a step's segments through ``run(state, starts, lens, rows, count, **mode)``: short segments
    from the request's slot and back, long ones as chunks with a carry (``ScanPlanner``)."""
    heads, d, e = sizes
    plan = ctx.plans[_PLANNER.key]
    n_short, n_chunks = plan.count["short_start"], plan.count["chunk_start"]
    if n_short:
        run(slots, plan.array["short_start"], plan.array["short_len"], plan.array["short_row"], n_short)
    if n_chunks:
        chunk = (plan.array["chunk_start"], plan.array["chunk_len"], plan.array["chunk_index"], n_chunks)
        states = ctx.empty((n_chunks, heads, d, e), dtype=torch.float32)
        decays = ctx.empty((n_chunks, heads, d), dtype=torch.float32)
        run(states, *chunk, mode=ops.GLA_OWN_STATE, decay_product=decays)
        ops.gla_carry(states, decays, slots, plan.array["carry"], plan.count["carry"] // 3)
        run(states, *chunk, mode=ops.GLA_FROM_STATE)


class TiedGateLinearAttention(Mixer):
    """Linear attention whose forget gate also decides what is written (HGRN2); per head, d channels and e values:

        q_t = silu(Wq x_t),  v_t = Wv x_t,  f_t = l + (1 - l) sigmoid(Wf x_t + b)      l, b: one number per channel
        S_t = diag(f_t) S_(t-1) + (1 - f_t) v_t^T,   o_t = S_t^T q_t                    S_0 = 0, float32
        y_t = Wo rms_e(o_t; w)                                                          w [e] shared by heads

    q, f and v are one stacked product.  The recurrence is the scan of :class:`GatedLinearAttention`
    (``kernels.ops.gla_scan``) with the gate made where the scan reads its logits, and the norm inside the scan where a
    head's values fit one block.

    names: dict with keys q, f, v, o (projection names), lower (the bound's full name) and norm."""
    graph_safe = True

    def __init__(self, hidden_size, n_heads, key_dim, value_dim, *, norm_eps, names, suffixes=(".weight", ".bias"),
                 norm_suffix=".weight"):
        self.hidden_size, self.n_heads = int(hidden_size), int(n_heads)
        self.key_dim, self.value_dim, self.norm_eps = int(key_dim), int(value_dim), float(norm_eps)
        kw, vw = self.n_heads * self.key_dim, self.n_heads * self.value_dim
        self.projection = StackedLinear(hidden_size, [(names["q"], kw), (names["f"], kw), (names["v"], vw)], suffixes=suffixes)
        self.columns = (0, kw, 2 * kw)
        self.gate_bias = Param((kw,), init="normal", std=1.0)
        self.gate_lower = Param((kw,), init="zeros")
        self.norm_weight = Param((self.value_dim,), init="norm", std=0.05)
        self._names = {names["f"] + suffixes[1]: self.gate_bias, names["lower"]: self.gate_lower,
                       names["norm"] + norm_suffix: self.norm_weight}
        self.out = Linear(vw, hidden_size, name=names["o"], suffixes=suffixes)
        self._needs_scratch = False

    def named_params(self):
        return dict(self._names)

    def children(self):
        return [self.projection, self.out]

    def finalize(self, device, dtype):
        super().finalize(device, dtype)
        for param in (self.gate_bias, self.gate_lower, self.norm_weight):      # float32 arithmetic: read as float32
            param.data = param.data.to(torch.float32).contiguous()
        self._needs_scratch = _scratch_needs(self.key_dim, self.value_dim)

    def cache_spec(self):
        return StateSpec((self.n_heads, self.key_dim, self.value_dim), torch.float32)

    def step_planners(self):
        return {**super().step_planners(), _PLANNER.key: _PLANNER}

    def input_projections(self):
        return [self.projection]

    def forward(self, ctx, x, cache, residual=None, out_float32=False, joint=None):
        """x [N, hidden] -> [N, hidden] (+ residual); ``cache`` is a StateView with one slot per request row."""
        projected, at = self.projection.columns_of(ctx, x, joint)
        mixed = self.scan(ctx, projected, at, cache)
        return self.out.forward(ctx, mixed, residual=residual, out_float32=out_float32)

    def scan(self, ctx, projected, at, cache):
        """The recurrence and the norm over the step's segments: columns of ``projected`` from ``at`` on -> [N, heads * e]."""
        n, sizes = projected.shape[0], (self.n_heads, self.key_dim, self.value_dim)
        mixed = ctx.empty((n, self.n_heads * self.value_dim))
        scratch = ctx.empty((n, self.n_heads * self.value_dim), dtype=torch.float32) \
            if _step_needs_scratch(ctx.plans[_PLANNER.key], self._needs_scratch) else None
        columns = (*(at + c for c in self.columns), None)

        def run(state, starts, lens, rows, count, **mode):
            ops.gla_scan(projected, columns, None, 1.0, self.norm_weight.data, self.norm_eps, state, starts, lens, rows, count,
                         *sizes, mixed, scratch=scratch, silu_inputs="q",
                         tied_gate=(self.gate_bias.data, self.gate_lower.data), **mode)

        _scan_step(ctx, cache.slots, run, sizes)
        if scratch is not None:
            ops.gla_norm_gate(scratch, projected, None, self.norm_weight.data, self.norm_eps, self.n_heads, self.value_dim,
                              mixed)
        return mixed


class MatrixMemory(Mixer):
    """The matrix memory of xLSTM (mLSTM); per head, d key channels and e values:

        q_t = Wq x_t d^(-1/2),  k_t = Wk x_t,  v_t = Wv x_t
        i_t = cap tanh((Wi x_t + bi) / cap),  f_t = log sigmoid(cap tanh((Wf x_t + bf) / cap))     one number per head
        m_t = max(f_t + m_(t-1), i_t)                                                              m_0 = 0
        S_t = exp(f_t + m_(t-1) - m_t) S_(t-1) + exp(i_t - m_t) k_t v_t^T,   n_t the same with k_t alone
        o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6)
        y_t = Wo ( rms_e(o_t) * w * sigmoid(Wg x_t) )                              w: one number per value of all heads

    q, k, v, g, i and f are one stacked product.  ``kernels.ops.mlstm_gates`` walks the gates and the running maximum of
    every segment and leaves a decay, a gain and a floor per token and head; with those the memory is the scan of
    :class:`GatedLinearAttention` (``kernels.ops.gla_scan``) with a column of ones behind the values, which is n; the
    scan divides, norms and gates its outputs too where a head's columns fit one block.  State: (S beside n, m), float32.

    names: dict with keys q, k, v, g, i, f, o (projection names) and norm."""
    graph_safe = True

    def __init__(self, hidden_size, n_heads, key_dim, value_dim, gate_cap, *, norm_eps, names,
                 suffixes=(".weight", ".bias"), norm_suffix=".weight", q_scale=None):
        self.hidden_size, self.n_heads = int(hidden_size), int(n_heads)
        self.key_dim, self.value_dim = int(key_dim), int(value_dim)
        self.gate_cap, self.norm_eps = float(gate_cap), float(norm_eps)
        if not self.gate_cap > 0:
            raise ValueError("the gates' cap must be positive")
        self.q_scale = float(q_scale) if q_scale is not None else self.key_dim ** -0.5
        kw, vw = self.n_heads * self.key_dim, self.n_heads * self.value_dim
        pieces = [("q", kw), ("k", kw), ("v", vw), ("g", vw), ("i", self.n_heads), ("f", self.n_heads)]
        self.projection = StackedLinear(hidden_size, [(names[k], rows) for k, rows in pieces], suffixes=suffixes)
        self.columns, at = {}, 0
        for key, rows in pieces:
            self.columns[key] = at
            at += rows
        self.i_bias = Param((self.n_heads,), init="normal", std=1.0)
        self.f_bias = Param((self.n_heads,), init="norm", std=1.0)
        self.norm_weight = Param((vw,), init="norm", std=0.05)
        self._names = {names["i"] + suffixes[1]: self.i_bias, names["f"] + suffixes[1]: self.f_bias,
                       names["norm"] + norm_suffix: self.norm_weight}
        self.out = Linear(vw, hidden_size, name=names["o"], suffixes=suffixes)
        self._needs_scratch = False

    def named_params(self):
        return dict(self._names)

    def children(self):
        return [self.projection, self.out]

    def finalize(self, device, dtype):
        super().finalize(device, dtype)
        for param in (self.i_bias, self.f_bias, self.norm_weight):
            param.data = param.data.to(torch.float32).contiguous()
        self._needs_scratch = _scratch_needs(self.key_dim, self.value_dim + 1, ones=True)

    def cache_spec(self):
        return (StateSpec((self.n_heads, self.key_dim, self.value_dim + 1), torch.float32),
                StateSpec((self.n_heads,), torch.float32))

    def step_planners(self):
        return {**super().step_planners(), _PLANNER.key: _PLANNER}

    def input_projections(self):
        return [self.projection]

    def forward(self, ctx, x, cache, residual=None, out_float32=False, joint=None):
        """x [N, hidden] -> [N, hidden] (+ residual); ``cache`` is a pair of StateViews (the memory, the maximum)."""
        projected, at = self.projection.columns_of(ctx, x, joint)
        mixed = self.scan(ctx, projected, at, cache)
        return self.out.forward(ctx, mixed, residual=residual, out_float32=out_float32)

    def scan(self, ctx, projected, at, cache):
        """Gates, recurrence, norm and output gate: columns of ``projected`` from ``at`` on -> [N, heads * e]."""
        memory, maximum = cache
        n, sizes = projected.shape[0], (self.n_heads, self.key_dim, self.value_dim + 1)
        column = {key: at + first for key, first in self.columns.items()}
        decay, gain, floor = ops.mlstm_gates(projected, (column["i"], column["f"]), (self.i_bias.data, self.f_bias.data),
                                             self.gate_cap, maximum.slots, ctx.seg_start, ctx.seg_len, ctx.seg_row,
                                             ctx.n_segments)
        mixed = ctx.empty((n, self.n_heads * self.value_dim))
        columns = (column["q"], column["k"], column["v"], column["g"])
        raw, finish = None, dict(floor=floor)
        if _step_needs_scratch(ctx.plans[_PLANNER.key], self._needs_scratch):      # a head's columns are spread over several blocks, which cannot norm them
            raw, finish = ctx.empty((n, self.n_heads, self.value_dim + 1), dtype=torch.float32), dict(raw_only=True)

        def run(state, starts, lens, rows, count, **mode):
            ops.gla_scan(projected, columns, None, self.q_scale, self.norm_weight.data, self.norm_eps, state, starts, lens, rows,
                         count, *sizes, mixed, scratch=raw, token_scalars=(decay, gain), ones=True, **finish, **mode)

        _scan_step(ctx, memory.slots, run, sizes)
        if raw is not None:
            ops.mlstm_finish(raw, floor, projected, column["g"], self.norm_weight.data, self.norm_eps, mixed)
        return mixed
