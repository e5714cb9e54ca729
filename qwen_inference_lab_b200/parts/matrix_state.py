"""Recurrent mixers with a state matrix per head and one decay per token and head: retention and the gated delta rule.

Both leave their projection's tail to a kernel that makes what enters the recurrence in float32 (``kernels.ops.rotate_rows``,
``kernels.ops.delta_prepare``) and share the recurrence itself (csrc/matrix_state.cu): segments of up to ``LONG_SEGMENT`` tokens
are walked token by token from the request's slot (``kernels.ops.state_scan``, the norm and the gate inside it where a block
holds all of a head's values), longer ones run as chunks in matrix products (``kernels.ops.state_chunks``).  The step plan is
the one of the other linear attentions (``parts.linear_attention.ScanPlanner``)."""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import Mixer, Param, StateSpec
from .linear import Linear, StackedLinear
from .linear_attention import ScanPlanner

_PLANNER = ScanPlanner()


class _MatrixStateMixer(Mixer):
    graph_safe = True

    def step_planners(self):
        return {**super().step_planners(), _PLANNER.key: _PLANNER}

    def children(self):
        return [self.projection, self.out]

    def input_projections(self):
        return [self.projection]

    def _settle_sizes(self):
        """Once on the device: may chunks be used, does a head's row of values take several blocks of the scan?"""
        self._chunks = self.key_dim <= ops.state_chunk_most_d()
        self._scratch = ops.state_scan_needs_scratch(self.key_dim, self.value_dim)

    def _recur(self, ctx, inputs, slots, gate, norm_weight, mixed):
        """The recurrence of ``inputs`` over the step's segments, the norm per head and the gate (rows, column) -> ``mixed``."""
        plan = ctx.plans[_PLANNER.key]
        if not self._chunks:          # heads too wide for the chunks' tiles: every segment token by token
            starts, lens, rows, n_short, n_chunks = ctx.seg_start, ctx.seg_len, ctx.seg_row, ctx.n_segments, 0
        else:
            starts, lens, rows = (plan.array[k] for k in ("short_start", "short_len", "short_row"))
            n_short, n_chunks = plan.count["short_start"], plan.count["chunk_start"]
        # the kernel that finishes raw outputs runs over all of the step's tokens, so all of them go there or none
        raw = ctx.empty(mixed.shape, dtype=torch.float32) if n_chunks or self._scratch else None
        if n_short:
            ops.state_scan(inputs, gate, norm_weight, self.norm_eps, slots, starts, lens, rows, n_short, out=mixed, raw=raw)
        if n_chunks:
            ops.state_chunks(inputs, slots, plan.array["chunk_start"], plan.array["chunk_len"], n_chunks, plan.array["carry"],
                             plan.count["carry"] // 3, raw)
        if raw is not None:
            ops.gla_norm_gate(raw, gate[0], gate[1], norm_weight, self.norm_eps, self.n_heads, self.value_dim, mixed)
        return mixed

    def forward(self, ctx, x, cache, residual=None, out_float32=False, joint=None):
        """x [N, hidden] -> [N, hidden] (+ residual); ``cache``: a StateView, or a tuple of them (see ``cache_spec``)."""
        projected, at = self.projection.columns_of(ctx, x, joint)
        mixed = self.scan(ctx, projected, at, cache)
        return self.out.forward(ctx, mixed, residual=residual, out_float32=out_float32)


class Retention(_MatrixStateMixer):
    """Linear attention with one fixed decay per head and rotated queries and keys; per head, d channels and e values:

        q_t = R(Wq x_t),  k_t = R(Wk x_t) k_scale,  v_t = Wv x_t          R: the rotation at the token's position
        S_t = decay S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t                S_0 = 0, float32
        y_t = Wo ( o_t / sqrt(mean_e(o_t^2) + eps) * silu(Wg x_t) )

    q, k, v and the gate are one stacked product.  names: dict with keys q, k, v, g, o (projection names).
    ``position``: a :class:`RotaryFrequencies`, or None."""

    def __init__(self, hidden_size, n_heads, key_dim, value_dim, decay, *, norm_eps, names, position=None, k_scale=None,
                 suffixes=(".weight", ".bias")):
        self.hidden_size, self.n_heads = int(hidden_size), int(n_heads)
        self.key_dim, self.value_dim, self.norm_eps = int(key_dim), int(value_dim), float(norm_eps)
        self.decay = [float(v) for v in decay]
        if len(self.decay) != self.n_heads or any(not 0.0 <= v <= 1.0 for v in self.decay):
            raise ValueError("one decay in [0, 1] per head")
        self.k_scale = float(k_scale) if k_scale is not None else self.key_dim ** -0.5
        self.position = position
        if position is not None and position.rotary_dim > self.key_dim:
            raise ValueError(f"{position.rotary_dim} rotated dimensions in heads of {self.key_dim}")
        kw, vw = self.n_heads * self.key_dim, self.n_heads * self.value_dim
        self.projection = StackedLinear(hidden_size, [(names["q"], kw), (names["k"], kw), (names["v"], vw), (names["g"], vw)],
                                        suffixes=suffixes)
        self.columns = (0, 2 * kw, 2 * kw + vw)                 # q (and k behind it), v, g
        self.out = Linear(vw, hidden_size, name=names["o"], suffixes=suffixes)
        self._decay = None

    def children(self):
        return super().children() + ([self.position] if self.position is not None else [])

    def finalize(self, device, dtype):
        super().finalize(device, dtype)
        self._decay = torch.tensor(self.decay, dtype=torch.float64).to(torch.float32).to(device)
        self._settle_sizes()

    def cache_spec(self):
        return StateSpec((self.n_heads, self.key_dim, self.value_dim), torch.float32)

    def scan(self, ctx, projected, at, cache):
        """Rotation, recurrence, norm and gate: columns of ``projected`` from ``at`` on -> [N, heads * e]."""
        rot, heads = self.position, self.n_heads
        qk = ops.rotate_rows(projected, at, 2 * heads, self.key_dim, rot.freq if rot is not None else None,
                             rot.rotary_dim if rot is not None else 0, rot.layout if rot is not None else 0, ctx.positions,
                             gain=rot.gain if rot is not None else 1.0, scaled_from=heads, scale=self.k_scale)
        inputs = ops.StateRows(qk, (projected, at + self.columns[1]), heads, heads, self.key_dim, self.value_dim,
                               head_decay=self._decay)
        mixed = ctx.empty((projected.shape[0], heads * self.value_dim))
        return self._recur(ctx, inputs, cache.slots, (projected, at + self.columns[2]), None, mixed)


class GatedDeltaRule(_MatrixStateMixer):
    """The gated delta rule; per head, d channels and e values, head h with q/k head floor(h / (heads / kv_heads)):

        q, k, v = silu(conv(W x))                     a short causal convolution over time per channel, n taps
        q_t <- unit(q_t) q_scale,  k_t <- unit(k_t)   unit(z) = z / sqrt(sum z^2 + 1e-6)
        beta_t = sigmoid(Wb x_t),  g_t = exp(-exp(A_log) softplus(Wa x_t + dt_bias))          one of each per head
        S <- g_t S,   u = beta_t (v_t - S^T k_t),   S <- S + k_t u^T,   o_t = S^T q_t         S_0 = 0, float32
        y_t = Wo ( o_t / sqrt(mean_e(o_t^2) + eps) * w * silu(Wg x_t) )                       w [e] shared by heads

    q, k, v, g, b and a are one stacked product.  State per request: the matrices, and the last n - 1 projected rows of
    q, k, v.  names: dict with keys q, k, v, g, b, a, o (projection names), A_log, dt_bias (full names) and norm."""

    def __init__(self, hidden_size, n_heads, n_kv_heads, key_dim, value_dim, taps, *, norm_eps, names, q_scale=None,
                 suffixes=(".weight", ".bias"), norm_suffix=".weight", conv_suffix=".conv"):
        if n_heads % n_kv_heads:
            raise ValueError(f"{n_heads} heads do not divide into {n_kv_heads} q/k heads")
        self.hidden_size, self.n_heads, self.n_kv_heads = int(hidden_size), int(n_heads), int(n_kv_heads)
        self.key_dim, self.value_dim, self.taps = int(key_dim), int(value_dim), int(taps)
        self.norm_eps = float(norm_eps)
        if self.taps < 1:
            raise ValueError("a convolution has at least one tap")
        self.q_scale = float(q_scale) if q_scale is not None else self.key_dim ** -0.5
        kw, vw = self.n_kv_heads * self.key_dim, self.n_heads * self.value_dim
        pieces = [("q", kw), ("k", kw), ("v", vw), ("g", vw), ("b", self.n_heads), ("a", self.n_heads)]
        self.projection = StackedLinear(hidden_size, [(names[key], rows) for key, rows in pieces], suffixes=suffixes)
        self.channels = 2 * kw + vw
        self.columns, at = {}, 0
        for key, rows in pieces:
            self.columns[key] = at
            at += rows
        self.conv = [Param((rows, self.taps), std=0.5) for _, rows in pieces[:3]]
        self.a_log = Param((self.n_heads,), init="normal", std=1.0)
        self.dt_bias = Param((self.n_heads,), init="normal", std=1.0)
        self.norm_weight = Param((self.value_dim,), init="norm", std=0.05)
        self._names = {names[key] + suffixes[0] + conv_suffix: param for (key, _), param in zip(pieces, self.conv)}
        self._names.update({names["A_log"]: self.a_log, names["dt_bias"]: self.dt_bias, names["norm"] + norm_suffix: self.norm_weight})
        self.out = Linear(vw, hidden_size, name=names["o"], suffixes=suffixes)
        self._taps = None

    def named_params(self):
        return dict(self._names)

    def finalize(self, device, dtype):
        super().finalize(device, dtype)
        for param in (self.a_log, self.dt_bias, self.norm_weight):       # float32 arithmetic: read as float32
            param.data = param.data.to(torch.float32).contiguous()
        self._taps = torch.cat([p.data.float() for p in self.conv], dim=0).t().contiguous()      # [taps, channels]
        for param in self.conv:
            param.data = None
        self._settle_sizes()

    def cache_spec(self):
        state = StateSpec((self.n_heads, self.key_dim, self.value_dim), torch.float32)
        return (state, StateSpec((self.taps - 1, self.channels), torch.float32)) if self.taps > 1 else state

    def scan(self, ctx, projected, at, cache):
        """Convolution, unit vectors, gates, recurrence, norm and output gate: columns of ``projected`` from ``at`` on
        -> [N, heads * e]."""
        if at:                       # the convolution's kernels read q, k and v from a row's first columns on
            projected, at = projected[:, at:at + self.projection.out_features].contiguous(), 0
        memory, rows = cache if self.taps > 1 else (cache, None)
        heads, kv_heads, d, e = self.n_heads, self.n_kv_heads, self.key_dim, self.value_dim
        qk, v, beta, log_decay = ops.delta_prepare(projected, (self.columns["b"], self.columns["a"]), self._taps,
                                                   rows.slots if rows is not None else None, self.a_log.data, self.dt_bias.data,
                                                   self.q_scale, ctx.positions, ctx.token_row, heads, kv_heads, d, e)
        if rows is not None and ctx.n_segments < ctx.n_tokens:       # some request brought more than one token
            ops.short_conv_state(projected, self.channels, rows.slots, ctx.seg_row, ctx.seg_start, ctx.seg_len, ctx.n_segments)
        inputs = ops.StateRows(qk, (v, 0), heads, kv_heads, d, e, log_decay=log_decay, beta=beta)
        mixed = ctx.empty((projected.shape[0], heads * e))
        return self._recur(ctx, inputs, memory.slots, (projected, self.columns["g"]), self.norm_weight.data, mixed)
