"""Matrix products ``y = x W^T (+ b) (+ residual)`` with checkpoint-layout weights.

Weights are row-major ``[out_features, in_features]`` as the reference's
``nn.Linear`` stores them (qil/model.py:32-40).  A bfloat16 weight under bfloat16
activations goes to the library GEMM, which is what the reference's engine uses
for its projections (qil/model.py:52-54,69-71: ``nn.Linear`` -> cuBLAS); every
other combination (the true 32-bit path, or a weight stored in float32 inside a
bfloat16 model) runs the engine's own float32 CUDA-core product.  Products of at
most 16 rows (decode steps) run the engine's own weight-streaming kernel instead
of the library.
"""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import Param, Part


def _library_mm_f32_out(a, weight):
    """bf16 x bf16 -> float32 product without rounding the result to bfloat16."""
    try:
        return torch.mm(a, weight.t(), out_dtype=torch.float32)
    except TypeError:
        return torch.mm(a, weight.t()).float()


class Linear(Part):
    graph_safe = True

    def __init__(self, in_features, out_features, *, name, bias=False, weight=None, suffixes=(".weight", ".bias")):
        """``weight`` may be another part's Param of the same shape (tied embeddings).  ``suffixes``: what a
        checkpoint appends to ``name`` for the weight and for the bias."""
        self.in_features, self.out_features = int(in_features), int(out_features)
        self.name, self.suffixes = name, tuple(suffixes)
        if weight is not None and weight.shape != (self.out_features, self.in_features):
            raise ValueError(f"shared weight {weight.shape} does not fit [{out_features}, {in_features}]")
        self.weight = weight if weight is not None else Param((out_features, in_features))
        self.bias = Param((out_features,), init="zeros") if bias else None

    def named_params(self):
        params = {self.name + self.suffixes[0]: self.weight}
        if self.bias is not None:
            params[self.name + self.suffixes[1]] = self.bias
        return params

    def finalize(self, device, dtype):
        if self.bias is not None and self.bias.data.dtype != self.weight.data.dtype:
            self.bias.data = self.bias.data.to(self.weight.data.dtype)   # the kernels read both as one dtype

    # The tensors the product runs with; StackedLinear overrides these.
    def _weight(self):
        return self.weight.data

    def _bias(self):
        return self.bias.data if self.bias is not None else None

    def forward(self, ctx, x, residual=None, out=None, out_float32=False, norm=None, out_scale=None, activation=None):
        """``x`` [N, in] -> [N, out]; adds ``residual`` [N, out] when given (may be ``out``).

        ``out_scale`` float32 [out]: a learned scale per output feature on the way into the residual, which is
        then updated in place: residual += out_scale * (x W^T + b).

        With ``norm`` (a Norm part) the product is of ``norm(x)``: fused into the kernel where it can be.
        A float32 ``residual`` under bfloat16 activations (a residual stream kept in float32) gives a
        float32 result: the product's float32 sums are added to it without a rounding in between.
        """
        weight, bias = self._weight(), self._bias()
        if norm is not None and norm.as_rms() is None:
            # a norm that no product kernel applies itself (float32 statistics of a float32 stream, a layer norm):
            # normed first, so that what follows is chosen by the rows the product really gets
            x, norm = norm.forward(ctx, x), None
        if activation is not None:
            # ``activation``: one of ``ops.PLAIN_ACTIVATIONS`` on the result, in the weight-streaming kernel's
            # epilogue for a decode step's rows, else by a kernel of its own
            if residual is not None or out_scale is not None or out_float32:
                raise ValueError("an activation goes with a plain product")
            if norm is None and ops.small_m_ok(x, weight):
                return ops.gemm_small_m(x, weight, bias=bias, out=out, activation=activation)
            result = self.forward(ctx, x, out=out, norm=norm)
            return ops.activation(result, activation, out=result)
        if out_scale is not None:
            if residual is None or out is not None:
                raise ValueError("an output scale goes with a residual, which is updated in place")
            if x.dtype == torch.bfloat16 and weight.dtype == torch.bfloat16:
                if norm is None and ops.small_m_ok(x, weight):
                    # a decode step's few rows: scale and residual in the weight-streaming kernel's epilogue
                    return ops.gemm_small_m(x, weight, bias=bias, residual=residual, out=residual, col_scale=out_scale,
                                            out_float32=residual.dtype == torch.float32)
                branch = self.forward(ctx, x, out_float32=residual.dtype == torch.float32, norm=norm)
                return ops.scaled_add(residual, branch, out_scale)
            if norm is not None:
                x = norm.forward(ctx, x)
            if residual.dtype != x.dtype:
                return ops.scaled_add(residual, ops.gemm_f32(x, weight, bias=bias), out_scale)
            return ops.gemm_f32(x, weight, bias=bias, residual=residual, out=residual, col_scale=out_scale)
        if residual is not None and residual.dtype == torch.float32 and x.dtype == torch.bfloat16 \
                and weight.dtype == torch.bfloat16:
            if norm is not None:
                x = norm.forward(ctx, x)
            if ops.small_m_ok(x, weight):
                return ops.gemm_small_m(x, weight, bias=bias, residual=residual, out=out, out_float32=True)
            result = _library_mm_f32_out(x, weight)
            if bias is not None:
                result += bias.float()
            ops.add_inplace(result, residual)
            if out is not None:
                out.copy_(result)
                return out
            return result
        if ops.small_m_ok(x, weight):
            # a decode step's few rows: the engine's weight-streaming kernel
            rms = norm.as_rms() if norm is not None else None
            if rms is not None and rms[0].dtype == torch.bfloat16:
                return ops.gemm_small_m(x, weight, bias=bias, residual=residual, out=out, out_float32=out_float32,
                                        norm_weight=rms[0], norm_eps=rms[1])
            if norm is not None:
                x = norm.forward(ctx, x)
            return ops.gemm_small_m(x, weight, bias=bias, residual=residual, out=out, out_float32=out_float32)
        if norm is not None:
            x = norm.forward(ctx, x)
        if x.dtype == torch.bfloat16 and weight.dtype == torch.bfloat16:
            if out_float32:
                result = _library_mm_f32_out(x, weight)
                if bias is not None:
                    result += bias.float()
                return result
            if residual is not None and bias is None:
                return torch.addmm(residual, x, weight.t(), out=out if out is not None else residual)
            if bias is not None:
                result = torch.addmm(bias, x, weight.t(), out=out)
            else:
                result = torch.mm(x, weight.t(), out=out) if out is not None else torch.mm(x, weight.t())
            if residual is not None:
                ops.add_inplace(result, residual)
            return result
        # float32 accumulate on the CUDA cores; activations keep their dtype unless float32 is asked for
        if out_float32 and x.dtype != torch.float32:
            x = ops.cast(x, torch.float32)
        return ops.gemm_f32(x, weight, bias=bias, residual=residual, out=out)


class StackedLinear(Linear):
    """Several checkpoint matrices over the same input, run as one product.

    ``pieces`` is a list of (checkpoint name, out_features); the rows are stacked in
    that order after loading (the reference keeps q/k/v and gate/up apart,
    qil/model.py:32-34,38-39; one product over the stack reads the input once).
    """

    def __init__(self, in_features, pieces, *, bias=False, suffixes=(".weight", ".bias")):
        self.in_features = int(in_features)
        self.suffixes = tuple(suffixes)
        self.pieces = [(name, int(rows)) for name, rows in pieces]
        self.out_features = sum(rows for _, rows in self.pieces)
        self.parts_w = [Param((rows, in_features)) for _, rows in self.pieces]
        self.parts_b = [Param((rows,), init="zeros") for _, rows in self.pieces] if bias else None
        self._w = None
        self._b = None

    def named_params(self):
        params = {}
        for i, (name, _) in enumerate(self.pieces):
            params[name + self.suffixes[0]] = self.parts_w[i]
            if self.parts_b is not None:
                params[name + self.suffixes[1]] = self.parts_b[i]
        return params

    def finalize(self, device, dtype):
        dtypes = {p.data.dtype for p in self.parts_w}
        common = torch.float32 if len(dtypes) > 1 else dtypes.pop()
        self._w = torch.cat([p.data.to(common) for p in self.parts_w], dim=0).contiguous()
        for p in self.parts_w:
            p.data = None
        if self.parts_b is not None:
            self._b = torch.cat([p.data.to(common) for p in self.parts_b], dim=0).contiguous()
            for p in self.parts_b:
                p.data = None

    def _weight(self):
        return self._w

    def _bias(self):
        return self._b

    def columns_of(self, ctx, x, joint=None, norm=None):
        """(buffer, first column) of this projection of ``x``: its place in the rows of a :class:`JointProjection` that
        has run already, or a product of its own."""
        if joint is not None and id(self) in joint.first_column:
            return joint.rows, joint.first_column[id(self)]
        return self.forward(ctx, x, norm=norm), 0


class JointProjection(Linear):
    """Several :class:`StackedLinear` of the same input (the first projections of sublayers that run side by side), as
    one product.  It owns no parameters: ``join`` (called once the parts are finalized) lays their stacked weights one
    below the other, each from a row that is a multiple of ``ALIGN`` on so that every part's columns start on a 16-byte
    boundary, and leaves the parts views of it: they still run by themselves as well.  Parts with biases or with
    weights of different dtypes are not joined (``forward_joint`` gives None and every part runs its own product)."""
    ALIGN = 8

    def __init__(self, projections):
        self.projections = list(projections)
        self._w = None
        self._first = {}

    def named_params(self):
        return {}

    def finalize(self, device, dtype):
        pass

    def join(self):
        weights = [p._weight() for p in self.projections]
        if len(weights) < 2 or any(p._bias() is not None for p in self.projections) or len({w.dtype for w in weights}) != 1 \
                or len({w.shape[1] for w in weights}) != 1:
            return
        at = 0
        for projection, w in zip(self.projections, weights):
            self._first[id(projection)] = at
            at += -(-w.shape[0] // self.ALIGN) * self.ALIGN
        self._w = torch.zeros((at, weights[0].shape[1]), dtype=weights[0].dtype, device=weights[0].device)
        for projection, w in zip(self.projections, weights):
            first = self._first[id(projection)]
            self._w[first:first + w.shape[0]] = w
            projection._w = self._w[first:first + w.shape[0]]
        self.out_features, self.in_features = self._w.shape

    def _weight(self):
        return self._w

    def _bias(self):
        return None

    def forward_joint(self, ctx, x):
        return None if self._w is None else JointRows(self.forward(ctx, x), self._first)


class JointRows:
    """The rows of a :class:`JointProjection` and the first column of every part's projection in them."""
    __slots__ = ("rows", "first_column")

    def __init__(self, rows, first_column):
        self.rows, self.first_column = rows, first_column
