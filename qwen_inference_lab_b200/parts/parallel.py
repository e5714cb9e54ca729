"""Two mixers side by side: both read the same input, each output is normed over the model width with a weight of
its own, and the mixer's result is a weighted sum of the two (half the sum, by default):

    y = share * ( left(h) / rms(left(h)) * w_left + right(h) / rms(right(h)) * w_right )

The two keep their own caches: the mixer's cache spec is the tuple of theirs, its view the tuple of their views.
A pair of scales in place of ``norm_eps``, weights and share (``scales`` = (left, right)) gives the plain weighted sum
y = left_scale * left(h) + right_scale * right(h); a block that joins several branches at once takes the two unsummed
(``branches``), of either kind of pair: the kernel that joins them norms them on the way.
Inside a block that norms its branches on the way into the stream (:class:`PostNormBlock`) the two norms, the sum,
the block's own norm and the residual sum are one kernel (``kernels.ops.rms_join``), so the mixer joins the stream
itself (``joins_stream``); ``forward`` without a stream returns y in float32.
"""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import Mixer, Param


class ParallelMixers(Mixer):
    """``left`` and ``right``: two mixers whose ``forward(ctx, h, cache, out_float32=True)`` gives float32 rows.
    names: dict with keys left_out, right_out (the two output norms' weights)."""
    def __init__(self, hidden_size, left, right, *, norm_eps=None, names=None, share=0.5, norm_suffix=".weight", scales=None):
        self.hidden_size, self.left, self.right = int(hidden_size), left, right
        self.scales = None if scales is None else (float(scales[0]), float(scales[1]))
        if (self.scales is None) == (norm_eps is None):
            raise ValueError("two mixers side by side are summed through a norm each, or by a scale each")
        self._names = {}
        if self.scales is None:
            self.norm_eps, self.share = float(norm_eps), float(share)
            self.left_weight = Param((hidden_size,), init="norm", std=0.05)
            self.right_weight = Param((hidden_size,), init="norm", std=0.05)
            self._names = {names["left_out"] + norm_suffix: self.left_weight, names["right_out"] + norm_suffix: self.right_weight}
        self.joins_stream = self.scales is None
        self.graph_safe = True
        self._counts = tuple(len(spec) if isinstance(spec, tuple) else 1 for spec in (left.cache_spec(), right.cache_spec()))

    def named_params(self):
        return dict(self._names)

    def children(self):
        return [self.left, self.right]

    def finalize(self, device, dtype):
        super().finalize(device, dtype)
        if self.scales is None and self.left_weight.data.dtype != self.right_weight.data.dtype:
            self.left_weight.data, self.right_weight.data = self.left_weight.data.float(), self.right_weight.data.float()
        if self.scales is None:        # the kernel that joins branches reads their weights as float32
            self._branch_weights = tuple(w.data.float().contiguous() for w in (self.left_weight, self.right_weight))

    def cache_spec(self):
        flat = []
        for spec in (self.left.cache_spec(), self.right.cache_spec()):
            flat.extend(spec if isinstance(spec, tuple) else (spec,))
        return tuple(flat)

    def _views(self, cache):
        n_left = self._counts[0]
        left, right = cache[:n_left], cache[n_left:]
        return (left if n_left > 1 else left[0]), (right if self._counts[1] > 1 else right[0])

    def input_projections(self):
        found = []
        for part in (self.left, self.right):
            found += part.input_projections() if hasattr(part, "input_projections") else []
        return found

    def branches(self, ctx, x, cache, joint=None):
        """[(left's float32 rows, its scale), (right's, its scale)]; with a third entry each, the weight of the norm that the
        rows still want (``norm_eps``), of a pair that is summed through norms."""
        views = self._views(cache)
        how = {} if joint is None else dict(joint=joint)
        found = [part.forward(ctx, x, view, out_float32=True, **how) for part, view in zip((self.left, self.right), views)]
        if self.scales is not None:
            return list(zip(found, self.scales))
        return [(rows, self.share, weight) for rows, weight in zip(found, self._branch_weights)]

    def forward(self, ctx, x, cache, stream=None, norm_weight=None, mult=1.0, out_float32=True, rows=None):
        """x [N, hidden] -> y float32 [N, hidden]; with ``stream`` (the residual stream, updated in place and
        returned): stream += mult * rms(y) * norm_weight, and ``rows`` (bfloat16, optional) receives the stream's
        new values rounded."""
        if self.scales is not None:
            if stream is not None:
                raise ValueError("a pair that is summed by scales gives its branches to the block")
            return ops.branch_join(torch.zeros(x.shape, dtype=torch.float32, device=x.device), self.branches(ctx, x, cache))
        left_view, right_view = self._views(cache)
        a = self.left.forward(ctx, x, left_view, out_float32=True)
        b = self.right.forward(ctx, x, right_view, out_float32=True)
        if stream is None:
            # y itself: each normed branch times its share, added into zeros
            stream = torch.zeros_like(a)
            for branch, weight in ((a, self.left_weight.data), (b, self.right_weight.data)):
                ops.rms_join(stream, branch, weight, self.norm_eps, self.share)
            return stream
        if norm_weight.dtype != self.left_weight.data.dtype:
            norm_weight = norm_weight.to(self.left_weight.data.dtype)
        return ops.rms_join(stream, a, norm_weight, self.norm_eps, mult, b=b, weight_a=self.left_weight.data,
                            weight_b=self.right_weight.data, pre=self.share, rows=rows)
