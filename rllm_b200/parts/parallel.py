"""Two mixers side by side on the same input: out = left_scale * left(h) + right_scale * right(h), each
side's output optionally behind an RMS norm of its own (`left_norm`, `right_norm`: PartSpecs of norms).

Parameters: left, right (PartSpec of registered mixer kinds, with their own prefixes), left_scale,
right_scale, left_norm, right_norm.  Each side keeps what it needs in the cache under its own need; this part's
need is the tuple of both and its cache view the tuple of their views.

Where both sides begin with one product on h (they name its matrix: INPUT_MATRIX), the two matrices are
stacked at load and run as one product.  Where both sides end with one product (OUTPUT_MATRIX) and no norm stands
behind it, those are stacked too, along the columns they read: each side writes the rows its product would read, times its
scale, beside the other's, and one product gives the sum (into the residual stream, if the block hands it over).  ``join(h, ctx, cache, position, x, extra, mult, copy)``: the kernel that
norms and adds the two sides also adds `extra` (a feed-forward's output, or None) and joins the sum, times
mult, to the float32 stream x; `copy`, if given, takes the new x in its own type.
"""
from __future__ import annotations

import torch

from ..csrc import ops
from .base import Mixer, build_part, register_part


@register_part("mixer", "parallel")
class ParallelMixer(Mixer):
    def __init__(self, params, prefix, runtime):
        super().__init__(params, prefix, runtime)
        self.left = build_part("mixer", params["left"], runtime)
        self.right = build_part("mixer", params["right"], runtime)
        self.left_scale, self.right_scale = float(params["left_scale"]), float(params["right_scale"])
        norm = lambda key: build_part("norm", params[key], runtime) if params.get(key) else None
        self.left_norm, self.right_norm = norm("left_norm"), norm("right_norm")
        self.w_both = self.w_ends = None
        self.CAPTURE_SAFE = bool(getattr(self.left, "CAPTURE_SAFE", False) and getattr(self.right, "CAPTURE_SAFE", False))

    def _parts(self):
        return [p for p in (self.left, self.right, self.left_norm, self.right_norm) if p is not None]

    def cache_need(self):
        return (self.left.cache_need(), self.right.cache_need())

    def expected_tensors(self):
        return {k: v for p in self._parts() for k, v in p.expected_tensors().items()}

    def load(self, tensors):
        for p in self._parts():
            p.load(tensors)
        names = [getattr(s, "INPUT_MATRIX", None) for s in (self.left, self.right)]
        if all(names):
            ws = [getattr(s, n) for s, n in zip((self.left, self.right), names)]
            self.w_both = torch.cat(ws, 0)
            self.split = ws[0].shape[0]
            setattr(self.left, names[0], self.w_both[:self.split])        # the sides keep views, not copies
            setattr(self.right, names[1], self.w_both[self.split:])
        ends = [getattr(s, "OUTPUT_MATRIX", None) for s in (self.left, self.right)]
        if all(ends) and self.left_norm is None and self.right_norm is None:
            self.w_ends = torch.cat([getattr(s, n) for s, n in zip((self.left, self.right), ends)], 1).contiguous()
            for s, n in zip((self.left, self.right), ends):
                setattr(s, n, None)
            for s, f in ((self.left, self.left_scale), (self.right, self.right_scale)):
                if hasattr(s, "scaled_norm"):
                    s.scaled_norm(f)                     # made here, not inside a captured step

    def _sides(self, h, ctx, cache, position):
        rows = self._rows(h)
        return (self.left.forward(h, ctx, cache[0], position, **rows[0]),
                self.right.forward(h, ctx, cache[1], position, **rows[1]))

    def _rows(self, h):
        """Keyword arguments of the two sides: their rows of the stacked product on h, if there is one."""
        if self.w_both is None:
            return {}, {}
        rows = ops.linear(h, self.w_both, out_dtype=torch.float32)
        return {"rows": rows[:, :self.split]}, {"rows": rows[:, self.split:]}

    def join(self, h, ctx, cache, position, x, extra=None, mult=1.0, copy=None, add=True):
        a, b = self._sides(h, ctx, cache, position)
        form = lambda n: (n.weight, n.eps) if n is not None else None
        return ops.join_sum_rows(a, x, mult, add, form(self.left_norm), self.left_scale, b, form(self.right_norm),
                                 self.right_scale, extra, copy)

    def forward(self, h, ctx, cache, position=None, residual=None):
        if self.w_ends is not None:
            k = self.left.output_columns
            ends = torch.empty((h.shape[0], self.w_ends.shape[1]), dtype=self.runtime.dtype, device=h.device)
            rows = self._rows(h)
            self.left.forward(h, ctx, cache[0], position, into=ends[:, :k], factor=self.left_scale, **rows[0])
            self.right.forward(h, ctx, cache[1], position, into=ends[:, k:], factor=self.right_scale, **rows[1])
            if residual is not None:
                ops.linear(ends, self.w_ends, out=residual, accumulate=True)
                return None
            return ops.linear(ends, self.w_ends, out_dtype=torch.float32)
        if self.left_norm is None and self.right_norm is None:
            a, b = self._sides(h, ctx, cache, position)
            return ops.axpby(self.left_scale, a, self.right_scale, b, a)
        out = torch.empty(h.shape, dtype=torch.float32, device=h.device)
        return self.join(h, ctx, cache, position, out, add=False)
