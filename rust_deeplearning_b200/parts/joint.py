"""Mixers whose input and output products can be shared.

A `ContextMixer` is a mixer split into three: one product of its input (`in_matrix`), what it does with the product's rows
(`context`, which returns its results and what is still to be done with them as an `ops.ContextSide`), and one output
product (`out_matrix`, optionally with `out_bias`).  `JointProducts` runs one such mixer, or several side by side on the same
input whose results are added up with constant factors:
    rows = x [W_in1; W_in2]^T;    y = [f1 c1 | f2 c2 | 1] [W_o1 | W_o2 | f1 b1 + f2 b2]^T
so that any number of mixers costs one product before and one after, and the sum is formed in the product's float
accumulators.  The factors are applied in float by the kernel that also applies norms and gates (`ops.context_finish`).  The
biases are columns of the output matrix against a column of ones; in bfloat16 they take two columns, the rounding and what it
left, so that 16 bits of them count.

Interface of a ContextMixer: `in_matrix` [n, hidden] (n a multiple of 8, so that the next mixer's columns start on a 16-byte
boundary), `out_matrix` [hidden, m], `out_bias` (float32 [hidden]) or None, `needs()`, and
`context(rows, batch, cache, run) -> ops.ContextSide`, rows being a column slice of the shared product's rows.  As a mixer of
its own it inherits `forward`.
"""
from __future__ import annotations

from typing import Sequence

import torch

from ..kernels import ops


def stacked(*matrices: torch.Tensor) -> torch.Tensor:
    """The matrices' rows one after another, followed by zero rows up to a multiple of 8."""
    n = sum(m.shape[0] for m in matrices)
    pad = [] if n % 8 == 0 else [torch.zeros((8 - n % 8, matrices[0].shape[1]), dtype=matrices[0].dtype, device=matrices[0].device)]
    return torch.cat([*matrices, *pad], dim=0).contiguous()


class JointProducts:
    def __init__(self, mixers: Sequence["ContextMixer"], factors: Sequence[float]):
        self.mixers, self.factors = list(mixers), [float(f) for f in factors]
        self.columns, at = [], 0
        for m in self.mixers:
            self.columns.append((at, at + m.in_matrix.shape[0]))
            at += m.in_matrix.shape[0]
        self.w_in = self.mixers[0].in_matrix if len(self.mixers) == 1 else torch.cat([m.in_matrix for m in self.mixers], dim=0).contiguous()
        w = self.mixers[0].out_matrix
        parts = [m.out_matrix for m in self.mixers]
        bias = None
        for m, f in zip(self.mixers, self.factors):
            if m.out_bias is not None:
                b = m.out_bias.to(torch.float32) * f
                bias = b if bias is None else bias + b
        self.n_ones = 0
        if bias is not None:
            hi = bias.to(w.dtype)
            terms = [hi] if w.dtype is torch.float32 else [hi, (bias - hi.to(torch.float32)).to(w.dtype)]
            parts += [t.view(-1, 1) for t in terms]
            self.n_ones = len(terms)
        n = sum(p.shape[1] for p in parts)
        if n % 8:
            parts.append(torch.zeros((w.shape[0], 8 - n % 8), dtype=w.dtype, device=w.device))
        self.w_out = torch.cat(parts, dim=1).contiguous() if len(parts) > 1 else w
        self.width = self.w_out.shape[1]
        for m in self.mixers:          # the shared matrices hold their values now
            m.in_matrix = m.out_matrix = None

    def forward(self, x, batch, caches, run: int, sink=None):
        rows = ops.linear(x, self.w_in)
        sides = []
        for m, f, (a, b), cache in zip(self.mixers, self.factors, self.columns, caches):
            side = m.context(rows[:, a:b], batch, cache, run)
            sides.append(side._replace(factor=side.factor * f))
        return ops.linear_branch(ops.context_finish(sides, self.width, self.n_ones, rows.dtype), self.w_out, sink)


class ContextMixer:
    in_matrix = out_matrix = out_bias = None
    takes_deferred_rows = True     # x goes into one product and nowhere else
    delivers_branch = True         # the output product may deliver the result through a stream's sink
    _products = None

    def context(self, rows, batch, cache, run: int) -> ops.ContextSide:
        raise NotImplementedError

    def forward(self, x, batch, cache, run: int, sink=None):
        if self._products is None:
            self._products = JointProducts([self], [1.0])
        return self._products.forward(x, batch, [cache], run, sink)
