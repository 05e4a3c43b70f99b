"""Two mixers side by side: both read the same input, and their outputs are added with a factor each,

    out = left_scale * left(h) + right_scale * right(h).

Each mixer keeps its own cache entry (the left one's is the layer call's, the right one's an entry beside it), and
neither projects for itself: ONE product makes all of what both read from h, ONE product takes what both leave, laid
side by side in a row and already multiplied by its factor, through both output matrices.  A mixer that can stand here
gives ``in_matrix`` / ``out_matrix`` / ``drop_matrices`` and ``mix(ctx, rows of its share of the input product, cache, dtype,
out=..., out_scale=...)``.
"""

from __future__ import annotations

import torch

from tokasaurus_b200.kernels import ops
from tokasaurus_b200.parts.base import Mixer


def _pad_up(n: int, to: int = 8) -> int:
    return -(-n // to) * to


class ParallelMixers(Mixer):
    def __init__(self, left: Mixer, right: Mixer, left_scale: float = 1.0, right_scale: float = 1.0):
        for m in (left, right):
            if not hasattr(m, "mix") or not hasattr(m, "in_matrix"):
                raise ValueError(f"{type(m).__name__} cannot share its products with a mixer beside it")
        self.left, self.right = left, right
        self.left_scale, self.right_scale = float(left_scale), float(right_scale)
        self.w_in: torch.Tensor | None = None
        self.w_out: torch.Tensor | None = None

    @property
    def graph_safe(self) -> bool:
        return self.left.graph_safe and self.right.graph_safe

    def inner_mixers(self):
        return (self.left, self.right)

    def weight_specs(self):
        return tuple(self.left.weight_specs()) + tuple(self.right.weight_specs())

    def kernel_modules(self, dtype):
        return tuple(self.left.kernel_modules(dtype)) + tuple(self.right.kernel_modules(dtype))

    def cache_need(self):
        return self.left.cache_need()

    def side_needs(self):
        return {"right": self.right.cache_need()}

    def bind(self, weights, rt) -> None:
        self.left.bind(weights, rt)
        self.right.bind(weights, rt)
        a, b = self.left.in_matrix(), self.right.in_matrix()
        # both shares start on rows that are a multiple of 8, so that vector loads of either find their alignment
        n_left, n_right = _pad_up(a.shape[0]), _pad_up(b.shape[0])
        self.in_rows = (a.shape[0], n_left, b.shape[0])
        self.w_in = torch.zeros((n_left + n_right, a.shape[1]), dtype=a.dtype, device=a.device)
        self.w_in[:a.shape[0]] = a
        self.w_in[n_left:n_left + b.shape[0]] = b
        c, d = self.left.out_matrix(), self.right.out_matrix()
        o_left = _pad_up(c.shape[1])
        self.out_at = (c.shape[1], o_left, d.shape[1])
        width = o_left + _pad_up(d.shape[1])
        self.out_padded = width != c.shape[1] + d.shape[1]
        self.w_out = torch.zeros((c.shape[0], width), dtype=c.dtype, device=c.device)
        self.w_out[:, :c.shape[1]] = c
        self.w_out[:, o_left:o_left + d.shape[1]] = d
        self.left.drop_matrices()
        self.right.drop_matrices()

    def forward(self, ctx, h, cache, out_rows=None, side=None):
        T = h.shape[0]
        proj = ops.linear(h, self.w_in, out_dtype=torch.float32)
        n, at, m = self.in_rows
        # (columns between the shares meet zeros of the matrix, but must be numbers themselves)
        make = torch.zeros if self.out_padded else torch.empty
        both = make((T, self.w_out.shape[1]), dtype=h.dtype, device=h.device)
        c, o_at, d = self.out_at
        self.left.mix(ctx, proj[:, :n], cache, h.dtype, out=both[:, :c], out_scale=self.left_scale)
        self.right.mix(ctx, proj[:, at:at + m], side["right"], h.dtype, out=both[:, o_at:o_at + d], out_scale=self.right_scale)
        if out_rows is not None:
            cut = torch.empty((out_rows.numel(), both.shape[1]), dtype=both.dtype, device=both.device)
            ops.gather_rows(both, out_rows, cut)
            both = cut
        return ops.linear_out_f32(both, self.w_out, ctx.status)
