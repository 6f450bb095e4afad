"""Mixers side by side: several mixers read the same input and their results are added, each times a constant."""

from __future__ import annotations

import torch

from ..kernels import lib, ops
from .base import Part, PartSpec, make_part, register_part
from .stacked import StackedMixer, stack_rows


class SideBySide(Part):
    """out = sum_i scale_i * mixer_i(h) over ``branches``: a list of (name prefix, mixer PartSpec, scale).

    The branches are ``StackedMixer`` parts: all their input projections run as ONE product and all their output
    projections as another one, over the branches' rows side by side; each branch multiplies its rows by its scale (fp32,
    before they are rounded), so the second product forms the weighted sum itself.  The output biases enter once, scaled.
    At most one branch may have a paged cache and at most one a state."""

    graph_safe = True

    def __init__(self, dtype, device, branches):
        super().__init__(dtype, device)
        self.branches = []
        for prefix, spec, scale in branches:
            part = make_part("mixer", spec if isinstance(spec, PartSpec) else PartSpec(*spec), dtype, device)
            if not isinstance(part, StackedMixer):
                raise ValueError(f"{type(part).__name__} cannot stand beside other mixers: it is no StackedMixer")
            self.branches.append((str(prefix), part, float(scale)))
        for what in ("cache_spec", "state_spec"):
            if sum(getattr(part, what)() is not None for _, part, _ in self.branches) > 1:
                raise ops.UnsupportedSize(f"several mixers with a {what.split('_')[0]} side by side are not implemented")
        self.heads_width = sum(part.heads_width for _, part, _ in self.branches)
        self.w_in = self.w_o = self.b_o = None
        self.cols: list = []

    def children(self):
        return {prefix: part for prefix, part, _ in self.branches}

    def loaded(self):
        rows, at = [], 0
        self.cols = []
        for _, part, scale in self.branches:
            self.cols.append(at)
            rows.append(part.w_in)
            at += part.w_in.shape[0]
            if part.b_o is not None:
                self.b_o = part.b_o * scale if self.b_o is None else self.b_o + part.b_o * scale
        self.w_in = stack_rows(rows)
        self.w_o = torch.cat([part.w_o for _, part, _ in self.branches], dim=1).contiguous()
        for _, part, _ in self.branches:
            part.w_in = part.w_o = part.b_o = None

    def kernel_libraries(self):
        return ["blockops", "elementwise", "gemm_f32" if self.dtype == torch.float32 else "gemm_tc"]

    def _one(self, what):
        return next((s for s in (getattr(part, what)() for _, part, _ in self.branches) if s is not None), None)

    def cache_spec(self):
        return self._one("cache_spec")

    def state_spec(self):
        return self._one("state_spec")

    def forward(self, ctx, h, call):
        h = ops.materialize(h)
        with lib.section("qkv"):
            proj = ops.materialize(ops.linear(h, self.w_in))
        rows = torch.empty((h.shape[0], self.heads_width), dtype=self.dtype, device=h.device)
        at = 0
        for (_, part, scale), col in zip(self.branches, self.cols):
            part.head_rows(ctx, h, proj, col, call, out=rows, out_col=at, scale=scale)
            at += part.heads_width
        with lib.section("o"):
            y = ops.linear(rows, self.w_o, partials_ok=True)
        return y if self.b_o is None else ops.BiasedRows(y, self.b_o)


register_part("mixer", "side_by_side", SideBySide)
