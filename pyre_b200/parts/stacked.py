"""What mixers share whose projections run as one product: their own, or, side by side, those of several mixers."""

from __future__ import annotations

import torch

from ..kernels import lib, ops
from .base import Part


def stack_rows(weights) -> torch.Tensor:
    """Weights [n_i, K] below one another, padded by zero rows to a multiple of 8 rows: a token's projections then start
    on 16-byte boundaries and the product stores whole vectors."""
    rows = sum(w.shape[0] for w in weights)
    pad = -rows % 8
    if pad:
        weights = list(weights) + [torch.zeros((pad, weights[0].shape[1]), dtype=weights[0].dtype, device=weights[0].device)]
    return torch.cat(list(weights), dim=0).contiguous() if len(weights) > 1 else weights[0]


class StackedMixer(Part):
    """A mixer that is one product in, something over heads, and one product out:

        proj = h w_in^T;  rows = head_rows(proj);  out = rows w_o^T (+ b_o)

    A subclass sets ``w_in`` [n, width], ``w_o`` [width, heads_width] and ``b_o`` (fp32 [width] or None) when it loads, has
    ``heads_width``, and implements ``head_rows``: the same class then runs by itself (``forward``) or beside others under a
    part that stacks the products of several such mixers (and takes these tensors away from them)."""

    w_in = w_o = b_o = None
    heads_width = 0

    def head_rows(self, ctx, h, proj, col: int, call, out=None, out_col: int = 0, scale: float = 1.0):
        """The heads' rows times ``scale`` [T, heads_width] from the mixer's projections, which are the columns of ``proj``
        from ``col`` on; written to the columns of ``out`` from ``out_col`` on when it is given.  ``h`` is the mixer's
        input, for a map that does not run in the stacked product."""
        raise NotImplementedError

    def forward(self, ctx, h, call):
        h = ops.materialize(h)
        with lib.section("qkv"):
            proj = ops.materialize(ops.linear(h, self.w_in))
        a = self.head_rows(ctx, h, proj, 0, call)
        with lib.section("o"):
            y = ops.linear(a, self.w_o, partials_ok=True)
        return y if self.b_o is None else ops.BiasedRows(y, self.b_o)
