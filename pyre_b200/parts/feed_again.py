"""A step on the residual stream that mixes the embedding's output into it again by a matrix: what a model runs before
each pass of a span of layers that it repeats."""

from __future__ import annotations

import torch

from ..kernels import lib, ops
from ..weights.specs import TensorSpec
from .base import Part, register_part


class FeedAgain(Part):
    """x = W [x; x0] with W [width, 2 width], x0 the embedding's output (the stream before the first layer).

    W splits into its two halves: W_b x0 is the same in every pass, so ``begin`` forms it once per step (fp32); a pass
    then reads the stream with everything pending added (one kernel that also rounds it for the product), multiplies by
    W_a, and sets the stream to the sum of both fp32 products.  The stream is never rounded."""

    graph_safe = True

    def __init__(self, dtype, device, width: int, tensor_name: str = "weight"):
        super().__init__(dtype, device)
        self.width, self.tensor_name = int(width), str(tensor_name)
        self.w_x = self.w_x0 = None

    def tensors(self):
        return {self.tensor_name: TensorSpec((self.width, 2 * self.width))}

    def load(self, tensors):
        w = tensors[self.tensor_name]
        self.w_x, self.w_x0 = w[:, :self.width].contiguous(), w[:, self.width:].contiguous()

    def kernel_libraries(self):
        return ["parallel_block", "elementwise"] + (["gemm_f32"] if self.dtype == torch.float32 else ["gemm_tc"])

    def _product(self, h, w):
        with lib.section("feed_again"):
            return ops.linear(h, w, out_dtype=torch.float32, partials_ok=True)

    def begin(self, ctx, x):
        """The embedding's output, before any layer has changed the stream ``x``."""
        h0 = ops.stream_rows(x, None, self.dtype)
        fixed = self._product(h0, self.w_x0)
        if isinstance(fixed, ops.PartialSums):
            fixed = fixed.parts[0] if fixed.n == 1 else ops.materialize(ops.PartialSums(fixed.parts, torch.float32))
        ctx.scratch[self] = (h0, fixed)

    def forward(self, ctx, x, pending, at_start: bool = False):
        """``at_start``: no layer has run yet, the stream is still the embedding's output."""
        h0, fixed = ctx.scratch[self]
        h = h0 if at_start and pending is None else ops.stream_rows(x, pending, self.dtype)
        ops.stream_set(x, fixed, self._product(h, self.w_x))
        return x, None


register_part("stream", "feed_again", FeedAgain)
