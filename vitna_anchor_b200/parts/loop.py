"""What a pass over looped layers begins with: x <- W_in [x | x0], x0 the embedding output.

Used as LayerRun.before of a pass's first run.  The two halves of the product's input lie side by side in one buffer in the compute dtype;
the right half is written once, right after the embedding (remember), and stays for every pass of the step; a pass that begins at the
embedding itself finds the left half written too.
"""
from __future__ import annotations

import torch

from .. import ops
from .base import Part, StepContext


class PassInput(Part):
    def __init__(self, hidden: int, w_in: torch.Tensor):
        if w_in.shape != (hidden, 2 * hidden):
            raise ValueError("the matrix in front of a pass is not [width, 2 width]")
        self.hidden, self.w_in = hidden, w_in.contiguous()

    def tensors(self):
        return [self.w_in]

    def _buffer(self, ctx: StepContext) -> torch.Tensor:
        return ctx.workspace.rows("loop.cat", ctx.num_tokens, 2 * self.hidden, ctx.dtype)

    def remember(self, x: torch.Tensor, ctx: StepContext) -> None:
        ops.pass_input(x, self._buffer(ctx), True, True)

    def forward(self, x: torch.Tensor, ctx: StepContext, at_embedding: bool = False) -> None:
        """at_embedding: x is still what remember() saw."""
        cat = self._buffer(ctx)
        if not at_embedding:
            ops.pass_input(x, cat, True, False)
        ops.linear(cat, self.w_in, x, ops.LINEAR_F32)
