"""What a pass over looped layers begins with, x0 the embedding output: x <- W_in [x | x0] (PassInput), or x += x0 (or not) and x += a vector of
the pass's own (PassOffset).

Used as LayerRun.before of a pass's first run.  PassInput:  The two halves of the product's input lie side by side in one buffer in the compute dtype;
the right half is written once, right after the embedding (remember), and stays for every pass of the step; a pass that begins at the
embedding itself finds the left half written too.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from .base import Part, StepContext
from .block import ScaledResidualBlock


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


class PassOffset(Part):
    """x += E[token] (with `table`: the embedding output is the token's row of it) and x += step.

    In front of a ScaledResidualBlock (deferred=True) nothing is launched here: that block's first kernel, which walks over the residual rows
    anyway, adds both."""

    def __init__(self, hidden: int, step: torch.Tensor, table: Optional[torch.Tensor] = None, deferred: bool = False):
        if step.shape != (hidden,) or (table is not None and (table.dim() != 2 or table.shape[1] != hidden)):
            raise ValueError("what a pass adds is not of the residual stream's width")
        self.step, self.table, self.deferred = step.to(torch.float32).contiguous(), table, bool(deferred)

    def tensors(self):
        return [self.step]                  # a row a token of the table is read, not the table

    def remember(self, x: torch.Tensor, ctx: StepContext) -> None:
        """The embedding output is read from the table again."""

    def forward(self, x: torch.Tensor, ctx: StepContext, at_embedding: bool = False) -> None:
        if self.deferred:
            ScaledResidualBlock.leave_addition(ctx, self.table, self.step)
        else:
            ops.residual_step(x, table=self.table, ids=ctx.tokens, add=self.step)
