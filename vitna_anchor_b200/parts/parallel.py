"""Two mixers side by side on the same input: out = left_scale * left(x) + right_scale * right(x).

A mixer that can stand beside another one is a SplitMixer: it says what it projects (w_in, rows) and what it gives back (w_out, columns) and
does in mix() what lies between the two products.  Alone it is product, mix(), product.  Two of them share BOTH products: their input
matrices are stacked by rows (one product with float32 results, of which each reads its own columns), and their output matrices side by
side (one product over their outputs side by side, added into the residual stream).  The scales are applied to the outputs inside
mix(), before they are rounded to the compute dtype: the stacked output matrix is the checkpoint's.

One of the two keeps pages (cache_spec is a KVSpec), the other a fixed-size state (a StateSpec), which the run of the pair names as the state
beside the pages; each sees the view with both.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from .. import ops
from ..cache.manager import KVSpec, LayerCacheView, StateSpec
from .base import Mixer, StepContext


class SplitMixer(Mixer):
    """A mixer made of an input product (w_in [rows, hidden], float32 results), mix(), and an output product (w_out [hidden, columns])."""

    def __init__(self, w_in: torch.Tensor, w_out: torch.Tensor):
        self.w_in, self.w_out = w_in.contiguous(), w_out.contiguous()
        self.out_width = w_out.shape[1]

    def vectors(self) -> List[torch.Tensor]:
        """The weights that are no part of the two products."""
        return []

    def tensors(self):
        return [t for t in (self.w_in, self.w_out) if t is not None] + self.vectors()

    def mix(self, proj: torch.Tensor, off: int, ctx: StepContext, cache: LayerCacheView, out: torch.Tensor, mult: float = 1.0) -> None:
        """From this mixer's columns of proj (float32 [T, *], at off) to out [T, out_width] in the compute dtype (its rows may lie apart), times mult."""
        raise NotImplementedError

    def forward(self, xn: torch.Tensor, ctx: StepContext, cache: LayerCacheView, residual: torch.Tensor, write_cache: bool = True, norm=None) -> None:
        if not write_cache:
            raise ValueError("this mixer writes the cache or state it reads")
        T, ws = ctx.num_tokens, ctx.workspace
        proj = ops.linear(xn, self.w_in, ws.rows("split.proj", T, self.w_in.shape[0], torch.float32), ops.LINEAR_F32)
        out = ws.rows("split.out", T, self.out_width, ctx.dtype)
        self.mix(proj, 0, ctx, cache, out)
        ops.linear(out, self.w_out, residual, ops.LINEAR_ACC_F32)


class ParallelMixer(Mixer):
    def __init__(self, left: SplitMixer, right: SplitMixer, left_scale: float = 1.0, right_scale: float = 1.0):
        if left.w_in.shape[1] != right.w_in.shape[1] or left.w_out.shape[0] != right.w_out.shape[0] or left.w_in.dtype != right.w_in.dtype:
            raise ValueError("mixers side by side read and give rows of one width and dtype")
        kinds = sorted(type(m.cache_spec()).__name__ for m in (left, right))
        if kinds != ["KVSpec", "StateSpec"]:
            raise ValueError("of two mixers side by side one keeps pages and the other a fixed-size state")
        self.left, self.right, self.left_scale, self.right_scale = left, right, float(left_scale), float(right_scale)
        self.w_in = torch.cat([left.w_in, right.w_in], dim=0).contiguous()
        self.w_out = torch.cat([left.w_out, right.w_out], dim=1).contiguous()
        self.right_off, self.widths = left.w_in.shape[0], (left.out_width, right.out_width)
        for m in (left, right):             # the stacked matrices take their place
            m.w_in = m.w_out = None

    def tensors(self):
        return [self.w_in, self.w_out] + self.left.vectors() + self.right.vectors()

    def _spec(self, kind):
        return next(s for s in (self.left.cache_spec(), self.right.cache_spec()) if isinstance(s, kind))

    def cache_spec(self):
        return self._spec(KVSpec)

    def state_spec(self):
        return self._spec(StateSpec)

    def forward(self, xn: torch.Tensor, ctx: StepContext, cache: Optional[LayerCacheView], residual: torch.Tensor, write_cache: bool = True,
                norm=None) -> None:
        if not write_cache:
            raise ValueError("mixers side by side write the cache and the state they read")
        T, ws, (wl, wr) = ctx.num_tokens, ctx.workspace, self.widths
        proj = ops.linear(xn, self.w_in, ws.rows("par.proj", T, self.w_in.shape[0], torch.float32), ops.LINEAR_F32)
        out = ws.rows("par.out", T, wl + wr, ctx.dtype)
        self.left.mix(proj, 0, ctx, cache, out[:, :wl], self.left_scale)
        self.right.mix(proj, self.right_off, ctx, cache, out[:, wl:], self.right_scale)
        ops.linear(out, self.w_out, residual, ops.LINEAR_ACC_F32)
