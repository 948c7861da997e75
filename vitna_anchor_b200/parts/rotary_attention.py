"""Grouped-query attention with biases, a rotation of part of each head, values of their own size and, optionally, a window.

With H query heads, G key-value heads (query head h reads key-value head h // (H / G)), keys of size dim and values of size vdim:

    q, k, v = W_q x + b_q, W_k x + b_k, W_v x + b_v        the first `rot_dims` values of every query and key head turned in pairs
                                                           (i, i + rot_dims / 2) by position * f_i
    o_h(i)  = sum_j softmax_j(scale q_h(i) . k(j)) v(j)    over the keys j <= i, with a window the last `window` of them
    out     = W_o [heads side by side]

The three projections are one product with float32 results, so biases and rotation see unrounded sums; q and the cached k, v are in the
compute dtype.  The frequencies come from the host as float32, angles are float32 position times float32 frequency with accurate cos and sin:
nothing is a table over positions.  A factor on the output (see ParallelMixer) rides on the values before they are cached.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..cache.manager import KVSpec, LayerCacheView
from .base import StepContext
from .parallel import SplitMixer


class RotaryAttention(SplitMixer):
    def __init__(self, hidden: int, num_heads: int, num_kv_heads: int, dim: int, vdim: int, scale: float, w_in: torch.Tensor, w_out: torch.Tensor,
                 b_in: Optional[torch.Tensor] = None, freq: Optional[torch.Tensor] = None, rot_dims: int = 0, window: int = 0):
        """w_in: W_q | W_k | W_v stacked by rows ([H dim + G dim + G vdim, hidden], compute dtype); b_in float32 over the same rows or None;
        freq float32 [rot_dims / 2]."""
        H, G = num_heads, num_kv_heads
        if H % G or w_in.shape != (H * dim + G * dim + G * vdim, hidden) or w_out.shape != (hidden, H * vdim):
            raise ValueError("the attention's weights do not fit the head counts")
        if b_in is not None and b_in.shape != (w_in.shape[0],):
            raise ValueError("the projections' bias does not fit their rows")
        if rot_dims % 2 or rot_dims > dim or (rot_dims and (freq is None or freq.shape != (rot_dims // 2,))):
            raise ValueError("the rotation does not fit the heads")
        super().__init__(w_in, w_out)
        self.hidden, self.H, self.G, self.dim, self.vdim, self.scale = hidden, H, G, dim, vdim, float(scale)
        self.rot_dims, self.window = int(rot_dims), int(window)
        f32 = lambda t: None if t is None else t.to(torch.float32).contiguous()
        self.b_in, self.freq = f32(b_in), f32(freq)

    def vectors(self):
        return [] if self.b_in is None else [self.b_in]

    def cache_spec(self):
        return KVSpec(self.G, self.dim, self.window, 0 if self.vdim == self.dim else self.vdim)

    def mix(self, proj: torch.Tensor, off: int, ctx: StepContext, cache: LayerCacheView, out: torch.Tensor, mult: float = 1.0) -> None:
        T, H, G = ctx.num_tokens, self.H, self.G
        meta = ctx.groups[cache.group]
        ps = ops._page_size_of(cache.pages, G, self.dim, self.vdim)
        q = ops.mixed_attn_prepare(proj, ctx.positions, meta.slot_mapping, None, None, -1.0, self.freq, self.rot_dims, None,
                                   ctx.workspace.rows("ratt.q", T, H * self.dim, ctx.dtype), cache.pages, H, G, self.dim, self.vdim, ps,
                                   bias=self.b_in, v_mult=mult, off=off)
        ops.attention_biased(q, cache.pages, meta, ctx, out, H, G, self.dim, self.vdim, ps, self.scale, self.window)
