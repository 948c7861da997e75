"""Grouped-query attention with a rotation of part of each head and, each of them optional, biases, norms of queries and keys, values of their
own size or taken from the projected keys, a window, a gate a head.

With H query heads, G key-value heads (query head h reads key-value head h // (H / G)), keys of size dim and values of size vdim:

    q, k, v = W_q x + b_q, W_k x + b_k, W_v x + b_v        with v_from_k there is no W_v: v = k as it is here
    q, k    each head / rms * weight (norms), then its first `rot_dims` values turned in pairs (i, i + rot_dims / 2), or (2i, 2i + 1) with
            `neighbours`, by position * f_i
    o_h(i)  = sum_j softmax_j(scale q_h(i) . k(j)) v(j)    over the keys j <= i, with a window the last `window` of them
    o_h(i)  times sigmoid((W_g x)_h)                       with a gate
    out     = W_o [heads side by side]

The projections, the gate's among them, are one product with float32 results, so biases, norms, rotation and the gate see unrounded sums; q and the
cached k, v are in the compute dtype.  The gate is applied where the attention kernels write their outputs.  The frequencies come from the host as float32, angles are float32 position times float32 frequency with accurate cos and sin:
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
                 b_in: Optional[torch.Tensor] = None, freq: Optional[torch.Tensor] = None, rot_dims: int = 0, window: int = 0, eps: float = -1.0,
                 q_norm: Optional[torch.Tensor] = None, k_norm: Optional[torch.Tensor] = None, neighbours: bool = False, v_from_k: bool = False,
                 gate: bool = False):
        """w_in: W_q | W_k | W_v | W_g stacked by rows ([H dim + G dim + G vdim + H, hidden], compute dtype; no W_v with v_from_k, no W_g without
        gate); b_in float32 over the rows of W_q | W_k | W_v or None; freq float32 [rot_dims / 2]; q_norm, k_norm [dim] (one weight for all heads)."""
        H, G = num_heads, num_kv_heads
        self.cols = H * dim + G * dim + (0 if v_from_k else G * vdim)           # the columns in front of the gate's
        if H % G or w_in.shape != (self.cols + (H if gate else 0), hidden) or w_out.shape != (hidden, H * vdim):
            raise ValueError("the attention's weights do not fit the head counts")
        if v_from_k and vdim != dim:
            raise ValueError("values that are the projected keys have the keys' size")
        if (q_norm is None) != (k_norm is None) or (q_norm is not None and (q_norm.shape != (dim,) or k_norm.shape != (dim,) or eps < 0)):
            raise ValueError("the queries' and keys' norm weights come together, have the keys' size and an eps")
        if b_in is not None and b_in.shape != (self.cols,):
            raise ValueError("the projections' bias does not fit their rows")
        if rot_dims % 2 or rot_dims > dim or (rot_dims and (freq is None or freq.shape != (rot_dims // 2,))):
            raise ValueError("the rotation does not fit the heads")
        if gate and w_in.shape[0] % 4:          # the product's rows end on 16 bytes whatever the number of gates
            w_in = torch.cat([w_in, torch.zeros(4 - w_in.shape[0] % 4, hidden, dtype=w_in.dtype, device=w_in.device)], dim=0)
        super().__init__(w_in, w_out)
        self.hidden, self.H, self.G, self.dim, self.vdim, self.scale = hidden, H, G, dim, vdim, float(scale)
        self.rot_dims, self.window = int(rot_dims), int(window)
        f32 = lambda t: None if t is None else t.to(torch.float32).contiguous()
        self.b_in, self.freq, self.q_norm, self.k_norm = f32(b_in), f32(freq), f32(q_norm), f32(k_norm)
        self.eps = float(eps) if q_norm is not None else -1.0
        self.neighbours, self.v_from_k, self.gate = bool(neighbours), bool(v_from_k), bool(gate)

    def vectors(self):
        return [t for t in (self.b_in, self.q_norm, self.k_norm) if t is not None]

    def cache_spec(self):
        return KVSpec(self.G, self.dim, self.window, 0 if self.vdim == self.dim else self.vdim)

    def mix(self, proj: torch.Tensor, off: int, ctx: StepContext, cache: LayerCacheView, out: torch.Tensor, mult: float = 1.0) -> None:
        T, H, G = ctx.num_tokens, self.H, self.G
        meta = ctx.groups[cache.group]
        ps = ops._page_size_of(cache.pages, G, self.dim, self.vdim)
        q = ops.mixed_attn_prepare(proj, ctx.positions, meta.slot_mapping, self.q_norm, self.k_norm, self.eps, self.freq, self.rot_dims, None,
                                   ctx.workspace.rows("ratt.q", T, H * self.dim, ctx.dtype), cache.pages, H, G, self.dim, self.vdim, ps,
                                   bias=self.b_in, v_mult=mult, off=off, neighbours=self.neighbours, v_from_k=self.v_from_k)
        gate = proj[:, off + self.cols:off + self.cols + H] if self.gate else None
        ops.attention_biased(q, cache.pages, meta, ctx, out, H, G, self.dim, self.vdim, ps, self.scale, self.window, gate=gate)
