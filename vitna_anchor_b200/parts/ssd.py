"""The state-space mixer (structured state-space duality): a recurrent mixer whose state per head is a matrix with ONE decay a head and token.

With H heads of P values, G groups of N state rows (head h reads group h // (H / G)) and a short causal convolution of `taps` weights a channel:

    [z | x | B | C | dt] = W_in h                     z, x: H P;  B, C: G N;  dt: H
    x, B, C <- silu(conv(x, B, C) + conv_b)
    dt <- softplus(dt + dt_bias);   S_t = exp(-exp(A_log) dt) S_(t-1) + dt B_t x_t^T;   y_t = S_t^T C_t + D x_t        per head; S starts at zero
    out = W_o (y silu(z) / rms * w)                   the root mean square in `norm_parts` equal parts of the H P values

The projection leaves float32; step sizes, decays, the state and the norm are float32; the convolution's results are in the compute dtype.
A request's state (S of every head and the last taps - 1 inputs of the convolution) lives in its state slot.  Prompts in bfloat16 run in
chunks on the tensor cores, single decoded tokens in one launch, float32 and state sizes the chunks do not take token after token.  All
launches depend on the step's counts and device arrays alone.
"""
from __future__ import annotations

import torch

from .. import ops
from ..cache.manager import LayerCacheView, StateSpec
from .base import StepContext
from .parallel import SplitMixer


class StateSpaceMixer(SplitMixer):
    def __init__(self, hidden: int, num_heads: int, groups: int, state: int, vdim: int, taps: int, w_in: torch.Tensor, conv: torch.Tensor, conv_b,
                 dt_bias: torch.Tensor, a_log: torch.Tensor, D: torch.Tensor, norm_weight: torch.Tensor, norm_parts: int, w_out: torch.Tensor, eps: float):
        """w_in [2 H P + 2 G N + H, hidden] in the order above (compute dtype); conv float32 [H P + 2 G N, taps], the last column the current
        token's; conv_b [H P + 2 G N] or None."""
        H, G, N, P = num_heads, groups, state, vdim
        if H % G:
            raise ValueError("heads do not divide into groups")
        inner, C = H * P, H * P + 2 * G * N
        if w_in.shape != (inner + C + H, hidden) or w_out.shape != (hidden, inner) or conv.shape != (C, taps) or (conv_b is not None and conv_b.shape != (C,)):
            raise ValueError("the state-space mixer's weights do not fit the head counts")
        if any(v.shape != (H,) for v in (dt_bias, a_log, D)) or norm_weight.shape != (inner,) or norm_parts < 1 or inner % norm_parts:
            raise ValueError("the state-space mixer's vectors do not fit the head counts")
        if N > ops.ssd_max_state() or taps > ops.ssd_max_taps():
            raise ValueError(f"the recurrence takes up to {ops.ssd_max_state()} rows of a state and a convolution of up to {ops.ssd_max_taps()} taps")
        super().__init__(w_in, w_out)
        self.hidden, self.H, self.G, self.N, self.P, self.taps, self.norm_parts, self.eps = hidden, H, G, N, P, int(taps), int(norm_parts), float(eps)
        f32 = lambda t: None if t is None else t.to(torch.float32).contiguous()
        self.conv, self.conv_b, self.dt_bias, self.a_log, self.D, self.norm_weight = (f32(t) for t in (conv, conv_b, dt_bias, a_log, D, norm_weight))

    def vectors(self):
        return [t for t in (self.conv, self.conv_b, self.dt_bias, self.a_log, self.D, self.norm_weight) if t is not None]

    def cache_spec(self):
        return StateSpec((ops.ssd_state_floats(self.H, self.G, self.N, self.P, self.taps),), torch.float32)

    def mix(self, proj: torch.Tensor, off: int, ctx: StepContext, cache: LayerCacheView, out: torch.Tensor, mult: float = 1.0) -> None:
        T, ws, H, G, N, P = ctx.num_tokens, ctx.workspace, self.H, self.G, self.N, self.P
        scratch = None
        if ctx.dtype == torch.bfloat16 and not ctx.decode_only:
            scratch = ws.flat(f"ssd.chunks/{H}/{N}/{P}", ops.ssd_chunked_scratch_bytes(ws.max_tokens, ws.max_segments, H, N, P), torch.uint8)
        ops.ssd(proj, off, self.conv, self.conv_b, self.dt_bias, self.a_log, self.D, self.norm_weight, self.eps, self.norm_parts, mult, ctx, cache.state,
                ws.rows("ssd.xbc", T, H * P + 2 * G * N, ctx.dtype), ws.rows("ssd.gates", T, 2 * H, torch.float32),
                ws.rows("ssd.y", T, H * P, torch.float32), out, H, G, N, P, self.taps, chunk_scratch=scratch)
