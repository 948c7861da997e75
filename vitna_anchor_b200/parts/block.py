"""Pre-norm residual block: x += mixer(norm1(x)); x += feed_forward(norm2(x))
(engine/src/model.c:906-972).

Output-norm residual block: x += m * norm1(mixer(x)); x += m * norm2(feed_forward(x)): the sublayers read the residual
stream as it is and the norm sits on what they give.

Sandwich-norm residual block: x += post1(mixer(pre1(x))); x += post2(feed_forward(pre2(x))), the four norms layer norms with weight
and bias.

Scaled residual block: x += c1 . mixer(norm1(x)); x += c2 . feed_forward(norm2(x)), c1 and c2 a number for every value of the row; then, if the layer has
one, an input from the token itself."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import ops

from ..cache.manager import LayerCacheView
from .base import Block, FeedForward, Mixer, Norm, Part, StepContext


class PreNormBlock(Block):
    def __init__(self, mixer_norm: Norm, mixer: Mixer, ffn_norm: Optional[Norm] = None, ffn: Optional[FeedForward] = None):
        """A layer without a feed-forward is the mixer's half alone."""
        if (ffn is None) != (ffn_norm is None):
            raise ValueError("a feed-forward and its norm come together")
        self.mixer_norm, self.mixer, self.ffn_norm, self.ffn = mixer_norm, mixer, ffn_norm, ffn

    def tensors(self):
        return [t for p in (self.mixer_norm, self.mixer, self.ffn_norm, self.ffn) if p is not None for t in p.tensors()]

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: Optional[LayerCacheView], write_cache: bool = True) -> None:
        if self.mixer.fuses_norm(self.mixer_norm, ctx):
            self.mixer.forward(x, ctx, cache, x, write_cache, norm=self.mixer_norm)
        else:
            self.mixer.forward(self.mixer_norm.forward(x, ctx, "block.xn"), ctx, cache, x, write_cache)
        if self.ffn is None:
            return
        if self.ffn.fuses_norm(self.ffn_norm, ctx):
            self.ffn.forward(x, ctx, x, norm=self.ffn_norm)
        else:
            self.ffn.forward(self.ffn_norm.forward(x, ctx, "block.xn"), ctx, x)


class OutputNormBlock(Block):
    """x <- x + mult * norm(sublayer(x)) for the mixer and then (unless absent) the feed-forward; the norms have the RMS form.

    The sublayers keep the framework's contract (they ADD their result into a float32 buffer), only that the buffer is not
    the residual stream but a zeroed row y; one kernel then norms y, scales it, sums it into the float32 residual row, zeroes
    y again and writes the next sublayer's input in the compute dtype.  The first block of a pass writes that input and zeroes
    y itself (a pass is numbered in ctx.extra["pass"] by the decoder), so a step that was given up half-way leaves nothing
    behind.  In float32 the sublayers read the residual stream itself."""

    def __init__(self, mixer_norm: Norm, mixer: Mixer, ffn_norm: Optional[Norm] = None, ffn: Optional[FeedForward] = None, mult: float = 1.0):
        if (ffn is None) != (ffn_norm is None):
            raise ValueError("a feed-forward and its norm come together")
        if mixer_norm.as_rms() is None or (ffn_norm is not None and ffn_norm.as_rms() is None):
            raise ValueError("the norms on the sublayers' outputs have the RMS form")
        self.mixer_norm, self.mixer, self.ffn_norm, self.ffn, self.mult = mixer_norm, mixer, ffn_norm, ffn, float(mult)

    def tensors(self):
        return [t for p in (self.mixer_norm, self.mixer, self.ffn_norm, self.ffn) if p is not None for t in p.tensors()]

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: Optional[LayerCacheView], write_cache: bool = True) -> None:
        T, W, ws = ctx.num_tokens, x.shape[1], ctx.workspace
        y = ws.flat(f"outnorm.y/{W}", ws.max_tokens * W, torch.float32, zero=True)[:T * W].view(T, W)
        xc = x if ctx.dtype == torch.float32 else ws.rows("outnorm.xc", T, W, ctx.dtype)
        copy = None if xc is x else xc
        this_pass = ctx.extra.get("pass", 0)
        if ctx.extra.get("outnorm.begun") != this_pass:
            ops.residual_norm_step(x, y, None, copy)
            ctx.extra["outnorm.begun"] = this_pass
        self.mixer.forward(xc, ctx, cache, y, write_cache)
        w, eps = self.mixer_norm.as_rms()
        ops.residual_norm_step(x, y, w, copy, eps, self.mult)
        if self.ffn is None:
            return
        self.ffn.forward(xc, ctx, y)
        w, eps = self.ffn_norm.as_rms()
        ops.residual_norm_step(x, y, w, copy, eps, self.mult)


class SandwichNormBlock(Block):
    """x <- x + post(sublayer(pre(x))) for the mixer and then (unless absent) the feed-forward; the four norms are layer norms with
    weight and bias (anything with .weight, .bias and .eps of the LayerNorm part).

    The sublayers do what they do everywhere in the framework (they ADD their result into a float32 buffer): the buffer is a zeroed row
    y, and ONE kernel between two sublayers norms y, sums it into the float32 residual row, zeroes y again and norms the new row for the
    next sublayer.  A block leaves its last sum pending for the next block's first kernel (two launches a layer instead of three); behind
    the last block SandwichFlush, the decoder's `collect` part, does what is left.  While something looks at the residual rows
    between the runs of the schedule (ctx.after_run), every block finishes its own sum."""

    PENDING = "sandwich.pending"

    def __init__(self, mixer_norm: Norm, mixer_post: Norm, mixer: Mixer, ffn_norm: Optional[Norm] = None, ffn_post: Optional[Norm] = None,
                 ffn: Optional[FeedForward] = None):
        if not ((ffn is None) == (ffn_norm is None) == (ffn_post is None)):
            raise ValueError("a feed-forward and its two norms come together")
        for n in (mixer_norm, mixer_post, ffn_norm, ffn_post):
            if n is not None and not (hasattr(n, "weight") and hasattr(n, "bias") and hasattr(n, "eps")):
                raise ValueError("the norms of this block are layer norms with weight and bias")
        self.mixer_norm, self.mixer_post, self.mixer, self.ffn_norm, self.ffn_post, self.ffn = mixer_norm, mixer_post, mixer, ffn_norm, ffn_post, ffn

    def tensors(self):
        return [t for p in (self.mixer_norm, self.mixer_post, self.mixer, self.ffn_norm, self.ffn_post, self.ffn) if p is not None for t in p.tensors()]

    @staticmethod
    def buffer(x: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        T, W, ws = ctx.num_tokens, x.shape[1], ctx.workspace
        return ws.flat(f"sandwich.y/{W}", ws.max_tokens * W, torch.float32, zero=True)[:T * W].view(T, W)

    @classmethod
    def take_pending(cls, ctx: StepContext):
        """The (weight, bias) of a sum that the block before left to do, if it did so in this pass."""
        left = ctx.extra.pop(cls.PENDING, None)
        return left[1] if left is not None and left[0] == ctx.extra.get("pass", 0) else None

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: Optional[LayerCacheView], write_cache: bool = True) -> None:
        T, W, ws = ctx.num_tokens, x.shape[1], ctx.workspace
        y = self.buffer(x, ctx)
        xn = ws.rows("block.xn", T, W, ctx.dtype)
        pair = lambda n: (n.weight, n.bias)
        eps = self.mixer_norm.eps
        ops.sandwich_step(x, y, self.take_pending(ctx), pair(self.mixer_norm), xn, eps)
        self.mixer.forward(xn, ctx, cache, y, write_cache)
        last = self.mixer_post
        if self.ffn is not None:
            ops.sandwich_step(x, y, pair(self.mixer_post), pair(self.ffn_norm), xn, eps)
            self.ffn.forward(xn, ctx, y)
            last = self.ffn_post
        if ctx.after_run is not None:
            ops.sandwich_step(x, y, pair(last), None, None, eps)
        else:
            ctx.extra[self.PENDING] = (ctx.extra.get("pass", 0), pair(last))


class SandwichFlush(Part):
    """Behind the last SandwichNormBlock: the sum that it left pending.  Used as a decoder's `collect` part."""

    def __init__(self, eps: float):
        self.eps = float(eps)

    def forward(self, x: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        post = SandwichNormBlock.take_pending(ctx)
        if post is not None:
            ops.sandwich_step(x, SandwichNormBlock.buffer(x, ctx), post, None, None, self.eps)
        return x


class TokenSide(Part):
    """A layer's own input from the token: e = side[token, off : off + dim], y = W_proj (gelu_tanh(W_gate x) . e), x += mult * y / rms(y) . weight.

    gate [dim, hidden], proj [hidden, dim] and side [vocab, *] in the compute dtype; weight float32 [hidden]."""

    def __init__(self, hidden: int, gate: torch.Tensor, proj: torch.Tensor, side: torch.Tensor, off: int, weight: torch.Tensor, eps: float, mult: float = 1.0):
        dim = gate.shape[0]
        if gate.shape != (dim, hidden) or proj.shape != (hidden, dim) or side.dim() != 2 or off < 0 or off + dim > side.shape[1] or weight.shape != (hidden,):
            raise ValueError("the per-layer input's weights do not fit the sizes")
        self.dim, self.off, self.eps, self.mult = dim, int(off), float(eps), float(mult)
        self.gate, self.proj, self.side = gate.contiguous(), proj.contiguous(), side.contiguous()
        self.weight = weight.to(torch.float32).contiguous()

    def tensors(self):
        return [self.gate, self.proj, self.weight]      # a piece of a row of `side` a token is read, not the table


@dataclass
class _Pending:
    """What a block left for the next block's first kernel."""
    in_pass: int
    scale: torch.Tensor
    side: Optional[TokenSide]


class ScaledResidualBlock(Block):
    """x <- x + c1 . mixer(LN1(x)), x <- x + c2 . ff(LN2(x)) (unless absent), then the layer's TokenSide (unless absent); c1 and c2 are float32 [hidden]
    (a layer's learned scale with any constant factor in it), the norms layer norms with weight and bias.

    The sublayers do what they do everywhere in the framework (they ADD their result into a float32 buffer): the buffer is a zeroed row y, and ONE
    kernel between two sublayers scales y, sums it into the float32 residual row, zeroes y and norms the new row for the next sublayer.  A block leaves
    its last sum AND its TokenSide pending for the next block's first kernel, which also adds what a pass over looped layers begins with (PassOffset); for
    few tokens the TokenSide's two products are part of that kernel too.  Behind the last block ScaledResidualFlush, the decoder's `collect`
    part, does what is left.  While something looks at the residual rows between the runs of the schedule (ctx.after_run), every block finishes its
    own sums."""

    PENDING, ADDITION = "scaled.pending", "scaled.addition"

    def __init__(self, mixer_norm: Norm, mixer: Mixer, mixer_scale: torch.Tensor, ffn_norm: Optional[Norm] = None, ffn: Optional[FeedForward] = None,
                 ffn_scale: Optional[torch.Tensor] = None, side: Optional[TokenSide] = None):
        if not ((ffn is None) == (ffn_norm is None) == (ffn_scale is None)):
            raise ValueError("a feed-forward, its norm and its scale come together")
        for n in (mixer_norm, ffn_norm):
            if n is not None and not (hasattr(n, "weight") and hasattr(n, "bias") and hasattr(n, "eps")):
                raise ValueError("the norms of this block are layer norms with weight and bias")
        for s in (mixer_scale, ffn_scale):
            if s is not None and s.shape != mixer_norm.weight.shape:
                raise ValueError("a sublayer's scale has a number for every value of the row")
        if ffn_norm is not None and ffn_norm.eps != mixer_norm.eps or side is not None and side.eps != mixer_norm.eps:
            raise ValueError("the norms of this block have one eps")
        f32 = lambda t: None if t is None else t.to(torch.float32).contiguous()
        self.mixer_norm, self.mixer, self.mixer_scale = mixer_norm, mixer, f32(mixer_scale)
        self.ffn_norm, self.ffn, self.ffn_scale, self.side = ffn_norm, ffn, f32(ffn_scale), side

    def tensors(self):
        own = [t for t in (self.mixer_scale, self.ffn_scale) if t is not None]
        return own + [t for p in (self.mixer_norm, self.mixer, self.ffn_norm, self.ffn, self.side) if p is not None for t in p.tensors()]

    def weight_bytes(self) -> int:
        parts = (self.mixer_norm, self.mixer, self.ffn_norm, self.ffn, self.side)
        return sum(p.weight_bytes() for p in parts if p is not None) + sum(4 * t.numel() for t in (self.mixer_scale, self.ffn_scale) if t is not None)

    @staticmethod
    def buffer(x: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        T, W, ws = ctx.num_tokens, x.shape[1], ctx.workspace
        return ws.flat(f"scaled.y/{W}", ws.max_tokens * W, torch.float32, zero=True)[:T * W].view(T, W)

    @classmethod
    def leave_addition(cls, ctx: StepContext, table: Optional[torch.Tensor], add: torch.Tensor) -> None:
        ctx.extra[cls.ADDITION] = (ctx.extra.get("pass", 0), table, add)

    @classmethod
    def begin(cls, x: torch.Tensor, ctx: StepContext, norm: Optional[Norm], eps: float, out: Optional[torch.Tensor]) -> None:
        """Everything that is left to do to the residual rows, and the normed rows for the next sublayer into out (norm None: not)."""
        this_pass = ctx.extra.get("pass", 0)
        left, more = ctx.extra.pop(cls.PENDING, None), ctx.extra.pop(cls.ADDITION, None)
        left = left if left is not None and left.in_pass == this_pass else None
        table, add = more[1:] if more is not None and more[0] == this_pass else (None, None)
        pair = None if norm is None else (norm.weight, norm.bias)
        y, scale, side = cls.buffer(x, ctx), None if left is None else left.scale, None if left is None else left.side
        rest = dict(table=table, ids=ctx.tokens, add=add, norm=pair, out=out, eps=eps)
        T, W = x.shape
        if side is None:
            ops.residual_step(x, y, scale, **rest)
        elif ops.token_side_takes(ctx.dtype, T, W, side.dim):
            ops.token_side(x, y, scale, side.gate, side.proj, side.side, side.off, side.weight, mult=side.mult, **rest)
        else:
            ws = ctx.workspace
            xc = x if ctx.dtype == torch.float32 else ws.rows("scaled.xc", T, W, ctx.dtype)
            ops.residual_step(x, y, scale, out=None if xc is x else xc, eps=eps)
            g = ops.linear_token_gate(xc, side.gate, side.side, side.off, ctx.tokens, ws.rows("side.a", T, side.dim, torch.float32),
                                      ws.rows("side.g", T, side.dim, ctx.dtype))
            z = ops.linear(g, side.proj, ws.rows("side.z", T, W, torch.float32), ops.LINEAR_F32)
            ops.residual_step(x, z=z, z_norm=side.weight, mult=side.mult, **rest)

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: Optional[LayerCacheView], write_cache: bool = True) -> None:
        xn = ctx.workspace.rows("block.xn", ctx.num_tokens, x.shape[1], ctx.dtype)
        y, eps = self.buffer(x, ctx), self.mixer_norm.eps
        self.begin(x, ctx, self.mixer_norm, eps, xn)
        self.mixer.forward(xn, ctx, cache, y, write_cache)
        last = self.mixer_scale
        if self.ffn is not None:
            ops.residual_step(x, y, last, norm=(self.ffn_norm.weight, self.ffn_norm.bias), out=xn, eps=eps)
            self.ffn.forward(xn, ctx, y)
            last = self.ffn_scale
        ctx.extra[self.PENDING] = _Pending(ctx.extra.get("pass", 0), last, self.side)
        if ctx.after_run is not None:
            self.begin(x, ctx, None, eps, None)


class ScaledResidualFlush(Part):
    """Behind the last ScaledResidualBlock: what it left pending.  Used as a decoder's `collect` part."""

    def __init__(self, eps: float):
        self.eps = float(eps)

    def forward(self, x: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        if ScaledResidualBlock.PENDING in ctx.extra:
            ScaledResidualBlock.begin(x, ctx, None, self.eps, None)
        return x
