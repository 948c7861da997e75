"""A decoder as data: blocks, and the order in which they run.

`blocks` are the distinct layers (each with weights of its own).  `schedule`
is the list of runs: which block runs, which cache layer it uses and whether it
writes it.  A block may be named twice (its weights run twice, each run with a
cache layer of its own unless told otherwise), and a run may read the cache
layer that another run wrote (write_cache=False).  Cache layers are numbered
0..num_caches-1; each gets what its mixer's cache_spec() asks for.

A mixer may need a fixed-size state BESIDE its pages (the memory of a short
convolution in front of an attention): it says so with state_spec(), and its
run names a second cache layer (`state`) that holds it; the mixer then sees
one view with both.  A token input with state_spec() (the token before a
step's first one) gets a cache layer of its own behind all others.

A run may name a part that changes the residual stream right before its block (`before`: what a pass over looped layers begins
with).  Such a part sees the embedding output once, right after it is made (remember), and is then called before its runs.
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import List, Optional, Sequence

import torch

from ..cache.manager import CacheSpec
from ..parts.base import Block, LogitsOutput, Norm, Part, PositionEncoding, StepContext, TokenInput


@dataclass(frozen=True)
class LayerRun:
    block: int                  # index into DecoderModel.blocks
    cache: int                  # cache layer this run uses
    write_cache: bool = True    # False: read what another run of the step wrote
    state: int = -1             # cache layer of the fixed-size state the mixer keeps beside its pages (-1: none)
    before: Optional[Part] = None       # changes the residual rows ahead of the block: before.forward(x, ctx, at_embedding)


class DecoderModel:
    def __init__(self, *, embedding: TokenInput, blocks: Sequence[Block], schedule: Sequence[LayerRun], final_norm: Norm,
                 lm_head: LogitsOutput, position: Optional[PositionEncoding], dtype: torch.dtype, vocab_size: int,
                 max_positions: int, config=None, collect: Optional[Part] = None):
        # collect: for a residual stream of another form than one float32 row a token (several rows joined by
        # hyper-connections): collect.forward(x, ctx) -> float32 [T, hidden], run once after the last block
        self.collect = collect
        self.embedding, self.blocks, self.schedule = embedding, list(blocks), list(schedule)
        self.final_norm, self.lm_head, self.position = final_norm, lm_head, position
        self.dtype, self.vocab_size, self.max_positions, self.config = dtype, vocab_size, max_positions, config
        n_caches = 1 + max((max(r.cache, r.state) for r in self.schedule), default=-1)
        specs: List[CacheSpec] = [None] * n_caches
        writers = [0] * n_caches
        for run in self.schedule:
            mixer = self.blocks[run.block].mixer
            spec = mixer.cache_spec()
            if specs[run.cache] is not None and specs[run.cache] != spec:
                raise ValueError(f"cache layer {run.cache} is used by mixers with different needs")
            specs[run.cache] = spec
            writers[run.cache] += bool(run.write_cache)
            beside = mixer.state_spec() if hasattr(mixer, "state_spec") else None
            if (beside is None) != (run.state < 0):
                raise ValueError("a run names a state layer exactly when its mixer keeps a state beside its pages")
            if beside is not None:
                if specs[run.state] is not None or run.state == run.cache:
                    raise ValueError(f"cache layer {run.state} holds one run's state and nothing else")
                specs[run.state] = beside
                writers[run.state] += 1
        for c, n in enumerate(writers):
            if specs[c] is not None and n != 1:
                raise ValueError(f"cache layer {c} has {n} writers in the schedule; it needs exactly one")
        self.entries: List[Part] = []                       # the parts that runs begin with, each once
        for run in self.schedule:
            if run.before is not None and all(run.before is not e for e in self.entries):
                self.entries.append(run.before)
        self._input_state = -1
        beside = embedding.state_spec() if hasattr(embedding, "state_spec") else None
        if beside is not None:
            self._input_state = len(specs)
            specs.append(beside)
        self._cache_specs = specs

    def cache_specs(self) -> List[CacheSpec]:
        return list(self._cache_specs)

    def parts(self) -> List[Part]:
        return [self.embedding, *self.blocks, self.final_norm, self.lm_head] + ([self.collect] if self.collect is not None else []) + self.entries

    def step_weight_bytes(self) -> int:
        """Bytes of weights a decode step reads: every block as often as it runs, the output matrix once,
        and one embedding row per token (not counted)."""
        per_block = [b.weight_bytes() for b in self.blocks]
        entries = sum(r.before.weight_bytes() for r in self.schedule if r.before is not None)
        return entries + sum(per_block[r.block] for r in self.schedule) + self.final_norm.weight_bytes() + self.lm_head.weight_bytes()

    @property
    def capture_safe(self) -> bool:
        """Whether every part says that a captured CUDA graph replays it faithfully (Part.capture_safe)."""
        def safe(part) -> bool:
            if not getattr(part, "capture_safe", True):
                return False
            return all(safe(sub) for sub in vars(part).values() if isinstance(sub, Part))
        return all(safe(p) for p in self.parts() if p is not None) and (self.position is None or safe(self.position))

    def forward(self, ctx: StepContext, logit_rows: Optional[torch.Tensor], out: Optional[torch.Tensor] = None) -> Optional[torch.Tensor]:
        """Run the batch; float32 logits [len(logit_rows), vocab] for the flat token indices in logit_rows
        (written into `out` when given, else into a new tensor)."""
        ctx.extra["pass"] = ctx.extra.get("pass", 0) + 1        # parts that do something once a pass tell passes apart by this
        x = self.embedding.forward(ctx) if self._input_state < 0 else self.embedding.forward(ctx, ctx.caches[self._input_state].state)
        if self.position is not None:
            self.position.on_embeddings(x, ctx)
        for part in self.entries:
            part.remember(x, ctx)
        for i, run in enumerate(self.schedule):
            if run.before is not None:
                run.before.forward(x, ctx, i == 0)
            cache = ctx.caches[run.cache] if run.cache >= 0 else None
            if run.state >= 0:
                cache = replace(cache, state=ctx.caches[run.state].state)
            self.blocks[run.block].forward(x, ctx, cache, run.write_cache)
            if ctx.after_run is not None:
                ctx.after_run(i)
        if self.collect is not None:
            x = self.collect.forward(x, ctx)
        if logit_rows is None or logit_rows.shape[0] == 0:
            return None
        if self.lm_head.fuses_norm(self.final_norm, ctx, logit_rows.shape[0]):
            return self.lm_head.forward_normed(x, logit_rows, self.final_norm, ctx, out=out)
        xn = self.final_norm.forward(x, ctx, "head.xn", logit_rows)
        return self.lm_head.forward(xn, ctx, out=out)
