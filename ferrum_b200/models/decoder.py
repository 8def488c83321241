"""A decoder put together from parts: embedding, blocks, a run order, final norm, head.

The run order is data: `schedule` is a list of `Run(block, cache_of)`.  `block` indexes
`blocks` (naming a block twice runs it twice, each run with cache planes of its own);
`cache_of = j` lets run k read the cache that run j wrote instead of writing one; `before` names one of the
model's `entries`, parts that rework the residual rows right before that run.  The model
never looks at which architecture it is; `weight_specs` and `cache_needs` are derived from
the parts.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional

import os

import torch

from ..parts.base import CacheNeed, Part

# FERRUM_NVTX=1: every step and every run of a block is an NVTX range (for a system profiler's timeline)
NVTX = os.environ.get("FERRUM_NVTX", "0") == "1"


@dataclass(frozen=True)
class Run:
    block: int
    cache_of: Optional[int] = None      # index of an earlier run whose cache this run reads
    before: Optional[int] = None        # index into the model's `entries`: a part that runs on the residual rows first


class DecoderModel(Part):
    graph_safe = True

    def __init__(self, config, dtype, embedding, position, blocks, final_norm, head, schedule=None,
                 block_prefix="blk.{}.", names=("token_embd.", "output_norm.", "output."), shared=(), entries=()):
        """shared: (prefix, part) pairs the model owns because several blocks refer to them (a table
        that every layer reads a slice of); they only bring parameters, the blocks call them.
        entries: (prefix, part) pairs that runs of the schedule name in `before`."""
        self.config, self.dtype = config, dtype
        self.embedding, self.position, self.blocks = embedding, position, list(blocks)
        self.final_norm, self.head = final_norm, head
        self.schedule: List[Run] = list(schedule) if schedule is not None else [Run(i) for i in range(len(self.blocks))]
        self._block_prefix, self._names = block_prefix, names
        self.shared, self.entries = list(shared), list(entries)
        self.on_run = None       # debugging hook: called as on_run(k, h) after run k of the schedule with the residual rows
        for k, run in enumerate(self.schedule):
            if not 0 <= run.block < len(self.blocks):
                raise ValueError(f"schedule entry {k} names block {run.block}, which does not exist")
            if run.cache_of is not None and not (0 <= run.cache_of < k and self.schedule[run.cache_of].cache_of is None):
                raise ValueError(f"schedule entry {k} must read the cache of an earlier run that writes one")
            if run.before is not None and not 0 <= run.before < len(self.entries):
                raise ValueError(f"schedule entry {k} names entry part {run.before}, which does not exist")

    # ------------------------------------------------------------------ structure
    def children(self):
        out = [(self._names[0], self.embedding)]
        if self.position is not None:
            out.append(("position.", self.position))
        out += self.shared + self.entries
        out += [(self._block_prefix.format(i), b) for i, b in enumerate(self.blocks)]
        out += [(self._names[1], self.final_norm), (self._names[2], self.head)]
        return out

    def weight_specs(self):
        """Canonical tensor name -> (ParamSpec, owner part, local name)."""
        return {name: (spec, part, local) for name, spec, part, local in self.named_specs()}

    def cache_needs(self):
        """One CacheNeed per schedule entry: what that run's mixer keeps per request, or what its
        block says it keeps (a block with a state of its own has a `cache_need`)."""
        out = []
        for r in self.schedule:
            b = self.blocks[r.block]
            out.append(b.cache_need() if hasattr(b, "cache_need") else b.mixer.cache_need())
        return out

    def embedding_need(self):
        """What the embedding keeps per request beside the runs of the schedule (a `CacheNeed`)."""
        return self.embedding.cache_need() if hasattr(self.embedding, "cache_need") else CacheNeed()

    @property
    def n_vocab(self):
        return self.head.n_vocab

    # ------------------------------------------------------------------ the forward pass
    def plan(self, ctx, cache):
        """Lets every run's mixer build this step's host-made work lists (see `Mixer.plan`)."""
        for k, run in enumerate(self.schedule):
            self.blocks[run.block].mixer.plan(ctx, cache.layer_cache(k))

    def forward(self, ctx, cache):
        """Run the batch described by ctx; returns float32 logits [want_capacity, V] whose
        first ctx.n_want rows are valid, or None when nothing is wanted."""
        state = cache.embedding_state
        h = self.embedding.forward(ctx) if state is None else self.embedding.forward(ctx, state)
        if self.position is not None:
            self.position.on_embedding(h, ctx)
        for k, run in enumerate(self.schedule):
            if NVTX:
                torch.cuda.nvtx.range_push(f"run {k} block {run.block}")
            if run.before is not None:
                self.entries[run.before][1].forward(h, ctx)
            self.blocks[run.block].forward(h, ctx, cache.layer_cache(k))
            if self.on_run is not None:
                ctx.flush_residual()
                self.on_run(k, h)
            if NVTX:
                torch.cuda.nvtx.range_pop()
        if ctx.n_want == 0:
            ctx.drop_pending()               # nobody reads the residual stream any more
            return None
        x = self.final_norm.forward(h, ctx, rows=ctx.want_rows, n_rows=ctx.n_want, tag="final_norm")
        ctx.flush_residual()
        return self.head.forward(x, ctx, ctx.n_want)
