"""Two mixers side by side: both read the same rows.

ParallelMixer: each result is RMS-normed over the width with a plain weight of its own, and the mixer's
result is half their sum,

    y = (rms(left(x)) * w_left + rms(right(x)) * w_right) / 2,    rms(v) = v / sqrt(mean(v^2) + eps).

ScaledPairMixer: the result is the sum with two fixed factors, y = s_left * left(x) + s_right * right(x).  Both
mixers end in an output matrix, so the pair lays their heads' rows side by side, each already multiplied by
its factor, and one product with the two matrices side by side makes the sum (and adds it to the residual).

The two may keep different things per request (one pages, the other a state row): the part asks the
cache for both and hands each mixer the same `LayerCache`.  The reference has one mixer per layer
(crates/model/src/llama.rs:185-257).
"""
from __future__ import annotations

import torch

from ..ops import lib as ops
from .base import CacheNeed, Mixer, ParamSpec
from .linear import RESIDUAL, STORE_F32, linear, linear_deferred


# Up to this many tokens in a step the right mixer runs on a second stream beside the left one.
SIDE_STREAM_MAX_TOKENS = 64


class _Pair(Mixer):
    graph_safe = True

    def __init__(self, left: Mixer, right: Mixer, names):
        self.left, self.right, self._names = left, right, names

    def children(self):
        return [(self._names[0], self.left), (self._names[1], self.right)]

    def cache_need(self):
        a, b = self.left.cache_need(), self.right.cache_need()
        if (a.paged is not None and b.paged is not None) or (a.state is not None and b.state is not None):
            raise ValueError("the two mixers of a parallel pair want the same kind of cache")
        return CacheNeed(paged=a.paged or b.paged, state=a.state or b.state)

    def plan(self, ctx, cache):
        self.left.plan(ctx, cache)
        self.right.plan(ctx, cache)

    @staticmethod
    def both(ctx, run_left, run_right):
        """Runs the two, the right one on a second stream in steps of a few tokens: the two meet only in the sum, and there
        every kernel of a chain waits for the one before it far longer than it computes (products on the second stream use the
        second lane's workspace; the two keep different things of the cache and use scratch buffers of their own)."""
        ctx.flush_residual()
        if ctx.n_tokens <= SIDE_STREAM_MAX_TOKENS and not ops.profiling() and str(ctx.device) != "cpu":
            side, fork, join = ctx.side_stream()
            main = torch.cuda.current_stream()
            fork.record(main)
            side.wait_event(fork)
            ctx.lane = 1
            try:
                with torch.cuda.stream(side):
                    run_right()
                    ctx.flush_residual()
                    join.record(side)
            finally:
                ctx.lane = 0
            run_left()
            ctx.flush_residual()
            main.wait_event(join)
        else:
            run_left()
            ctx.flush_residual()
            run_right()
            ctx.flush_residual()


class ParallelMixer(_Pair):
    def __init__(self, width, left: Mixer, right: Mixer, eps, names=("left.", "right.")):
        super().__init__(left, right, names)
        self.width, self.eps = width, float(eps)
        self.w_left_out = self.w_right_out = None

    def param_specs(self):
        return {"left_out": ParamSpec((self.width,), kind="vector", init="ones_normal"),
                "right_out": ParamSpec((self.width,), kind="vector", init="ones_normal")}

    def forward(self, x, ctx, cache, residual, accumulate=True, defer=False):
        if accumulate:
            raise ValueError("a parallel pair hands its result to a block that norms it")
        cap, E = ctx.token_capacity, self.width
        ya = ctx.buf("pair_left", (cap, E), torch.float32)
        yb = ctx.buf("pair_right", (cap, E), torch.float32)
        self.both(ctx, lambda: self.left.forward(x, ctx, cache, ya, accumulate=False),
                  lambda: self.right.forward(x, ctx, cache, yb, accumulate=False))
        ops.dual_norm_mean(ya, yb, self.w_left_out, self.w_right_out, self.eps, residual, ctx.n_tokens)
        return None


class ScaledPairMixer(_Pair):
    """left, right: mixers with `heads_width`, `forward_heads(x, ctx, cache, out, scale)` and `take_output_weight()`."""

    def __init__(self, width, left: Mixer, right: Mixer, left_scale, right_scale, dtype, names=("left.", "right.")):
        super().__init__(left, right, names)
        self.width, self.dtype = width, dtype
        self.left_scale, self.right_scale = float(left_scale), float(right_scale)
        self.w_out = None

    def finalize(self):
        super().finalize()
        self.w_out = torch.cat([self.left.take_output_weight(), self.right.take_output_weight()], dim=1).contiguous()

    def forward(self, x, ctx, cache, residual, accumulate=True, defer=False):
        n = self.left.heads_width
        heads = ctx.buf("pair_heads", (ctx.token_capacity, n + self.right.heads_width), self.dtype)
        self.both(ctx, lambda: self.left.forward_heads(x, ctx, cache, heads[:, :n], self.left_scale),
                  lambda: self.right.forward_heads(x, ctx, cache, heads[:, n:], self.right_scale))
        if defer and not accumulate:
            part = linear_deferred(heads, self.w_out, ctx, ctx.n_tokens)
            if part is not None:
                return part
        linear(heads, self.w_out, residual, RESIDUAL if accumulate else STORE_F32, ctx, M=ctx.n_tokens)
        return None
