"""Two mixers whose memory is a matrix per head with a decay per key channel.

Both keep S (D x Dv per head, float32, zero before the first token) in the request's state row and
walk it with the same kernel; they differ in where a token's read-out stands and in what makes q, k, v
and the decay.

GatedLinearAttention: q = W_q x * D^(-1/2), k = W_k x, v = W_v x, and a decay
a = sigmoid(W_a2 (W_a1 x) + b)^(1/tau) per head and key channel.  Per token

    S <- diag(a) S + k v^T;   o = S^T q

Each head's o is divided by its root mean square and multiplied by one weight vector of Dv for all heads,
the heads side by side by silu(W_g x), and projected back.

TimeMixing (the RWKV form): every projection sees its own blend of a token's row and the row before it,
x + (x_before - x) * mu (zeros before the first token; the last row is part of the state).  r, k, v and the
gate come from W_r, W_k, W_v, W_g, the decay is w = exp(-exp(W_w2 tanh(W_w1 x_w) + w0)).  Per token

    o = (S + diag(u) k v^T)^T r;   S <- diag(w) S + k v^T

so the current token enters its own read-out with the bonus u and the state afterwards.  Each head's o is
divided by its root mean square; the heads side by side are multiplied by a weight of their joint size and
by silu of the gate, and projected back.

Everything after the projections is float32.  The reference has no recurrent mixer
(crates/model/src/llama.rs:185-257 is its only one).
"""
from __future__ import annotations

import torch

from ..ops import lib as ops
from .base import CacheNeed, Mixer, ParamSpec, StateNeed
from .linear import RESIDUAL, STORE_F32, linear, linear_deferred


def _draw_keep(shape, g, device, std):
    """U(1, 4): logits of a decay that keeps most of a row from token to token."""
    return 1.0 + 3.0 * torch.rand(shape, generator=g, device=device, dtype=torch.float32)


def _draw_log_rate(shape, g, device, std):
    """U(-5, 0): logarithms of decay rates between exp(-5) and 1."""
    return -5.0 * torch.rand(shape, generator=g, device=device, dtype=torch.float32)


class _HeadsMixer(Mixer):
    """A mixer that fills rows of heads (`forward_heads`) and has one output matrix after them, which an owner may
    take over (`take_output_weight`) to make the output product itself."""
    graph_safe = True

    def take_output_weight(self):
        w, self.w_o_weight = self.w_o_weight, None
        return w

    def forward(self, x, ctx, cache, residual, accumulate=True, defer=False):
        T = ctx.n_tokens
        out = ctx.buf("cdecay_out", (ctx.token_capacity, self.heads_width), self.dtype)
        self.forward_heads(x, ctx, cache, out)
        if defer and not accumulate:
            part = linear_deferred(out, self.w_o_weight, ctx, T)
            if part is not None:
                return part
        linear(out, self.w_o_weight, residual, RESIDUAL if accumulate else STORE_F32, ctx, M=T)
        return None


class GatedLinearAttention(_HeadsMixer):
    def __init__(self, width, heads, dim, vdim, tau, eps, dtype, decay_rank=None):
        """decay_rank: the inner size of the decay's pair of matrices; None: whatever the weights' file has (random
        weights are then drawn with half the key size)."""
        if not 0 < dim <= ops.RECURRENT_MAX_DIM:
            raise ValueError(f"key size {dim} is outside the kernel's limit ({ops.RECURRENT_MAX_DIM})")
        if not tau > 0:
            raise ValueError("the decay's root must be positive")
        self.width, self.H, self.D, self.Dv = width, int(heads), int(dim), int(vdim)
        self.tau, self.eps, self.dtype = float(tau), float(eps), dtype
        self._free_rank = decay_rank is None
        self.rank = int(decay_rank) if decay_rank is not None else max(1, self.D // 2)
        for n in ("q_weight", "k_weight", "v_weight", "g_weight", "a1_weight", "a2_weight", "a2_bias", "norm_weight", "o_weight"):
            setattr(self, "w_" + n, None)
        self.w_in = None

    @property
    def heads_width(self):
        return self.H * self.Dv

    def param_specs(self):
        E, H, D, Dv = self.width, self.H, self.D, self.Dv
        return {"q.weight": ParamSpec((H * D, E)), "k.weight": ParamSpec((H * D, E)), "v.weight": ParamSpec((H * Dv, E)),
                "g.weight": ParamSpec((H * Dv, E)),
                "a1.weight": ParamSpec((self.rank, E), free=(0,) if self._free_rank else ()),
                "a2.weight": ParamSpec((H * D, self.rank), free=(1,) if self._free_rank else ()),
                "a2.bias": ParamSpec((H * D,), kind="vector", init=_draw_keep),
                "norm.weight": ParamSpec((Dv,), kind="vector", init="ones_normal"),
                "o.weight": ParamSpec((E, H * Dv))}

    def finalize(self):
        self.rank = self.w_a1_weight.shape[0]
        if self.w_a2_weight.shape[1] != self.rank:
            raise ValueError("the two matrices of the decay disagree on their inner size")
        self.w_in = torch.cat([self.w_q_weight, self.w_k_weight, self.w_v_weight, self.w_g_weight, self.w_a1_weight], dim=0).contiguous()
        self.w_q_weight = self.w_k_weight = self.w_v_weight = self.w_g_weight = self.w_a1_weight = None

    def cache_need(self):
        return CacheNeed(state=StateNeed((self.H * self.D * self.Dv,), torch.float32))

    def forward_heads(self, x, ctx, cache, out, scale=1.0):
        """The gated heads side by side, times `scale`, into out [T, heads_width]: everything but the output product."""
        T, cap, H, D, Dv = ctx.n_tokens, ctx.token_capacity, self.H, self.D, self.Dv
        proj = ctx.buf("gla_proj", (cap, self.w_in.shape[0]), torch.float32)
        linear(x, self.w_in, proj, STORE_F32, ctx, M=T)
        ok, ov = H * D, 2 * H * D
        og = ov + H * Dv
        oa = og + H * Dv
        dec = ctx.buf("cdecay_dec", (cap, H * D), torch.float32)
        ops.channel_decay_gate(proj[:, oa:oa + self.rank], self.w_a2_weight, self.w_a2_bias, "sigmoid_root", T, dec, tau=self.tau)
        o = ctx.buf("cdecay_o", (cap, H * Dv), torch.float32)
        ops.channel_decay(proj[:, :ok], proj[:, ok:ov], proj[:, ov:og], dec, T, ctx, H, D, Dv, cache.state, o, out_scale=D ** -0.5)
        ops.head_gate_norm(o, proj[:, og:oa], self.w_norm_weight, self.eps, T, H, Dv, out, gate_act="silu", out_scale=scale)


class TimeMixing(_HeadsMixer):
    STREAMS = ("r", "k", "v", "g", "w")      # the projections' inputs; all but the last share one grouped product

    def __init__(self, width, heads, dim, eps, dtype, decay_rank=None):
        """decay_rank: the inner size of the decay's pair of matrices; None: whatever the weights' file has (random
        weights are then drawn with half the head size)."""
        if not 0 < dim <= ops.RECURRENT_MAX_DIM:
            raise ValueError(f"head size {dim} is outside the kernel's limit ({ops.RECURRENT_MAX_DIM})")
        self.width, self.H, self.D, self.eps, self.dtype = width, int(heads), int(dim), float(eps), dtype
        self._free_rank = decay_rank is None
        self.rank = int(decay_rank) if decay_rank is not None else max(1, self.D // 2)
        for s in self.STREAMS:
            setattr(self, "w_mu_" + s, None)
        for n in ("r_weight", "k_weight", "v_weight", "g_weight", "w1_weight", "w2_weight", "w0", "u", "norm_weight", "o_weight"):
            setattr(self, "w_" + n, None)
        self.w_mu = self.w_rkvg = None

    @property
    def heads_width(self):
        return self.H * self.D

    def param_specs(self):
        E, H, D = self.width, self.H, self.D
        out = {"mu." + s: ParamSpec((E,), kind="vector", init="uniform") for s in self.STREAMS}
        out.update({s + ".weight": ParamSpec((H * D, E)) for s in self.STREAMS[:-1]})
        out.update({"w1.weight": ParamSpec((self.rank, E), free=(0,) if self._free_rank else ()),
                    "w2.weight": ParamSpec((H * D, self.rank), free=(1,) if self._free_rank else ()),
                    "w0": ParamSpec((H * D,), kind="vector", init=_draw_log_rate), "u": ParamSpec((H, D), kind="vector", init="uniform"),
                    "norm.weight": ParamSpec((H * D,), kind="vector", init="ones_normal"), "o.weight": ParamSpec((E, H * D))})
        return out

    def finalize(self):
        self.rank = self.w_w1_weight.shape[0]
        if self.w_w2_weight.shape[1] != self.rank:
            raise ValueError("the two matrices of the decay disagree on their inner size")
        self.w_mu = torch.stack([getattr(self, "w_mu_" + s) for s in self.STREAMS]).contiguous()
        self.w_rkvg = torch.stack([getattr(self, f"w_{s}_weight") for s in self.STREAMS[:-1]]).contiguous()
        for s in self.STREAMS:
            setattr(self, "w_mu_" + s, None)
        for s in self.STREAMS[:-1]:
            setattr(self, f"w_{s}_weight", None)
        self.w_u = self.w_u.contiguous()

    def cache_need(self):
        return CacheNeed(state=StateNeed((self.H * self.D * self.D + self.width,), torch.float32))     # S, then the last token's row

    def forward_heads(self, x, ctx, cache, out, scale=1.0):
        """The gated heads side by side, times `scale`, into out [T, heads_width]: everything but the output product."""
        T, cap, H, D, E = ctx.n_tokens, ctx.token_capacity, self.H, self.D, self.width
        n, N = len(self.STREAMS), H * D
        mixed = ctx.buf("tmix_in", (n * cap, E), self.dtype)[:n * T].view(n, T, E)
        counts = ctx.buf("tmix_counts", (n - 1,), torch.int32)
        ops.token_shift_mix(x, self.w_mu, T, ctx, cache.state[:, H * D * D:], mixed, counts)
        # r, k, v and the gate: one grouped product, "expert" i being the i-th matrix with the i-th blend's T rows (in
        # float32, where the CUDA cores' plain product is the faster one, four products)
        proj = ctx.buf("tmix_proj", ((n - 1) * cap, N), torch.float32)
        if self.dtype == torch.float32:
            for i in range(n - 1):
                linear(mixed[i], self.w_rkvg[i], proj[i * T:(i + 1) * T], STORE_F32, ctx, M=T)
        else:
            ops.moe_gemm(mixed[:n - 1].view((n - 1) * T, E), self.w_rkvg, counts, (n - 1) * T, proj, N, err=ctx.err)
        low = ctx.buf("tmix_low", (cap, self.rank), torch.float32)
        linear(mixed[n - 1], self.w_w1_weight, low, STORE_F32, ctx, M=T)
        dec = ctx.buf("tmix_dec", (cap, N), torch.float32)
        ops.channel_decay_gate(low, self.w_w2_weight, self.w_w0, "exp_exp", T, dec, tanh=True)
        o = ctx.buf("tmix_o", (cap, N), torch.float32)
        r, k, v, g = (proj[i * T:(i + 1) * T] for i in range(n - 1))
        ops.channel_decay(r, k, v, dec, T, ctx, H, D, D, cache.state, o, bonus=self.w_u)
        ops.head_gate_norm(o, g, self.w_norm_weight, self.eps, T, H, D, out, gate_act="silu", out_scale=scale)
