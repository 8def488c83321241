"""RMSNorm: x * rsqrt(mean(x^2) + eps) * w (crates/kernels/src/scalar.rs:143-156).  With
`groups` > 1 the row is cut into that many equal consecutive parts, each divided by its own root
mean square (the reference has one group).  `zero_centred`: the file stores the weight around zero and
the norm multiplies by 1 + w."""
from __future__ import annotations

import torch

from ..ops import lib as ops
from .base import Norm, ParamSpec


class RMSNorm(Norm):
    graph_safe = True

    def __init__(self, width: int, eps: float, out_dtype, groups: int = 1, zero_centred: bool = False):
        if groups < 1 or width % groups:
            raise ValueError(f"{groups} groups do not divide a width of {width}")
        self.width, self.eps, self.out_dtype, self.groups = width, float(eps), out_dtype, int(groups)
        self.zero_centred = bool(zero_centred)
        self.w_weight = None

    def param_specs(self):
        return {"weight": ParamSpec((self.width,), kind="vector", init="normal" if self.zero_centred else "ones_normal")}

    def finalize(self):
        if self.zero_centred:
            self.w_weight = 1.0 + self.w_weight          # (a float32 vector: the kernels see a plain weight)

    def forward(self, h, ctx, rows=None, n_rows=None, tag="norm"):
        """h float32 [T, width] -> compute-dtype rows; `rows` (int32) picks source rows."""
        n = n_rows if n_rows is not None else ctx.n_tokens
        cap = ctx.want_capacity if rows is not None else ctx.token_capacity
        out = ctx.buf(tag + ("_rows" if rows is not None else ""), (cap, self.width), self.out_dtype)
        if ctx.pending_experts is not None:
            ctx.flush_residual()
        if self.groups > 1:
            ctx.flush_residual()
            ops.rmsnorm(h, self.w_weight, out, self.eps, rows=rows, n_rows=n, groups=self.groups)
            return out
        if rows is None and ctx.pending_add is not None:
            p = ctx.take_pending_add(h)
            if p is not None:
                if ops.norm_scaled_add_can_norm(h, p.y if p.partials is None else None, p.w, self.w_weight, out):
                    ops.norm_scaled_add(h, p.y, p.w, p.mult, p.eps, n, partials=p.partials, norm=(self.w_weight, self.eps, out))
                    return out
                ops.norm_scaled_add(h, p.y, p.w, p.mult, p.eps, n, partials=p.partials)
        elif ctx.pending_add is not None:
            ctx.flush_residual()
        ops.rmsnorm(h, self.w_weight, out, self.eps, rows=rows, n_rows=n, partials=ctx.take_pending_residual(h))
        return out


def _alpha_init(shape, g, device, std):
    return 0.5 + 0.1 * torch.randn(shape, generator=g, device=device, dtype=torch.float32)


class DynamicTanh(Norm):
    """tanh(alpha * x) * w + b with a scalar alpha: no statistic of the row enters, so the kernel is elementwise and makes
    whatever residual sum is still open on its way (a product left in partials, or a routed feed-forward's unsummed expert
    rows).  `scale` multiplies the result (it is folded into w and b once, in float32): a model whose logits are scaled
    by a constant gives it to its last norm, since the head is linear.  The reference's norm is `RMSNorm`'s."""
    graph_safe = True

    def __init__(self, width: int, out_dtype, scale: float = 1.0):
        self.width, self.out_dtype, self.scale = width, out_dtype, float(scale)
        self.w_weight = self.w_bias = self.w_alpha = None

    def param_specs(self):
        return {"weight": ParamSpec((self.width,), kind="vector", init="ones_normal"), "bias": ParamSpec((self.width,), kind="vector"),
                "alpha": ParamSpec((), kind="vector", init=_alpha_init)}

    def finalize(self):
        self.w_alpha = self.w_alpha.reshape(1).contiguous()
        if self.scale != 1.0:
            self.w_weight, self.w_bias = self.w_weight * self.scale, self.w_bias * self.scale

    def forward(self, h, ctx, rows=None, n_rows=None, tag="norm"):
        n = n_rows if n_rows is not None else ctx.n_tokens
        cap = ctx.want_capacity if rows is not None else ctx.token_capacity
        out = ctx.buf(tag + ("_rows" if rows is not None else ""), (cap, self.width), self.out_dtype)
        partials = ctx.take_pending_residual(h)
        experts = ctx.take_pending_experts(h) if partials is None else None
        if partials is None and experts is None:
            ctx.flush_residual()
        ops.dyn_tanh(h, self.w_alpha, self.w_weight, self.w_bias, out, rows=rows, n_rows=n, partials=partials, experts=experts)
        return out
