"""A plain, slow Tikunex decoder in float64: whole sequences, no cache, one function per mechanism.

It shares no code with the package: it reads config.json and the safetensors file itself and
works on torch float64 tensors on the CPU.  `round_to` (a torch dtype or None) rounds where a
16-bit engine rounds: weights, the inputs of matrix products, cached keys and values.

Notation: x [T, E] is the residual stream, n(v, w) = v / sqrt(mean(v^2) + eps) * (1 + w).  The model is

    x = x0 = n(embed[token]);  layers;  head n(x)

and a layer is x += mixer(n(x)); x += ff(n(x)) (when it has a feed-forward); then a branch of its own for
every token, read from a second table.  The layers of the loop run several times in a row; every pass starts
with x = W [x; x0].  The mixer is gated linear attention, or a windowed attention that keeps the first keys
beside an RWKV-style recurrence, summed with two fixed factors.
"""
from __future__ import annotations

import json
import math
import os
import struct

import torch

F64 = torch.float64


# --------------------------------------------------------------------------- files
def read_safetensors(path):
    """name -> float64 (or int64) tensor."""
    with open(path, "rb") as f:
        n = struct.unpack("<Q", f.read(8))[0]
        header = json.loads(f.read(n))
        data = f.read()
    out = {}
    kinds = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32}
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        a, b = meta["data_offsets"]
        raw = bytearray(data[a:b])
        dt = meta["dtype"]
        if dt in kinds:
            t = torch.frombuffer(raw, dtype=kinds[dt]).to(F64) if raw else torch.zeros(0, dtype=F64)
        elif dt == "I32":
            t = torch.frombuffer(raw, dtype=torch.int32).to(torch.int64)
        else:
            raise ValueError(f"{name}: dtype {dt}")
        out[name] = t.reshape(meta["shape"]).clone()
    return out


def load(folder):
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(folder, "model.safetensors"))


# --------------------------------------------------------------------------- small functions
def rnd(t, round_to):
    return t if round_to is None else t.to(round_to).to(F64)


def rms(v, eps):
    return v / torch.sqrt((v * v).mean(dim=-1, keepdim=True) + eps)


def centred_norm(v, w, eps):
    """An RMS norm whose weight is stored around zero."""
    return rms(v, eps) * (1.0 + w)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def matmul(x, w, round_to):
    """x W^T with both operands rounded as a 16-bit engine rounds them."""
    return rnd(x, round_to) @ rnd(w, round_to).T


# --------------------------------------------------------------------------- attention
def sink_window_mask(T, size, keep_first):
    """[T, T] bool: query i sees key j <= i that is fewer than `size` positions back or among the first `keep_first`
    (size 0: every earlier key)."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    seen = (i - j < size) | (j < keep_first) if size else torch.ones(T, T, dtype=torch.bool)
    return (j <= i) & seen


def masked_softmax(scores, mask):
    s = scores.masked_fill(~mask, -math.inf)
    e = torch.exp(s - s.max(dim=-1, keepdim=True).values)
    return e / e.sum(dim=-1, keepdim=True)


def attention(x, w, pre, m, round_to=None):
    """Grouped-query attention without positions in the scores; returns the heads side by side (no output matrix)."""
    T = x.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rnd(matmul(x, w[pre + "q"], round_to).reshape(T, H, D), round_to)
    k = rnd(matmul(x, w[pre + "k"], round_to).reshape(T, G, D), round_to)
    v = rnd(matmul(x, w[pre + "v"], round_to).reshape(T, G, Dv), round_to)
    mask = m.get("mask") or {}
    seen = sink_window_mask(T, mask.get("size") or 0, mask.get("keep_first") or 0)
    out = torch.zeros(T, H, Dv, dtype=F64)
    for h in range(H):
        g = h // (H // G)
        out[:, h] = masked_softmax((q[:, h] @ k[:, g].T) * m["scale"], seen) @ v[:, g]
    return out.reshape(T, H * Dv)


# --------------------------------------------------------------------------- the RWKV-style recurrence
def shifted_mix(x, mu):
    """x + (the row before - x) * mu, zeros before the first row."""
    before = torch.cat([torch.zeros_like(x[:1]), x[:-1]], dim=0)
    return x + (before - x) * mu


def rwkv_walk(r, k, v, dec, u):
    """r, k, dec [T, H, D], v [T, H, Dv], u [H, D]; S_0 = 0:  o = (S + (u k) v^T)^T r, then S = dec S (rows) + k v^T."""
    T, H, D = r.shape
    S = torch.zeros(H, D, v.shape[2], dtype=F64)
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S + u[:, :, None] * kv, r[t])
        S = dec[t][:, :, None] * S + kv
    return out


def rwkv(x, w, pre, m, eps, round_to=None):
    """Returns the gated heads side by side (no output matrix)."""
    T = x.shape[0]
    H, D = m["heads"], m["dim"]
    x = rnd(x, round_to)             # (what the token before leaves behind is its rounded row)
    mix = {s: shifted_mix(x, w[pre + "mu." + s]) for s in "rkvgw"}
    r, k, v = (matmul(mix[s], w[pre + s], round_to).reshape(T, H, D) for s in "rkv")
    gate = silu(matmul(mix["g"], w[pre + "g"], round_to))
    low = torch.tanh(matmul(mix["w"], w[pre + "w1"], round_to))          # (stays 32-bit on its way into the decay)
    dec = torch.exp(-torch.exp(low @ rnd(w[pre + "w2"], round_to).T + w[pre + "w0"])).reshape(T, H, D)
    o = rms(rwkv_walk(r, k, v, dec, w[pre + "u"]), eps).reshape(T, H * D)
    return o * w[pre + "norm"] * gate


def parallel_mixer(x, w, pre, m, eps, round_to=None):
    """The two scaled results, each through its own output matrix."""
    a = attention(x, w, pre + "left.", m["left"], round_to) * m["left_scale"]
    b = rwkv(x, w, pre + "right.", m["right"], eps, round_to) * m["right_scale"]
    return matmul(a, w[pre + "left.o"], round_to) + matmul(b, w[pre + "right.o"], round_to)


# --------------------------------------------------------------------------- gated linear attention
def gla_walk(q, k, v, alpha):
    """q, k, alpha [T, H, D], v [T, H, Dv]; S_0 = 0:  S = alpha S (rows) + k v^T;  o = S^T q."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=F64)
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out


def gla(x, w, pre, m, eps, round_to=None):
    T = x.shape[0]
    H, D, Dv = m["heads"], m["dim"], m["vdim"]
    q = matmul(x, w[pre + "q"], round_to).reshape(T, H, D) * D ** -0.5
    k = matmul(x, w[pre + "k"], round_to).reshape(T, H, D)
    v = matmul(x, w[pre + "v"], round_to).reshape(T, H, Dv)
    z = matmul(x, w[pre + "a1"], round_to) @ rnd(w[pre + "a2"], round_to).T + w[pre + "a2.b"]
    alpha = (torch.sigmoid(z) ** (1.0 / m["tau"])).reshape(T, H, D)
    o = (rms(gla_walk(q, k, v, alpha), eps) * w[pre + "norm"]).reshape(T, H * Dv)
    return matmul(o * silu(matmul(x, w[pre + "g"], round_to)), w[pre + "o"], round_to)


# --------------------------------------------------------------------------- feed-forward
def gated_unit(x, w, pre, round_to=None):
    return matmul(silu(matmul(x, w[pre + "gate"], round_to)) * matmul(x, w[pre + "up"], round_to), w[pre + "down"], round_to)


def route(x, w, pre, r, round_to=None, margins=None):
    """(chosen [T, top] indices, weights [T, top]): the largest biased logits, and the softmax over those alone.
    `margins` (a list) receives, per token, by how much the last chosen logit beats the first one left out, in units
    of the spread of the token's logits (infinite when every expert is chosen)."""
    z = matmul(x, w[pre + "router"], round_to) + w[pre + "router.b"]
    order = torch.sort(z, dim=-1, descending=True, stable=True)
    top = r["top"]
    if margins is not None:
        if z.shape[1] > top:
            margins.append((order.values[:, top - 1] - order.values[:, top]) / z.std(dim=-1).clamp_min(1e-30))
        else:
            margins.append(torch.full((x.shape[0],), math.inf, dtype=F64))
    return order.indices[:, :top], torch.softmax(order.values[:, :top], dim=-1)


def mixture(x, w, pre, mlp, round_to=None, margins=None):
    idx, wt = route(x, w, pre, mlp["router"], round_to, margins)
    y = torch.zeros_like(x)
    for e in range(mlp["router"]["experts"]):
        hit = idx == e
        rows = hit.any(dim=-1)
        if rows.any():
            y[rows] += (wt * hit).sum(dim=-1)[rows][:, None] * gated_unit(x[rows], w, f"{pre}e{e}.", round_to)
    return y


def side_branch(x, e, w, pre, eps, round_to=None):
    """rms(proj(gelu(gate x) * e)) * w: what a token's part e of the second table adds."""
    g = gelu_tanh(matmul(x, w[pre + "gate"], round_to)) * rnd(e, round_to)
    return rms(matmul(g, w[pre + "proj"], round_to), eps) * w[pre + "norm"]


# --------------------------------------------------------------------------- the model
def run_order(cfg):
    """(layer, first layer of a pass of the loop?) in the order in which they run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    out = [(i, False) for i in range(a)]
    for _ in range(loop["times"]):
        out += [(i, i == a) for i in range(a, b)]
    return out + [(i, False) for i in range(b, n)]


def forward(cfg, w, tokens, round_to=None, trace=None, margins=None):
    """Logits [T, vocab] of one sequence; `trace` (a list) receives x after every layer run, `margins` (a list) every
    router's margins per token (see `route`)."""
    eps = cfg["norm"]["eps"]
    ids = torch.tensor(tokens, dtype=torch.long)
    x = centred_norm(w["embed"][ids], w["embed.norm"], eps)
    x0 = x.clone()
    side = (cfg.get("token_side") or {}).get("dim", 0)
    for i, enters in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if enters:
            x = matmul(torch.cat([x, x0], dim=-1), w["loop.in"], round_to)
        h = centred_norm(x, w[p + "norm1"], eps)
        m = layer["mixer"]
        x = x + (gla if layer["type"] == "gla" else parallel_mixer)(h, w, p + "mix.", m, eps, round_to)
        if layer.get("mlp"):
            x = x + mixture(centred_norm(x, w[p + "norm2"], eps), w, p + "mlp.", layer["mlp"], round_to, margins)
        if side:
            x = x + side_branch(x, w["side.embed"][ids][:, i * side:(i + 1) * side], w, p + "side.", eps, round_to)
        if trace is not None:
            trace.append(x.clone())
    return matmul(centred_norm(x, w["final.norm"], eps), w["head"], round_to)
