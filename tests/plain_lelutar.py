"""A plain, slow Lelutar decoder in float64: whole sequences, no cache, one function per mechanism.

It shares no code with the package: it reads config.json and the safetensors file itself and works on torch
float64 tensors on the CPU.  `round_to` (a torch dtype or None) rounds where a 16-bit engine rounds: weights, the
inputs of matrix products, cached keys, values and latents.

Notation: x [T, E] is the residual stream, d(v) = tanh(alpha v) w + b (scalar alpha, vectors w and b).  The model is

    x = scale * embed[token] + bigram[row(previous token, token)];  layers;  mult * (head d(x))

and a layer is x += mixer(d(x)); x += ff(d(x)) (when it has a feed-forward).  A layer may run with the tensors of
another one.  The mixer is grouped-query attention with a rotation, or attention over a cached latent with or without a
rotated part, a sink in the softmax and a gate per head; the feed-forward squares relu, dense or as a mixture of
experts that are chosen in groups.
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


def dyn_tanh(v, w, name):
    """No mean and no variance: an element answers for itself."""
    return torch.tanh(v * w[name + ".alpha"]) * w[name] + w[name + ".b"]


def relu2(z):
    return torch.clamp(z, min=0.0) ** 2


def matmul(x, w, round_to):
    """x W^T with both operands rounded as a 16-bit engine rounds them."""
    return rnd(x, round_to) @ rnd(w, round_to).T


# --------------------------------------------------------------------------- embedding
def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """The second table's row of every token: a hash of the pair (token before, token); the last row for the first token."""
    return [buckets if i == 0 else (tokens[i - 1] * mul_prev + t * mul_cur) % buckets for i, t in enumerate(tokens)]


def embed(cfg, w, tokens):
    e = cfg["embedding"]
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)] * e["scale"]
    b = e.get("bigram")
    if b:
        x = x + w["bigram"][torch.tensor(bigram_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"]), dtype=torch.long)]
    return x


# --------------------------------------------------------------------------- positions
def frequencies(rot):
    """(frequency per pair, factor on cos and sin)."""
    n, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    s = rot.get("scaling")
    if not s:
        return f, 1.0

    def pair_of(turns):          # the (real-valued) pair that makes `turns` turns over the original length
        return n * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(pair_of(s["fast"])), 0)
    hi = min(math.ceil(pair_of(s["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / s["factor"] * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, rot):
    """x [T, ..., D]: the leading rot.dims elements turn by their position, neighbours (2i, 2i + 1) paired."""
    f, mult = frequencies(rot)
    T = x.shape[0]
    ang = torch.arange(T, dtype=F64)[:, None] * torch.tensor(f, dtype=F64)[None, :]
    shape = (T,) + (1,) * (x.dim() - 2) + (len(f),)
    c, s = (torch.cos(ang) * mult).reshape(shape), (torch.sin(ang) * mult).reshape(shape)
    out = x.clone()
    n = rot["dims"]
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out[..., 0:n:2] = u * c - v * s
    out[..., 1:n:2] = v * c + u * s
    return out


# --------------------------------------------------------------------------- attention
def causal(T):
    return torch.ones(T, T, dtype=torch.bool).tril()


def softmax_with_sink(scores, mask, sink=None):
    """Weights over the visible keys; exp(sink) joins the denominator alone."""
    s = scores.masked_fill(~mask, -math.inf)
    top = s.max(dim=-1, keepdim=True).values
    if sink is not None:
        top = torch.clamp(top, min=float(sink))
    e = torch.exp(s - top)
    total = e.sum(dim=-1, keepdim=True)
    if sink is not None:
        total = total + torch.exp(sink - top)
    return e / total


def attention(x, w, pre, m, eps, round_to=None):
    T = x.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (matmul(x, w[pre + "q"], round_to) + w[pre + "q.b"]).reshape(T, H, D)
    k = (matmul(x, w[pre + "k"], round_to) + w[pre + "k.b"]).reshape(T, G, D)
    v = rnd((matmul(x, w[pre + "v"], round_to) + w[pre + "v.b"]).reshape(T, G, Dv), round_to)
    if m.get("rot"):
        q, k = rotate(q, m["rot"]), rotate(k, m["rot"])
    q, k = rnd(q, round_to), rnd(k, round_to)
    out = torch.zeros(T, H, Dv, dtype=F64)
    for h in range(H):
        g = h // (H // G)
        out[:, h] = softmax_with_sink((q[:, h] @ k[:, g].T) * m["scale"], causal(T)) @ v[:, g]
    return matmul(out.reshape(T, H * Dv), w[pre + "o"], round_to)


def latent_attention(x, w, pre, m, eps, round_to=None):
    """Keys and values expanded per head from a normed latent; a rotated key part shared by all heads where the
    mixer has one.  In 16 bits the latent and the rotated part are rounded as cached, the expanded keys and values are not."""
    T = x.shape[0]
    H, D, Dv, R, Rr = m["heads"], m["dim"], m["vdim"], m["kv_rank"], m.get("rot_dim") or 0
    cq = rms(matmul(x, w[pre + "dq"], round_to), eps) * w[pre + "dq.norm"]
    q = matmul(cq, w[pre + "uq"], round_to).reshape(T, H, D + Rr)
    down = matmul(x, w[pre + "dkv"], round_to)
    c = rnd(rms(down[:, :R], eps) * w[pre + "dkv.norm"], round_to)
    k = (c @ rnd(w[pre + "uk"], round_to).T).reshape(T, H, D)
    v = (c @ rnd(w[pre + "uv"], round_to).T).reshape(T, H, Dv)
    qr, kr = q[..., D:], down[:, R:]
    if Rr and m.get("rot"):
        qr, kr = rotate(qr, m["rot"]), rotate(kr, m["rot"])
    qr, kr = rnd(qr, round_to), rnd(kr, round_to)
    gate = torch.sigmoid(matmul(x, w[pre + "g"], round_to))
    out = torch.zeros(T, H, Dv, dtype=F64)
    for h in range(H):
        s = q[:, h, :D] @ k[:, h].T
        if Rr:
            s = s + qr[:, h] @ kr.T
        out[:, h] = gate[:, h, None] * (softmax_with_sink(s * m["scale"], causal(T), w[pre + "sink"][h]) @ v[:, h])
    return matmul(out.reshape(T, H * Dv), w[pre + "o"], round_to)


MIXERS = {"attention": attention, "latent_attention": latent_attention, "latent_attention_2": latent_attention}


# --------------------------------------------------------------------------- feed-forward
def unit(x, w, pre, round_to=None):
    return matmul(relu2(matmul(x, w[pre + "up"], round_to)), w[pre + "down"], round_to)


def choose(s, correction, top, groups):
    """Indices [top] of one token's experts: only the best groups count, a group being worth its two largest corrected
    scores; among those the largest corrected scores.  Also the smaller of the two margins the choices were made by."""
    pick = (s + correction).tolist()
    n = len(pick)
    allowed, margin = list(range(n)), math.inf
    if groups:
        size = n // groups["count"]
        worth = [sum(sorted(pick[g * size:(g + 1) * size], reverse=True)[:2]) for g in range(groups["count"])]
        order = sorted(range(groups["count"]), key=lambda g: -worth[g])
        kept = set(order[:groups["keep"]])
        if groups["keep"] < groups["count"]:
            margin = worth[order[groups["keep"] - 1]] - worth[order[groups["keep"]]]
        allowed = [e for e in allowed if e // size in kept]
    order = sorted(allowed, key=lambda e: -pick[e])
    if len(order) > top:
        margin = min(margin, pick[order[top - 1]] - pick[order[top]])
    return order[:top], margin


def route(x, w, pre, r, round_to=None, margins=None):
    """(chosen [T, top], weights [T, top]).  `margins` (a list) receives per token by how much the closest of its
    choices was decided, in units of the spread of the token's corrected scores."""
    s = torch.sigmoid(matmul(x, w[pre + "router"], round_to))
    idx, tight = [], []
    for t in range(x.shape[0]):
        chosen, margin = choose(s[t], w[pre + "correction"], r["top"], r.get("groups"))
        idx.append(chosen)
        tight.append(margin / max(float((s[t] + w[pre + "correction"]).std(correction=0)), 1e-30))
    if margins is not None:
        margins.append(torch.tensor(tight, dtype=F64))
    idx = torch.tensor(idx, dtype=torch.long)
    wt = s.gather(1, idx)
    return idx, wt / (wt.sum(dim=-1, keepdim=True) + 1e-20)


def mixture(x, w, pre, mlp, round_to=None, margins=None):
    idx, wt = route(x, w, pre, mlp["router"], round_to, margins)
    y = torch.zeros_like(x)
    for e in range(mlp["router"]["experts"]):
        hit = idx == e
        rows = hit.any(dim=-1)
        if rows.any():
            y[rows] += (wt * hit).sum(dim=-1)[rows][:, None] * unit(x[rows], w, f"{pre}e{e}.", round_to)
    return y


# --------------------------------------------------------------------------- the model
def tensors_of(cfg, i):
    """The layer whose tensors layer i runs with."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg, w, tokens, round_to=None, trace=None, margins=None):
    """Logits [T, vocab] of one sequence; `trace` (a list) receives x after every layer, `margins` (a list) every
    router's margins per token (see `route`)."""
    eps = cfg["norm"]["eps"]
    x = embed(cfg, w, list(tokens))
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{tensors_of(cfg, i)}."
        x = x + MIXERS[layer["type"]](dyn_tanh(x, w, p + "norm1"), w, p + "mix.", layer["mixer"], eps, round_to)
        mlp = layer.get("mlp")
        if mlp:
            h = dyn_tanh(x, w, p + "norm2")
            x = x + (unit(h, w, p + "mlp.", round_to) if mlp["kind"] == "dense" else mixture(h, w, p + "mlp.", mlp, round_to, margins))
        if trace is not None:
            trace.append(x.clone())
    return matmul(dyn_tanh(x, w, "final.norm"), w["head"], round_to) * cfg["logit_scale"]
