"""Lelutar on the GPU against the plain implementation (plain_lelutar.py): every mechanism alone,
then whole models under every way of cutting the work, then generation through the engine."""
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_lelutar as P
from helpers import Replay, assert_close_16bit, assert_close_f32, mixed_schedule, pages_were_reused, peak_pages
from lelutar_configs import LELUTAR, write_model
from mixer_helpers import fill_part as fill_any_part, make_ctx, run_mixers_in_portions

pytestmark = pytest.mark.gpu
TD = {"float32": torch.float32, "bfloat16": torch.bfloat16, "float16": torch.float16}
F64 = torch.float64

# 16-bit bound for whole models, in standard deviations of a row's logits (routing weights multiply whole rows).  A lost
# key, page, pair row or expert moves a row by far more.
C_MODEL = {"bfloat16": 0.09, "float16": 0.012}
CONFIGS = {k: v[0] for k, v in LELUTAR.items()}
CLOSE_CALL = 0.01       # (spreads of a router's choice scores)
CLEAR_CALL = 0.04
_TOKENS = {}


def rounding_of(dtype):
    return None if dtype == "float32" else TD[dtype]


def close(x, ref, dtype, what):
    """Rows of logits against the plain ones.  `ref` may be (logits, sure): in 16 bits a token whose router nearly ties in
    the plain run may take another expert in the engine, which is no fault; such rows are left out, and they must be few."""
    if dtype == "float32":
        assert_close_f32(x, ref, what)
        return
    ref, sure = ref
    sure = sure[:len(ref)]
    assert sure.mean() > 0.8, f"{what}: {int((~sure).sum())} of {len(sure)} tokens route by a close call"
    assert_close_16bit(np.asarray(x)[sure], np.asarray(ref)[sure], what, dtype, c=C_MODEL[dtype])


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {k: write_model(cfg, str(tmp_path_factory.mktemp("lel_" + k)), seed) for k, (cfg, seed) in LELUTAR.items()}


def plain(folder, dtype, tokens):
    """Logits; for a 16-bit type (logits, which tokens route by a clear margin in every routed layer)."""
    cfg, w = P.load(folder)
    margins = []
    logits = P.forward(cfg, w, tokens, rounding_of(dtype), None, margins).numpy()
    if dtype == "float32":
        return logits
    sure = np.ones(len(tokens), dtype=bool)
    for m in margins:
        sure &= m.numpy() > CLOSE_CALL
    return logits, sure


def session(folder, dtype, max_tokens, **kw):
    from ferrum_b200.engine.trace import TraceSession
    return TraceSession(folder, dtype, max_tokens, **kw)


def tokens_for(name, n, seed, folders=None):
    """n random tokens.  Given the models' folders, tokens at which no router of the model decides by a close call (in the
    plain run that rounds to bfloat16): a token that would is drawn again, front to back, since a 16-bit engine may send it
    to another expert, and every later token would differ too."""
    rng = np.random.default_rng(seed)
    vocab = CONFIGS[name]["vocab"]
    toks = rng.integers(0, vocab, n).tolist()
    if folders is None:
        return toks
    if (name, n, seed) not in _TOKENS:
        cfg, w = P.load(folders[name])
        good = 0                       # (a token's result depends on the tokens up to it: what is clear stays clear)
        for _ in range(40 * n):
            margins = []
            upto = min(n, good + 24)
            P.forward(cfg, w, toks[:upto], torch.bfloat16, None, margins)
            unsure = (torch.stack(margins).min(0).values < CLEAR_CALL).nonzero().flatten() if margins else []
            if len(unsure) == 0:
                good = upto
                if good == n:
                    break
                continue
            good = int(unsure[0])
            toks[good] = int(rng.integers(0, vocab))
        else:
            raise AssertionError("no tokens with clear routing found")
        _TOKENS[(name, n, seed)] = toks
    return list(_TOKENS[(name, n, seed)])


def short_name(name):
    """A part's parameter name as the plain implementation calls the tensor."""
    name = name.replace("output.weight", "o").replace("_norm.weight", ".norm").replace(".bias", ".b")
    return name[:-7] if name.endswith(".weight") else name


def fill_part(part, seed, td, prefix, std=0.3, fixed=None):
    return fill_any_part(part, seed, td, prefix, short_name, std, fixed)


def inputs(n, E, td, seed=10):
    g = torch.Generator(device="cuda").manual_seed(seed)
    return torch.randn(n, E, device="cuda", generator=g).to(td)


def batch_of(lens, slots, pos0=None, max_tokens=4096, max_requests=8, tokens=None):
    from ferrum_b200.engine.batch import StepContext, StepEntry
    ctx = StepContext("cuda", max_tokens, max_requests, [])
    ctx.fill([StepEntry(s, pos0[i] if pos0 else 0, tokens[i] if tokens else [1] * n) for i, (s, n) in enumerate(zip(slots, lens))], [])
    return ctx


# ================================================================= the norm and what it finishes on the way
@pytest.mark.parametrize("dtype", ["float32", "bfloat16", "float16"])
@pytest.mark.parametrize("E,T", [(52, 9), (33, 70), (256, 64), (1030, 3), (1032, 65), (2048, 300), (4, 2000)])
def test_dynamic_tanh_alone(cuda, dtype, E, T):
    """All rows, chosen rows, and rows whose expert sum is still open (made once, in place)."""
    from ferrum_b200.ops import lib as ops
    td = TD[dtype]
    g = torch.Generator(device="cuda").manual_seed(E)
    x = torch.randn(T, E, device="cuda", generator=g) * 3.0
    w, b = 1.0 + 0.3 * torch.randn(E, device="cuda", generator=g), torch.randn(E, device="cuda", generator=g)
    alpha = torch.tensor([0.7], device="cuda")
    tol = 1e-6 if dtype == "float32" else (2e-2 if dtype == "bfloat16" else 3e-3)

    def check(out, rows):
        ref = torch.tanh(0.7 * rows.double()) * w.double() + b.double()
        assert ((out.double() - ref).abs() / ref.abs().clamp_min(1.0)).max() < tol
    out = torch.full((T, E), float("nan"), device="cuda", dtype=td)
    ops.dyn_tanh(x, alpha, w, b, out)
    check(out, x)
    rows = torch.randperm(T, device="cuda", generator=g)[:max(1, T // 2)].int()
    picked = torch.full((len(rows), E), float("nan"), device="cuda", dtype=td)
    ops.dyn_tanh(x, alpha, w, b, picked, rows=rows)
    check(picked, x[rows.long()])
    top = 3
    ex = torch.randn(T * top, E, device="cuda", generator=g)
    row_of = torch.randperm(T * top, device="cuda", generator=g).int()
    wt = torch.rand(T * top, device="cuda", generator=g)
    want = x.double() + (ex.double()[row_of.long()] * wt.double()[:, None]).view(T, top, E).sum(1)
    for pick in (None, rows):
        h = x.clone()
        out = torch.full((T if pick is None else len(rows), E), float("nan"), device="cuda", dtype=td)
        ops.dyn_tanh(h, alpha, w, b, out, rows=pick, experts=ops.ExpertSum(ex, row_of, top, wt))
        at = slice(None) if pick is None else rows.long()
        assert (h[at].double() - want[at]).abs().max() < 1e-5
        check(out, h[at])
        if pick is not None:
            left = torch.ones(T, dtype=torch.bool, device="cuda")
            left[rows.long()] = False
            assert torch.equal(h[left], x[left])


@pytest.mark.parametrize("M,E,K", [(1, 640, 384), (8, 4096, 1024), (40, 3328, 2048)])
def test_dynamic_tanh_sums_a_product_left_in_partials(cuda, M, E, K):
    from ferrum_b200.parts import DynamicTanh
    from ferrum_b200.parts.linear import RESIDUAL, linear
    norm = DynamicTanh(E, torch.bfloat16, scale=0.25)
    w = fill_part(norm, 3, torch.bfloat16, "n.")
    ctx = batch_of([M], [0])
    x, wt, h0 = inputs(M, K, torch.bfloat16), inputs(E, K, torch.bfloat16, 2), inputs(M, E, torch.float32, 3)
    h = h0.clone()
    linear(x, wt, h, RESIDUAL, ctx, M=M)
    assert ctx.pending_residual is not None
    out = norm.forward(h, ctx)
    assert ctx.pending_residual is None
    want = h0.double() + x.double() @ wt.double().T
    assert (h.double() - want).abs().max() < 1e-3 * want.abs().max()
    ref = 0.25 * (torch.tanh(want.cpu() * w["n.alpha"]) * w["n.weight"] + w["n.bias"])
    assert (out.double().cpu() - ref).abs().max() < 2e-2


def test_open_sums_reach_norms_that_do_not_know_them(cuda):
    """An RMS norm after a mixture whose sum is still open reads the finished rows."""
    from ferrum_b200.ops import lib as ops
    from ferrum_b200.parts import RMSNorm
    E, T = 64, 5
    norm = RMSNorm(E, 1e-5, torch.float32)
    norm.w_weight = torch.ones(E, device="cuda")
    ctx = batch_of([T], [0])
    h, ex = inputs(T, E, torch.float32), inputs(T, E, torch.float32, 5)
    want = h.double() + ex.double()
    ctx.pending_experts = (h, ops.ExpertSum(ex, torch.arange(T, device="cuda", dtype=torch.int32), 1, None))
    out = norm.forward(h, ctx)
    assert ctx.pending_experts is None and (out.double() - P.rms(want, 1e-5)).abs().max() < 1e-5


# ================================================================= the embedding of tokens and pairs
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("buckets,mul_prev,mul_cur", [(61, 31, 7), (1, 5, 3), (997, 2000003, 1999993)])
def test_pairs_across_portions_and_slots(cuda, dtype, buckets, mul_prev, mul_cur):
    """Requests in several slots, their tokens cut into portions of several sizes down to one, some left out of a step, and
    a slot that a later request takes over: every token's row comes from its own predecessor."""
    from ferrum_b200.engine.batch import StepContext, StepEntry
    from ferrum_b200.parts import BigramTable, TokenEmbedding
    td, V, E = TD[dtype], 1501, 37
    emb = TokenEmbedding(V, E, scale=2.5, bigram=BigramTable(buckets, E, mul_prev, mul_cur))
    g = torch.Generator(device="cuda").manual_seed(1)
    emb.w_weight = torch.randn(V, E, device="cuda", generator=g).to(td)
    emb.bigram.w_weight = torch.randn(buckets + 1, E, device="cuda", generator=g).to(td)
    assert emb.cache_need().state.dtype == torch.int32
    cfg = {"embedding": {"scale": 2.5, "bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}}
    w = {"embed": emb.w_weight.double().cpu(), "bigram": emb.bigram.w_weight.double().cpu()}
    rng = np.random.default_rng(3)
    seqs = {"a": rng.integers(0, V, 40).tolist(), "b": rng.integers(0, V, 9).tolist(), "c": rng.integers(0, V, 23).tolist(), "d": rng.integers(0, V, 6).tolist()}
    slot = {"a": 2, "b": 0, "c": 3, "d": 0}                      # d takes b's slot over
    state = torch.zeros(5, 1, dtype=torch.int32, device="cuda")
    state[1], state[4] = 77, 78
    ctx = StepContext("cuda", 64, 5, [])
    at, got = {k: 0 for k in seqs}, {k: [] for k in seqs}
    for step in ([("a", 7), ("b", 1), ("c", 2)], [("c", 1), ("a", 1), ("b", 8)], [("c", 20), ("d", 1), ("a", 2)], [("a", 1)], [("d", 5), ("a", 29)]):
        ctx.fill([StepEntry(slot[k], at[k], seqs[k][at[k]:at[k] + n]) for k, n in step], [])
        h = emb.forward(ctx, state)[:ctx.n_tokens].double().cpu()
        t = 0
        for k, n in step:
            got[k].append(h[t:t + n])
            at[k] += n
            t += n
        assert ctx.err.item() == 0
    assert all(at[k] == len(seqs[k]) for k in seqs)
    for k in seqs:
        ref = P.embed(cfg, w, seqs[k])
        assert (torch.cat(got[k]) - ref).abs().max() < 1e-5, k
    assert state[1].item() == 77 and state[4].item() == 78          # nobody else's entry
    ctx.fill([StepEntry(1, 0, [V])], [])
    emb.forward(ctx, state)
    assert ctx.err.item() == 1


# ================================================================= attention over cached rows with a sink
def latent_reference(q, rows, pos, H, R, scale, sink, gate):
    """q [n, H, Dk] of queries at `pos`, rows [keys, Dk]: float64; values are the rows' first R elements."""
    out = np.zeros((len(pos), H, R))
    for t, p in enumerate(pos):
        for h in range(H):
            s = rows[:p + 1] @ q[t, h] * scale
            top = max(s.max(), sink[h])
            w = np.exp(s - top)
            out[t, h] = gate[t, h] * (w / (w.sum() + np.exp(sink[h] - top))) @ rows[:p + 1, :R]
    return out


@pytest.mark.parametrize("dtype", ["float32", "bfloat16", "float16"])
@pytest.mark.parametrize("H,R,Rr,page", [(3, 11, 4, 8), (5, 32, 16, 16), (20, 64, 0, 8), (16, 128, 32, 32), (1, 96, 0, 16), (2, 1, 0, 8)])
def test_attention_over_cached_rows_with_a_sink(cuda, dtype, H, R, Rr, page):
    """Rows scattered over the pool, in every way the work is handed out.  One row dominates: a far one, at a page's border,
    the last one of the prompt.  Sinks from one that takes nothing to one that takes nearly everything."""
    from ferrum_b200.ops import lib as ops
    rng = np.random.default_rng(H * 100 + R)
    n_keys, td, Dk, scale = 620, TD[dtype], R + Rr, 0.37
    n_pages = -(-n_keys // page)
    order = rng.permutation(n_pages + 5)[:n_pages]
    table = [int(p) for p in order]
    for hot in (3, page * 9, page * 9 - 1, n_keys - 41):
        rows = rng.standard_normal((n_keys, Dk)) * 0.3
        u = rng.standard_normal(Dk)
        u /= np.sqrt((u * u).sum())
        rows[hot] = u * 3.0
        rt = torch.tensor(rows, device="cuda").to(td)
        rows = rt.double().cpu().numpy()
        plane = torch.zeros(n_pages + 5, 1, 1, page, Dk, device="cuda", dtype=td)
        for lp in range(n_pages):
            n = min(page, n_keys - lp * page)
            plane[order[lp], 0, 0, :n] = rt[lp * page:lp * page + n]
        for pos0, n in ((n_keys - 40, 40), (n_keys - 1, 1), (max(hot - 2, 0), 5), (0, 3)):
            n = min(n, n_keys - pos0)
            ctx = make_ctx([(pos0, n)], widths=[[table]])
            pos = list(range(pos0, pos0 + n))
            strong = 8.0 if dtype == "float32" else 6.0
            q = np.tile(u * strong, (n, H)) + rng.standard_normal((n, H * Dk)) * 0.1
            qt = torch.tensor(q, device="cuda").to(td)
            sink = np.linspace(-20.0, strong * 3.0 * scale + 2.0, H) if H > 1 else np.array([strong * 3.0 * scale])
            st = torch.tensor(sink, device="cuda", dtype=torch.float32)
            gate = torch.rand(n, H, device="cuda") + 0.5
            ref = latent_reference(qt.double().cpu().numpy().reshape(n, H, Dk), rows, pos, H, R, scale, st.double().cpu().numpy(), gate.double().cpu().numpy())
            modes = [("cores", False)] + ([("tensor", False), ("tensor", True)] if dtype != "float32" and Dk % 16 == 0 and R % 32 == 0 else [])
            for kind, wide in modes:
                for split in ((False, True) if n == 1 else (False,)):
                    out = torch.full((n, H * R), float("nan"), device="cuda", dtype=td)
                    part, slots = None, 0
                    if split:
                        slots = n_keys // ops.attention_latent_split() + 2
                        part = torch.full((n * H * slots * (R + 2),), float("nan"), device="cuda")
                    ops.attention_latent(qt, out, gate, n, ctx, ctx.block_tables[0], plane, plane.stride(0), page, H, Dk, R, scale, 0, n == 1,
                                         part=part, split_slots=slots, tensor_cores=kind == "tensor", sink=st, wide_weights=wide)
                    got = out.double().cpu().numpy().reshape(n, H, R)
                    assert ctx.err.item() == 0
                    tol = {"float32": 2e-5, "bfloat16": 1.2e-2, "float16": 2e-3}[dtype]
                    assert np.abs(got - ref).max() < tol * max(np.abs(ref).max(), 0.1), (hot, pos0, n, kind, wide, split)
    # (a sink that is left out shows in the reference)
    assert abs(latent_reference(q.reshape(n, H, Dk), rows, pos, H, R, scale, sink * 0 - 1e9, np.ones((n, H))) -
               latent_reference(q.reshape(n, H, Dk), rows, pos, H, R, scale, sink, np.ones((n, H)))).max() > 0.01


@pytest.mark.parametrize("H,R,Rr", [(16, 64, 32), (4, 128, 0), (2, 512, 64)])
def test_wide_weights_keep_float32_precision(cuda, H, R, Rr):
    """The float32 partials of single tokens (before anything is rounded to the output type), bfloat16 rows: with wide weights
    the weighted sum is as good as float32 arithmetic makes it, without them it shows the weights' rounding."""
    from ferrum_b200.ops import lib as ops
    rng = np.random.default_rng(R)
    page, n_keys, Dk, td = 16, 500, R + Rr, torch.bfloat16
    n_pages = -(-n_keys // page)
    rt = torch.tensor(rng.standard_normal((n_pages * page, Dk)), device="cuda").to(td)
    plane = rt.view(n_pages, 1, 1, page, Dk).contiguous()
    ctx = make_ctx([(n_keys - 1, 1)], widths=[[list(range(n_pages))]])
    qt = torch.tensor(rng.standard_normal((1, H * Dk)) * 0.4, device="cuda").to(td)
    rows, q = rt.double()[:n_keys], qt.double().view(H, Dk)
    s = q @ rows.T * 0.2
    ref = torch.softmax(s, dim=1) @ rows[:, :R]
    errs = {}
    for wide in (False, True):
        slots = n_keys // ops.attention_latent_split() + 2
        part = torch.zeros(H * slots * (R + 2), device="cuda")
        out = torch.zeros(1, H * R, device="cuda", dtype=td)
        ops.attention_latent(qt, out, None, 1, ctx, ctx.block_tables[0], plane, plane.stride(0), page, H, Dk, R, 0.2, 0, True, part=part,
                             split_slots=slots, tensor_cores=True, wide_weights=wide)
        p = part.view(H, slots, R + 2).double()[:, :-(-n_keys // ops.attention_latent_split())]
        f = torch.exp(p[..., 0] - p[..., 0].max(dim=1, keepdim=True).values)
        o = (p[..., 2:] * f[..., None]).sum(1) / (p[..., 1] * f).sum(1)[:, None]
        errs[wide] = float((o - ref).abs().max() / ref.abs().max())
    assert errs[True] < 2e-5 and errs[False] > 5 * errs[True], errs


def plain_heads(q, k, v, pos, scale):
    """q [n, H, D], k and v [keys, G, D] float64: causal grouped-query attention of queries at `pos`."""
    G = k.shape[1]
    out = torch.zeros_like(q)
    for t, p in enumerate(pos):
        for h in range(q.shape[1]):
            g = h // (q.shape[1] // G)
            out[t, h] = torch.softmax(k[:p + 1, g] @ q[t, h] * scale, dim=0) @ v[:p + 1, g]
    return out


@pytest.mark.parametrize("dtype", ["bfloat16", "float16"])
@pytest.mark.parametrize("H,G,D,page", [(8, 2, 64, 16), (4, 4, 128, 8), (16, 1, 64, 32), (6, 2, 128, 16)])
def test_grouped_attention_with_wide_weights(cuda, dtype, H, G, D, page):
    """Values of +-64 around a small signal: what the weights lose to rounding shows in the result unless they keep their
    precision.  Prompt portions, one token over a range that is cut among CTAs, the first tokens; a far dominant key."""
    from ferrum_b200.cache.storage import LayerCache
    from ferrum_b200.parts import ShapedAttention
    td, n_keys, rng = TD[dtype], 620, np.random.default_rng(D)
    n_pages = -(-n_keys // page)
    order = rng.permutation(n_pages + 4)[:n_pages]
    k = rng.standard_normal((n_keys, G, D)) * 0.4
    v = rng.standard_normal((n_keys, G, D))
    v[0::2] += 64.0
    v[1::2] -= 64.0
    kt, vt = torch.tensor(k, device="cuda").to(td), torch.tensor(v, device="cuda").to(td)
    plane = torch.zeros(n_pages + 4, 2, G, page, D, device="cuda", dtype=td)
    for lp in range(n_pages):
        n = min(page, n_keys - lp * page)
        plane[order[lp], 0, :, :n] = kt[lp * page:lp * page + n].transpose(0, 1)
        plane[order[lp], 1, :, :n] = vt[lp * page:lp * page + n].transpose(0, 1)
    cache = LayerCache(group=0, plane=plane, page_stride=plane.stride(0), page_size=page, writes=True, state=None)
    mixer = ShapedAttention(32, H, G, D, D, td, 0.2, wide_weights=True)
    assert mixer.on_tensor_cores()

    def run(q, pos0, n):
        ctx = make_ctx([(pos0, n)], widths=[[[int(p) for p in order]]])
        out = torch.full((n, H * D), float("nan"), device="cuda", dtype=td)
        mixer._flash(q, out, ctx, cache, ctx.block_tables[0])
        assert ctx.err.item() == 0
        return out.double().view(n, H, D)
    unit = 2.0 ** (-8 if dtype == "bfloat16" else -11)            # (a result's own rounding is half of this)
    for pos0, n in ((n_keys - 170, 170), (n_keys - 70, 70), (n_keys - 1, 1), (100, 2), (0, 5), (0, 140)):
        qt = torch.tensor(rng.standard_normal((n, H * D)) * 0.5, device="cuda").to(td)
        ref = plain_heads(qt.double().view(n, H, D), kt.double(), vt.double(), list(range(pos0, pos0 + n)), 0.2)
        errs = []
        for mixer.wide_weights in (True, False):
            errs.append(((run(qt, pos0, n) - ref).abs() / ref.abs().clamp_min(1.0)).max().item())
        assert errs[0] < unit + 2e-3, (pos0, n, errs)
        if n in (70, 170):
            assert errs[1] > 2.0 * errs[0], errs
    mixer.wide_weights = True
    hot = page * 7 - 1                       # a page's last row, far back
    kt[hot] *= 8.0
    plane[order[hot // page], 0, :, hot % page] = kt[hot]
    for pos0, n in ((n_keys - 70, 70), (n_keys - 1, 1), (hot - 1, 3), (hot - 100, 300)):
        if pos0 < 0:
            continue
        qt = (kt[hot].double().repeat_interleave(H // G, dim=0).reshape(1, H * D).repeat(n, 1) * 2.0).to(td)
        got = run(qt, pos0, n)
        for i in range(n):
            near = (got[i] - vt[hot].double().repeat_interleave(H // G, dim=0)).abs().max()
            assert (near < 1.0) == (pos0 + i >= hot), (pos0, i)


# ================================================================= mixers alone, whole and in portions
CUTS = ([61], [20, 1, 1, 2, 30, 7], [2] * 30 + [1], [1] * 61)


def check_mixer(mixer, ref, x, td, dtype, page=8):
    for cut in CUTS:
        got = run_mixers_in_portions([mixer], [x], cut, td, page=page, max_tokens=128)[0]
        assert torch.isfinite(got).all(), cut
        assert (got - ref).abs().max() < (2e-4 if dtype == "float32" else 4e-2) * ref.abs().max(), cut


def table_of(rot, dim, n_pos=256):
    from ferrum_b200.parts import RotaryEmbedding
    from ferrum_b200.parts.rope import yarn
    if not rot:
        return None
    f, mag = None, 1.0
    if rot.get("scaling"):
        s = rot["scaling"]
        f, mag = yarn(rot["dims"], rot["base"], s["factor"], s["original"], s["fast"], s["slow"])
    return RotaryEmbedding(dim, rot["dims"], rot["base"], None, "adjacent", n_pos, "cuda", frequencies=f, magnitude=mag)


YARN = {"factor": 4.0, "original": 40, "fast": 8.0, "slow": 1.0}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,D,Dv,rot", [(6, 2, 10, 14, {"base": 60.0, "dims": 6, "scaling": YARN}), (4, 4, 32, 16, {"base": 500.0, "dims": 32, "scaling": YARN}),
                                          (3, 1, 8, 24, {"base": 20.0, "dims": 8}), (2, 1, 2, 1, {"base": 9.0, "dims": 2, "scaling": YARN}), (10, 2, 6, 6, None),
                                          (7, 1, 64, 96, {"base": 10000.0, "dims": 64, "scaling": YARN}), (2, 2, 128, 128, {"base": 100.0, "dims": 40}),
                                          (8, 1, 40, 64, {"base": 500.0, "dims": 24, "scaling": YARN}), (16, 1, 128, 128, None), (17, 1, 64, 64, None)])
def test_rotating_attention_alone(cuda, dtype, H, G, D, Dv, rot):
    from ferrum_b200.parts import ShapedAttention
    td, E = TD[dtype], 40
    scale = 0.45 if D < 64 else 0.1
    mixer = ShapedAttention(E, H, G, D, Dv, td, scale, rotary=table_of(rot, D), qkv_bias=True, wide_weights=True)
    assert mixer.on_tensor_cores() == (dtype == "bfloat16" and max(D, Dv) in (64, 128) and Dv >= D and H // G <= 16)
    w = fill_part(mixer, 9, td, "p.")
    x = inputs(61, E, td)
    m = {"heads": H, "kv_heads": G, "dim": D, "vdim": Dv, "scale": scale, "rot": rot}
    ref = P.attention(x.double().cpu(), w, "p.", m, 1e-5, rounding_of(dtype))
    check_mixer(mixer, ref, x, td, dtype)
    if rot:                   # what a half-split pairing, or a magnitude that is left out, would give is something else
        off = P.attention(x.double().cpu(), w, "p.", dict(m, rot=None), 1e-5, rounding_of(dtype))
        assert (off - ref).abs().max() > 1e-2 * ref.abs().max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,D,Rr,Dv,R,Rq,rot", [(3, 7, 0, 9, 11, 13, None), (5, 6, 4, 10, 18, 17, {"base": 30.0, "dims": 4, "scaling": YARN}),
                                                (8, 16, 0, 24, 64, 32, None), (4, 24, 32, 40, 96, 56, {"base": 300.0, "dims": 32, "scaling": YARN}),
                                                (20, 8, 16, 8, 32, 24, {"base": 100.0, "dims": 16}), (1, 1, 2, 1, 1, 1, {"base": 5.0, "dims": 2}),
                                                (2, 64, 64, 128, 256, 96, {"base": 5000.0, "dims": 64, "scaling": YARN})])
def test_latent_attention_alone(cuda, dtype, H, D, Rr, Dv, R, Rq, rot):
    """Without positions and with a rotated key part that all heads share; a sink that matters, a gate per head."""
    from ferrum_b200.parts import LatentAttention
    td, E, eps = TD[dtype], 40, 1e-3
    mixer = LatentAttention(E, H, D, Rr, Dv, R, Rq, eps, 0.4, td, rotary=table_of(rot, Rr), sink=True, wide_weights=True)
    sink = torch.linspace(-1.0, 4.0, H) if H > 1 else torch.tensor([2.0])
    w = fill_part(mixer, 11, td, "p.", std=0.3 if R < 100 else 0.1, fixed={"sink": sink})       # (scores of a moderate size)
    x = inputs(61, E, td, seed=12)
    m = {"heads": H, "dim": D, "rot_dim": Rr, "vdim": Dv, "kv_rank": R, "q_rank": Rq, "scale": 0.4, "rot": rot}
    rd = rounding_of(dtype)
    ref = P.latent_attention(x.double().cpu(), w, "p.", m, eps, rd)
    check_mixer(mixer, ref, x, td, dtype)
    lost = P.latent_attention(x.double().cpu(), dict(w, **{"p.sink": torch.full((H,), -1e9, dtype=F64)}), "p.", m, eps, rd)
    assert (lost - ref).abs().max() > 2e-2 * ref.abs().max()


def test_one_block_run_twice_keeps_two_caches(cuda):
    """The same mixer as two entries of a schedule, on different rows: each run reads the rows it cached itself."""
    from ferrum_b200.parts import LatentAttention
    td, E, eps = torch.float32, 40, 1e-4
    mixer = LatentAttention(E, 3, 8, 0, 8, 12, 10, eps, 0.5, td, sink=True)
    w = fill_part(mixer, 13, td, "p.")
    xs = [inputs(50, E, td, seed=s) for s in (1, 2)]
    m = {"heads": 3, "dim": 8, "vdim": 8, "kv_rank": 12, "q_rank": 10, "scale": 0.5}
    for cut in ([50], [7, 1, 1, 20, 21]):
        got = run_mixers_in_portions([mixer, mixer], xs, cut, td)
        for x, y in zip(xs, got):
            ref = P.latent_attention(x.double().cpu(), w, "p.", m, eps)
            assert (y - ref).abs().max() < 2e-4 * ref.abs().max()


# ================================================================= feed-forwards
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E,F,T", [(52, 36, 9), (128, 96, 1), (256, 512, 16), (256, 300, 70), (512, 1024, 130), (128, 264, 600), (64, 4096, 3)])
def test_plain_unit_alone(cuda, dtype, E, F, T):
    from ferrum_b200.parts import PlainUnit
    td = TD[dtype]
    ffn = PlainUnit(E, F, td)
    w = fill_part(ffn, 31, td, "f.", std=0.2)
    x = inputs(T, E, td, seed=32)
    ref = P.unit(x.double().cpu(), w, "f.", rounding_of(dtype))
    ctx = batch_of([T], [0])
    h0 = inputs(T, E, torch.float32, seed=33)
    h = h0.clone()
    ffn.forward(x, ctx, h)
    ctx.flush_residual()
    assert ctx.err.item() == 0
    assert ((h - h0).double().cpu() - ref).abs().max() < (2e-4 if dtype == "float32" else 2e-2) * ref.abs().max()
    y = torch.full((T, E), float("nan"), device="cuda")
    ffn.forward(x, ctx, y, accumulate=False)
    assert (y - (h - h0)).abs().max() < 1e-3 * ref.abs().max()


@pytest.mark.parametrize("dtype", ["bfloat16", "float16"])
@pytest.mark.parametrize("M,N,K", [(1, 130, 64), (8, 2048, 4096), (20, 136, 264), (100, 640, 1024), (300, 1000, 72), (513, 513, 4096), (2048, 1536, 512), (700, 4104, 8192)])
def test_product_with_squared_relu(cuda, dtype, M, N, K):
    """The epilogue of every tensor-core product kernel, also where several CTAs share a tile (long K, few tiles); N may be odd
    (then the threads write the rows themselves)."""
    from ferrum_b200.ops import lib as ops
    td = TD[dtype]
    x, w = inputs(M, K, td) * 0.5, inputs(N, K, td, 2) * K ** -0.5
    ctx = batch_of([1], [0])
    ws, cnt = ctx.gemm_scratch(M, N, K, False)
    out = torch.full((M, N), float("nan"), device="cuda", dtype=td)
    ops.gemm_tc(x, w, out, ops.TC_RELU2, ctx.err, ws, cnt)
    ref = torch.clamp(x.double() @ w.double().T, min=0.0) ** 2
    assert ctx.err.item() == 0
    assert (out.double() - ref).abs().max() < (1e-2 if dtype == "bfloat16" else 2e-3) * ref.abs().max() and (out == 0).double().mean() > 0.3


@pytest.mark.parametrize("T", [2, 40])
def test_group_choice_by_hand(cuda, T):
    """Only the best groups' experts can be chosen, also when every choice score is below zero; a group is worth its two largest
    together; ties go to the lower index; the weights are the uncorrected scores over their sum."""
    from ferrum_b200.ops import lib as ops
    logit = lambda p: math.log(p / (1.0 - p))
    rows = [[0.9, 0.1, 0.6, 0.6, 0.5, 0.2], [0.3, 0.3, 0.3, 0.3, 0.3, 0.3]] * (T // 2)
    logits = torch.tensor([[logit(p) for p in r] for r in rows], device="cuda")
    x = torch.arange(T, device="cuda", dtype=torch.float32)[:, None].repeat(1, 8)

    def route(top, groups, correction, eps=1e-20, lg=logits):
        n = lg.shape[1]
        expert_of, rank_of, row_of = (torch.full((T * top,), -7, dtype=torch.int32, device="cuda") for _ in range(3))
        weight_of, counts = torch.zeros(T * top, device="cuda"), torch.full((n,), 9, dtype=torch.int32, device="cuda")
        xg = torch.zeros(T * top, 8, device="cuda")
        ops.moe_route(lg, T, n, top, x, False, expert_of, rank_of, weight_of, counts, xg, row_of, scores="sigmoid", renormalize=True,
                      correction=torch.tensor(correction, device="cuda"), groups=groups, renorm_eps=eps)
        first = torch.cumsum(counts, 0) - counts
        for pair in range(T * top):
            e, row = expert_of[pair].item(), row_of[pair].item()
            assert first[e] <= row < first[e] + counts[e] and xg[row, 0].item() == pair // top
        return expert_of.view(T, top).tolist()[:2], weight_of.view(T, top).tolist()[:2]
    zero = [0.0] * 6
    chosen, wt = route(2, (3, 1), zero)
    assert chosen == [[2, 3], [0, 1]] and wt[0] == pytest.approx([0.5, 0.5])
    chosen, wt = route(3, (3, 2), zero)
    assert chosen == [[0, 2, 3], [0, 1, 2]] and wt[0] == pytest.approx([0.9 / 2.1, 0.6 / 2.1, 0.6 / 2.1], rel=1e-5)
    assert route(2, None, zero)[0] == [[0, 2], [0, 1]]
    low = [-2.0, -2.0, -2.0, -2.0, -1.0, -1.0]
    chosen, wt = route(2, (3, 1), low)
    assert chosen == [[4, 5], [4, 5]] and wt[0] == pytest.approx([0.5 / 0.7, 0.2 / 0.7], rel=1e-5)
    assert route(3, (3, 2), low)[0] == [[4, 5, 2], [4, 5, 0]]
    assert route(2, (6, 2), zero)[0] == [[0, 2], [0, 1]] and route(4, (3, 3), zero)[0] == [[0, 2, 3, 4], [0, 1, 2, 3]]
    assert route(2, (3, 1), zero, eps=1.0)[1][0] == pytest.approx([0.6 / 2.2, 0.6 / 2.2], rel=1e-5)
    tiny = torch.full((T, 6), -200.0, device="cuda")             # every score underflows to zero: zero weights, nothing undefined
    assert route(2, (3, 1), zero, lg=tiny)[1][0] == [0.0, 0.0]


@pytest.mark.parametrize("n_exp,top,groups", [(12, 3, (4, 2)), (64, 6, (8, 4)), (256, 8, (8, 4)), (256, 8, (64, 7)), (96, 5, (96, 40)), (40, 3, (5, 5)), (7, 7, (1, 1))])
def test_group_choice_against_the_plain_one(cuda, n_exp, top, groups):
    """Random scores with corrections of both signs; the two routing kernels (few and many tokens)."""
    from ferrum_b200.ops import lib as ops
    g = torch.Generator(device="cuda").manual_seed(n_exp)
    for T in (3, 200):
        logits = torch.randn(T, n_exp + 3, device="cuda", generator=g)[:, :n_exp]
        corr = torch.randn(n_exp, device="cuda", generator=g) * 0.4 - 0.5
        expert_of, rank_of, row_of = (torch.full((T * top,), -7, dtype=torch.int32, device="cuda") for _ in range(3))
        weight_of, counts = torch.zeros(T * top, device="cuda"), torch.zeros(n_exp, dtype=torch.int32, device="cuda")
        x, xg = torch.zeros(T, 8, device="cuda"), torch.zeros(T * top, 8, device="cuda")
        ops.moe_route(logits, T, n_exp, top, x, False, expert_of, rank_of, weight_of, counts, xg, row_of, scores="sigmoid", renormalize=True,
                      correction=corr, groups=groups, renorm_eps=1e-20)
        s = torch.sigmoid(logits.double().cpu())
        compared = 0
        for t in range(T):
            want, margin = P.choose(s[t], corr.double().cpu(), top, {"count": groups[0], "keep": groups[1]})
            if margin < 1e-5:
                continue
            assert sorted(expert_of.view(T, top)[t].tolist()) == sorted(want), t
            chosen = expert_of.view(T, top)[t].long().cpu()
            assert (weight_of.view(T, top)[t].double().cpu() - s[t][chosen] / s[t][chosen].sum()).abs().max() < 1e-6
            compared += 1
        assert compared > 0.9 * T and counts.sum().item() == T * top


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E,F,n_exp,top,groups,T", [(52, 20, 10, 3, (5, 3), 37), (128, 64, 6, 2, (3, 2), 300), (40, 24, 1, 1, (1, 1), 9), (64, 32, 16, 4, (4, 2), 70),
                                                    (72, 100, 4, 4, None, 11), (128, 128, 4, 2, (2, 1), 1000), (256, 80, 7, 1, (7, 3), 2), (64, 48, 40, 8, (8, 4), 16)])
def test_ungated_experts_alone(cuda, dtype, E, F, n_exp, top, groups, T):
    """Sizes that take each of the product kernels and both routing kernels; the sum is made by the norm after it, by whoever
    else asks for the rows, or into a buffer."""
    from ferrum_b200.parts import DynamicTanh, RoutedFeedForward
    td = TD[dtype]
    ffn = RoutedFeedForward(E, F, n_exp, top, td, act="relu2", gated=False, scores="sigmoid", renormalize=True, scale_input=False, correction=True,
                            groups=groups, renorm_eps=1e-20, defer_sum=True)
    w = fill_part(ffn, 21, td, "f.", std=0.3, fixed={"correction": torch.linspace(-1.0, 0.3, n_exp)})
    x = inputs(T, E, td, seed=22)
    margins = []
    router = {"experts": n_exp, "top": top}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    ref = P.mixture(x.double().cpu(), w, "f.", {"router": router}, rounding_of(dtype), margins)
    ctx = batch_of([T], [0])
    h0 = inputs(T, E, torch.float32, seed=23)
    sure = (margins[0] > (1e-6 if dtype == "float32" else CLEAR_CALL)).numpy()
    assert sure.any() and sure.mean() >= min(0.5, 1.0 - 1.0 / T)
    tol = 2e-4 if dtype == "float32" else 4e-2
    h = h0.clone()
    ffn.forward(x, ctx, h)
    assert ctx.pending_experts is not None and torch.equal(h, h0)
    norm = DynamicTanh(E, torch.float32)
    fill_part(norm, 24, td, "n.")
    out = norm.forward(h, ctx)
    assert ctx.err.item() == 0 and ctx.pending_experts is None
    assert ((h - h0).double().cpu() - ref)[sure].abs().max() < tol * ref.abs().max()
    want = torch.tanh(h.double() * norm.w_alpha.double()) * norm.w_weight.double() + norm.w_bias.double()
    assert (out.double() - want).abs().max() < 1e-5
    h2 = h0.clone()
    ffn.forward(x, ctx, h2)
    ctx.flush_residual()
    assert (h2 - h).abs().max() < 1e-4 * ref.abs().max()
    y = torch.full((T, E), float("nan"), device="cuda")
    ffn.forward(x, ctx, y, accumulate=False)
    assert ctx.pending_experts is None and (y - (h - h0)).abs().max() < 1e-4 * ref.abs().max()


# ================================================================= whole models, every way of cutting the work
CASES = [(n, d) for n in ("A", "B") for d in ("float32", "bfloat16")] + [("E", "bfloat16")]


@pytest.mark.parametrize("name,dtype", CASES + [("C", "float32"), ("C", "bfloat16"), ("D", "float32"), ("D", "bfloat16"), ("E", "float32")])
def test_whole_prompt_and_first_tokens(cuda, folders, name, dtype):
    toks = tokens_for(name, 140, 10, folders)
    r = Replay(session(folders[name], dtype, 160))
    r.step([("a", toks, "all")], end=["a"])
    close(r.logits("a", len(toks)), plain(folders[name], dtype, toks), dtype, f"{name} whole")
    r = Replay(session(folders[name], dtype, 64))
    r.step([("b", toks[:1], "all")])
    r.step([("b", toks[1:3], "all")])
    r.step([("b", toks[3:4], "all")], end=["b"])
    close(r.logits("b", 4), plain(folders[name], dtype, toks[:4]), dtype, f"{name} first tokens")


@pytest.mark.parametrize("name", ["A", "B", "C", "D", "E"])
def test_residual_rows_after_every_layer_run(cuda, folders, name):
    toks = tokens_for(name, 25, 11, folders)
    cfg, w = P.load(folders[name])
    taps = []
    P.forward(cfg, w, toks, None, taps)
    s = session(folders[name], "float32", 64)
    got = []
    s.model.on_run = lambda k, h: got.append(h[:len(toks)].double().cpu())
    s.run_step({"step": 0, "entries": [{"id": "a", "tokens": toks, "want": []}], "end": ["a"]})
    assert len(got) == len(taps) == len(cfg["layers"])
    for k, (g, t) in enumerate(zip(got, taps)):
        assert (g - t).abs().max() < 1e-4 * t.abs().max(), k


@pytest.mark.parametrize("name,dtype", CASES + [("D", "float32")])
def test_prefill_then_long_decoding(cuda, folders, name, dtype):
    """30 tokens at once, then 120 one by one from a captured graph."""
    toks = tokens_for(name, 150, 12, folders)
    ref = plain(folders[name], dtype, toks)
    s = session(folders[name], dtype, 160, page_size=8)
    r = Replay(s)
    r.step([("a", toks[:30], "all")])
    for t in toks[30:]:
        r.step([("a", [t], "all")])
    close(r.logits("a", len(toks)), ref, dtype, f"{name} prefill+decode")
    assert s.runner.graph_replays > 0          # single tokens ran from a captured graph


@pytest.mark.parametrize("name", ["A", "C"])
def test_token_by_token_from_the_first(cuda, folders, name):
    toks = tokens_for(name, 70, 17, folders)
    ref = plain(folders[name], "float32", toks)
    r = Replay(session(folders[name], "float32", 80, page_size=8))
    for t in toks:
        r.step([("a", [t], "all")])
    close(r.logits("a", len(toks)), ref, "float32", f"{name} token by token")


@pytest.mark.parametrize("name,dtype", CASES + [("C", "float32"), ("D", "float32")])
@pytest.mark.parametrize("sizes", [[2], [5, 2, 7, 3, 2, 16, 17, 2, 31, 1, 33, 2], [64, 3, 1]])
def test_portions(cuda, folders, name, dtype, sizes):
    toks = tokens_for(name, 131, 13, folders)
    ref = plain(folders[name], dtype, toks)
    r = Replay(session(folders[name], dtype, 144, page_size=16))
    i = k = 0
    while i < len(toks):
        n = min(sizes[k % len(sizes)], len(toks) - i)
        r.step([("a", toks[i:i + n], "all")])
        i += n
        k += 1
    close(r.logits("a", len(toks)), ref, dtype, f"{name} portions {sizes[:3]}")


@pytest.mark.parametrize("name,dtype", CASES)
@pytest.mark.parametrize("page_size", [8, 32])
def test_mixed_batches_reuse_pages_and_slots(cuda, folders, name, dtype, page_size):
    """Six requests through four slots, portions beside single tokens; the pool has fewer pages than all requests need
    together: finished requests' pages and slots go to later ones (whose first token has no predecessor)."""
    lens = {"a": 70, "b": 45, "c": 33, "d": 90, "e": 50, "f": 21}
    toks = {k: tokens_for(name, n, 20 + i, folders) for i, (k, n) in enumerate(lens.items())}
    schedule = mixed_schedule(lens)
    pool = peak_pages(schedule, page_size)
    s = session(folders[name], dtype, pool * page_size, page_size=page_size, max_requests=4)
    slots_seen, owners = {}, {}
    r = Replay(s)
    for entries, ended in schedule:
        r.step([(k, toks[k][first:first + n], "all") for k, first, n in entries], end=ended)
        for k, slot in s.slots.items():
            slots_seen.setdefault(slot, set()).add(k)
        for g in range(s.cache.manager.n_groups):
            for k, slot in s.slots.items():
                for p in s.cache.manager.table(g, slot):
                    if p >= 0:
                        owners.setdefault((g, p), set()).add(k)
        assert s.cache.manager.check() == ""
    assert pages_were_reused(owners) and any(len(v) > 1 for v in slots_seen.values())
    for k in toks:
        close(r.logits(k, lens[k]), plain(folders[name], dtype, toks[k]), dtype, f"{name} mixed {k}")


@pytest.mark.parametrize("name", ["A", "B", "D"])
def test_logits_do_not_depend_on_the_batch(cuda, folders, name):
    """float32: a request's logits beside three others equal those it gets alone to rounding."""
    toks = {k: tokens_for(name, n, 40 + i, folders) for i, (k, n) in enumerate({"a": 50, "b": 9, "c": 31, "d": 2}.items())}
    alone = {}
    for k, t in toks.items():
        r = Replay(session(folders[name], "float32", 64))
        r.step([(k, t, "all")], end=[k])
        alone[k] = r.logits(k, len(t))
    r = Replay(session(folders[name], "float32", 128))
    r.step([(k, t[:len(t) // 2], "all") for k, t in toks.items()])
    r.step([(k, t[len(t) // 2:], "all") for k, t in reversed(list(toks.items()))], end=list(toks))
    for k, t in toks.items():
        assert np.abs(r.logits(k, len(t)) - alone[k]).max() < 3e-5 * max(1.0, np.abs(alone[k]).max()), k


def test_a_long_prompt_and_a_far_token(cuda, folders):
    """700 tokens at once equal the same in portions and the plain run, and two prompts that differ in one early token still
    differ at the end (nothing is windowed)."""
    for name in ("A", "B"):
        toks = tokens_for(name, 700, 31)
        other = list(toks)
        other[5] = (other[5] + 1) % CONFIGS[name]["vocab"]
        out = []
        for t, cuts in ((toks, [700]), (toks, [50, 2, 400, 248]), (other, [700])):
            r = Replay(session(folders[name], "float32", 704))
            i = 0
            for n in cuts:
                r.step([("a", t[i:i + n], "all")])
                i += n
            out.append(r.logits("a", len(t)))
        close(out[0], plain(folders[name], "float32", toks), "float32", f"{name} long")
        assert np.abs(out[0] - out[1]).max() < 5e-5 * np.abs(out[0]).max()
        d = np.abs(out[0] - out[2]).max(axis=1)
        assert d[5] > 1e-3 and d[-20:].min() > 1e-5 and d[:5].max() < 1e-5


@pytest.mark.parametrize("dtype", ["bfloat16", "float16"])
def test_long_requests_on_the_tensor_core_attention(cuda, folders, dtype):
    """Three requests of hundreds of tokens, portions of all sizes beside single tokens in one batch: rows go to every kernel of the
    tensor-core attention (the work lists' three classes, key ranges cut among CTAs) in the same step."""
    lens = {"a": 400, "b": 333, "c": 290}
    toks = {k: tokens_for("E", n, 70 + i, folders) for i, (k, n) in enumerate(lens.items())}
    s = session(folders["E"], dtype, 1200, page_size=16)
    assert all(b.mixer.on_tensor_cores() for b in s.model.blocks[:2])
    r, at = Replay(s), {k: 0 for k in lens}
    sizes = {"a": [150, 1, 3, 200, 1, 40], "b": [1, 2, 17, 130, 1, 180], "c": [64, 190, 1, 1, 30, 2]}
    step = 0
    while any(at[k] < lens[k] for k in lens):
        entries = []
        for k in lens:
            n = min(sizes[k][step % 6], lens[k] - at[k])
            if n:
                entries.append((k, toks[k][at[k]:at[k] + n], "all"))
                at[k] += n
        r.step(entries)
        step += 1
    for k in lens:
        close(r.logits(k, lens[k]), plain(folders["E"], dtype, toks[k]), dtype, f"E long {k}")


def plain_generate(cfg, w, prompt, n, rd=None):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(P.forward(cfg, w, seq, rd)[-1].argmax()))
    return seq[len(prompt):]


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("B", "float32"), ("B", "bfloat16"), ("D", "float32"), ("E", "bfloat16")])
def test_greedy_generation_through_the_engine(cuda, folders, name, dtype):
    """Engine.generate (scheduler, sampler, chunked prompts, several requests, steps planned ahead whose tokens never leave the
    device) against the plain implementation; in bfloat16 a token may differ only at a near-tie of the plain logits."""
    from ferrum_b200.engine.api import Engine
    cfg, w = P.load(folders[name])
    prompts = [tokens_for(name, n, 60 + n, folders) for n in (23, 5, 41)]
    eng = Engine(folders[name], dtype=dtype, page_size=8, num_pages=40, max_batch_tokens=32, max_batch_seqs=4, chunk_size=16,
                 max_model_len=96)
    outs = eng.generate(prompts, max_new_tokens=20)
    compared = 0
    for p, got in zip(prompts, outs):
        if dtype == "float32":
            assert got == plain_generate(cfg, w, p, 20)
            continue
        seq = list(p)
        for t in got:
            margins = []
            logits = P.forward(cfg, w, seq, rounding_of(dtype), None, margins)[-1].numpy()
            if margins and float(torch.stack(margins).min()) < CLEAR_CALL:
                break           # a generated token routes by a close call: from here on the engine may differ rightly
            if t != int(np.argmax(logits)):
                assert logits.max() - logits[t] <= 0.2 * logits.std(), (len(seq), t)
            seq.append(t)
            compared += 1
    assert dtype == "float32" or compared >= 3, compared
    assert eng.stats()["pages_used"] == [0] * eng.cache.manager.n_groups


def test_preempted_requests_start_over(cuda, folders):
    """So few pages that requests are preempted and recomputed from their first token."""
    from ferrum_b200.engine.api import Engine
    cfg, w = P.load(folders["A"])
    prompts = [tokens_for("A", n, 80 + n) for n in (20, 17, 12)]
    eng = Engine(folders["A"], dtype="float32", page_size=8, num_pages=9, max_batch_tokens=64, max_batch_seqs=3, max_model_len=64)
    outs = eng.generate(prompts, max_new_tokens=16)
    assert eng.stats()["preemptions"] > 0
    for p, got in zip(prompts, outs):
        assert got == plain_generate(cfg, w, p, 16)


def test_trace_run_program_and_command_line(cuda, folders, tmp_path):
    """bin/trace_run as a user runs it on a Lelutar folder (a subprocess, JSON lines in, .f32 files
    out), and `ferrum generate` on the same folder against the plain implementation."""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    toks = tokens_for("A", 40, 16, folders)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[30:], "want": []}, {"id": "y", "tokens": toks[:2], "want": [1]}], "end": ["y"]},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[:1], "want": [0]}], "end": ["x"]}]
    out = tmp_path / "out"
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folders["A"], "--dtype", "float32",
                        "--out", str(out), "--max-tokens", "128"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=900)
    assert p.returncode == 0, p.stderr[-2000:]
    assert p.stdout.split() == ["done", "0", "done", "1", "done", "2"]
    ref = plain(folders["A"], "float32", toks + toks[:1])
    assert_close_f32(np.fromfile(out / "0.f32", dtype="<f4").reshape(2, -1), ref[[0, 29]], "trace_run step 0")
    assert_close_f32(np.fromfile(out / "1.f32", dtype="<f4").reshape(1, -1), ref[[1]], "trace_run step 1")
    assert_close_f32(np.fromfile(out / "2.f32", dtype="<f4").reshape(1, -1), ref[[40]], "trace_run step 2")
    cfg, w = P.load(folders["A"])
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "ferrum"), "generate", "--model", folders["A"], "--dtype", "float32",
                        "--prompt-tokens", ",".join(str(t) for t in toks[:12]), "--max-new-tokens", "6"],
                       capture_output=True, text=True, timeout=900)
    assert p.returncode == 0, p.stderr[-2000:]
    want = plain_generate(cfg, w, toks[:12], 6)
    assert ",".join(str(t) for t in want) in p.stdout.replace(" ", ""), (p.stdout, want)


def test_float16_prefill_and_decoding(cuda, folders):
    """The kernels with float16 storage (weights, activations, cached rows): a prompt, then single tokens, against the
    plain implementation rounding to float16 where the engine does."""
    toks = tokens_for("B", 150, 14, folders)
    ref, sure = plain(folders["B"], "float16", toks)
    r = Replay(session(folders["B"], "float16", 192))
    r.step([("a", toks[:100], "all")])
    for t in toks[100:]:
        r.step([("a", [t], "all")])
    assert_close_16bit(r.logits("a", len(toks))[sure], ref[sure], "B float16", "float16", c=C_MODEL["float16"])
