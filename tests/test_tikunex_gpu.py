"""Tikunex on the GPU against the plain implementation (plain_tikunex.py): every mechanism alone,
then whole models under every way of cutting the work, then generation through the engine."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_tikunex as P
from helpers import Replay, assert_close_16bit, assert_close_f32, mixed_schedule, pages_were_reused, peak_pages
from mixer_helpers import fill_part as fill_any_part, make_ctx, run_mixers_in_portions
from tikunex_configs import TIKUNEX, write_model

pytestmark = pytest.mark.gpu
TD = {"float32": torch.float32, "bfloat16": torch.bfloat16, "float16": torch.float16}
F64 = torch.float64

# 16-bit bound for whole models, in standard deviations of a row's logits: like the other design with routed experts and
# recurrences, this one answers to rounding strongly (routing weights multiply whole rows, recurrences and repeated
# passes carry every rounding along).  A lost key, page, state row or expert moves a row by about one.
C_MODEL = {"bfloat16": 0.25, "float16": 0.04}
CONFIGS = {k: v[0] for k, v in TIKUNEX.items()}
CLOSE_CALL = 0.01       # (spreads of a router's logits)
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
    return {name: write_model(cfg, str(tmp_path_factory.mktemp("tikunex_" + name)), seed) for name, (cfg, seed) in TIKUNEX.items()}


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
    name = name.replace("output.weight", "o").replace(".bias", ".b")
    return name[:-7] if name.endswith(".weight") else name


def fill_part(part, seed, td, prefix, std=0.3, fixed=None):
    return fill_any_part(part, seed, td, prefix, short_name, std, fixed)


# ================================================================= the attention kernel alone
def attention_reference(q, k, v, pos, H, G, scale, size, keep):
    """q [n, H, D] of queries at `pos`; k, v [keys, G, D]: float64 softmax over the window and the kept first keys."""
    out = np.zeros((len(pos), H, v.shape[2]))
    for t, p in enumerate(pos):
        seen = np.array([j for j in range(p + 1) if not size or p - j < size or j < keep])
        for h in range(H):
            g = h // (H // G)
            s = k[seen, g] @ q[t, h] * scale
            w = np.exp(s - s.max())
            out[t, h] = (w / w.sum()) @ v[seen, g]
    return out


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,D,page,size,keep", [(3, 1, 14, 8, 19, 3), (8, 2, 64, 16, 44, 16), (6, 2, 80, 16, 130, 1), (4, 4, 40, 32, 257, 150),
                                                  (2, 1, 200, 8, 7, 9), (1, 1, 32, 16, 1, 2), (4, 2, 64, 16, 300, 0), (4, 1, 32, 16, 5, 300)])
def test_attention_kernel_keeps_the_first_keys(cuda, dtype, H, G, D, page, size, keep):
    """Keys and values lie in pages scattered over the pool; a page that no query of the step may read is missing from the
    block table.  In turn one key dominates (it is scaled up and every query points at it): the one that the window just
    sees and one query later does not, the last kept one, the first one that is not kept.  Its value is the output exactly
    while it is seen.  A prompt portion, a single token over its whole range, a single token whose keys are cut among CTAs,
    and the sequence's first tokens."""
    from ferrum_b200.ops import lib as ops
    rng = np.random.default_rng(H * 1000 + D)
    n_keys, td, scale = 700, TD[dtype], 0.5
    n_pages = -(-n_keys // page)
    order = rng.permutation(n_pages + 5)[:n_pages]
    edge = (n_keys - 1 - size - 3) // page * page           # a page's first row, just inside the window of `edge + size - 1`
    hots = {"window": edge} | ({"kept": keep - 1} if keep else {}) | {"left": keep}
    for what, hot in hots.items():
        k = rng.standard_normal((n_keys, G, D)) * 0.3
        v = rng.standard_normal((n_keys, G, D))
        k[hot] *= 5.0
        kt, vt = torch.tensor(k, device="cuda").to(td), torch.tensor(v, device="cuda").to(td)
        k, v = kt.double().cpu().numpy(), vt.double().cpu().numpy()
        plane = torch.zeros(n_pages + 5, 2, G, page, D, device="cuda", dtype=td)
        for lp in range(n_pages):
            n = min(page, n_keys - lp * page)
            plane[order[lp], 0, :, :n] = kt[lp * page:lp * page + n].transpose(0, 1)
            plane[order[lp], 1, :, :n] = vt[lp * page:lp * page + n].transpose(0, 1)
        at = max(edge + size - 2, 0)                         # three queries around the window's edge at `edge`
        for pos0, n in ((n_keys - 40, 40), (n_keys - 1, 1), (at, 3), (max(keep + size - 2, 0), 3), (0, 9)):
            n = min(n, n_keys - pos0)
            first = max(0, pos0 - size + 1) // page
            table = [int(order[lp]) if lp >= first or lp * page < keep else -1 for lp in range(n_pages)]
            ctx = make_ctx([(pos0, n)], widths=[[table]])
            pos = list(range(pos0, pos0 + n))
            q = np.tile(k[hot].repeat(H // G, axis=0).reshape(1, H * D) * 4.0, (n, 1)) + rng.standard_normal((n, H * D)) * 0.1
            qt = torch.tensor(q, device="cuda").to(td)
            ref = attention_reference(qt.double().cpu().numpy().reshape(n, H, D), k, v, pos, H, G, scale, size, keep)
            for mode in (["rows", "tokens", "split"] if n == 1 else ["rows", "tokens"]):
                out = torch.full((n, H * D), float("nan"), device="cuda")
                part, slots, q_start = None, 0, None
                if mode == "split":
                    split = ops.attention_generic_split()
                    slots = min(n_keys, size + split) // split + 2 + -(-keep // split)
                    part = torch.full((n * H * slots * (D + 2),), float("nan"), device="cuda")
                if mode == "tokens":
                    q_start = ctx.q_start
                ops.attention_generic(qt, out, n, ctx.positions, ctx.req_of_token, ctx.block_tables[0], plane, plane.stride(0), page,
                                      H, G, D, scale, size, ctx.err, part=part, split_slots=slots, q_start=q_start, n_reqs=1,
                                      keep_first=keep, out_scale=-1.5)
                got = out.double().cpu().numpy().reshape(n, H, D) / -1.5
                assert ctx.err.item() == 0, (what, pos0, n, mode)
                assert np.abs(got - ref).max() < (2e-5 if dtype == "float32" else 2e-2) * max(np.abs(ref).max(), 0.05), (what, pos0, n, mode)
                for i, p in enumerate(pos):
                    seen = p >= hot and (p - hot < size or hot < keep)
                    if p - hot < size and p < size:
                        continue                             # (few keys in sight: nothing far to tell apart)
                    near = np.abs(got[i, 0] - v[hot, 0]).max()
                    assert (near < 0.05 * np.abs(v).max()) == seen, (what, pos0, i, mode)


# ================================================================= mixers alone, whole and in portions
CUTS = ([61], [20, 1, 1, 2, 30, 7], [2] * 30 + [1], [1] * 61)


def check_mixers(mixers, refs, xs, td, dtype, page=8, cuts=CUTS):
    for cut in cuts:
        got = run_mixers_in_portions(mixers, xs, cut, td, page=page, max_tokens=max(128, xs[0].shape[0]))
        for i, ref in enumerate(refs):
            assert torch.isfinite(got[i]).all(), (cut, i)
            assert (got[i] - ref).abs().max() < (2e-4 if dtype == "float32" else 4e-2) * ref.abs().max(), (cut, i)


def inputs(n, E, td, seed=10):
    g = torch.Generator(device="cuda").manual_seed(seed)
    return torch.randn(n, E, device="cuda", generator=g).to(td)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,D,Dv,size,keep", [(3, 1, 10, 14, 19, 3), (8, 2, 64, 64, 24, 9), (4, 4, 12, 6, 17, 0), (2, 2, 6, 6, 1, 1), (6, 2, 80, 40, 5, 20),
                                                (4, 2, 8, 24, 0, 0)])
def test_window_attention_with_kept_keys_alone(cuda, dtype, H, G, D, Dv, size, keep):
    """Through pages that are given back and pages that stay, in portions that cut windows, pages and the kept keys anywhere."""
    from ferrum_b200.parts import ShapedAttention
    td, E = TD[dtype], 40
    mixer = ShapedAttention(E, H, G, D, Dv, td, 0.45, window=size, keep_first=keep)
    w = fill_part(mixer, 9, td, "p.")
    x = inputs(61, E, td)
    c = {"heads": H, "kv_heads": G, "dim": D, "vdim": Dv, "scale": 0.45, "mask": {"size": size, "keep_first": keep}}
    rd = rounding_of(dtype)
    ref = P.matmul(P.attention(x.double().cpu(), w, "p.", c, rd), w["p.o"], rd)
    check_mixers([mixer], [ref], [x], td, dtype)
    if keep and size:
        lost = P.matmul(P.attention(x.double().cpu(), w, "p.", dict(c, mask={"size": size, "keep_first": keep - 1}), rd), w["p.o"], rd)
        assert (lost - ref).abs().max() > 1e-2 * ref.abs().max()              # (the last kept key matters to the result)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,D,Dv,tau,rank", [(3, 10, 14, 4.0, 5), (2, 64, 32, 16.0, 16), (1, 5, 33, 1.0, 2), (4, 32, 64, 2.0, 24), (2, 100, 72, 8.0, 130),
                                             (1, 200, 9, 32.0, 8)])
def test_gated_linear_attention_alone(cuda, dtype, H, D, Dv, tau, rank):
    from ferrum_b200.parts import GatedLinearAttention
    td, E, eps = TD[dtype], 40, 1e-5
    mixer = GatedLinearAttention(E, H, D, Dv, tau, eps, td, rank)
    # biases from channels that forget nearly all to channels that keep nearly all
    w = fill_part(mixer, 11, td, "p.", std=0.5, fixed={"a2.bias": torch.linspace(-9.0, 9.0, H * D)})
    x = inputs(61, E, td, seed=12)
    ref = P.gla(x.double().cpu(), w, "p.", {"heads": H, "dim": D, "vdim": Dv, "tau": tau}, eps, rounding_of(dtype))
    check_mixers([mixer], [ref], [x], td, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,D,rank,E", [(5, 6, 3, 52), (2, 64, 8, 64), (1, 4, 1, 32), (3, 33, 7, 40), (2, 130, 16, 72), (8, 32, 40, 128)])
def test_time_mixing_alone(cuda, dtype, H, D, rank, E):
    """The recurrence behind token shifts: the row before a portion's first token and the memory carried between steps."""
    from ferrum_b200.parts import TimeMixing
    td, eps = TD[dtype], 1e-5
    mixer = TimeMixing(E, H, D, eps, td, rank)
    fixed = {"w0": torch.linspace(-8.0, 3.0, H * D), "u": torch.linspace(-2.0, 4.0, H * D).reshape(H, D)}
    w = fill_part(mixer, 13, td, "p.", std=0.4, fixed=fixed)
    x = inputs(61, E, td, seed=14)
    rd = rounding_of(dtype)
    c = {"heads": H, "dim": D}
    ref = P.matmul(P.rwkv(x.double().cpu(), w, "p.", c, eps, rd), w["p.o"], rd)
    check_mixers([mixer], [ref], [x], td, dtype)
    w0 = dict(w, **{"p.u": torch.zeros(H, D, dtype=F64)})
    assert (P.matmul(P.rwkv(x.double().cpu(), w0, "p.", c, eps, rd), w["p.o"], rd) - ref).abs().max() > 1e-2 * ref.abs().max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("left_scale,right_scale", [(0.7, 1.6), (-2.0, 0.25), (1.0, 0.0)])
def test_scaled_pair_alone(cuda, dtype, left_scale, right_scale):
    """Window attention and the recurrence with one output product for both: pages AND a state, and the two factors."""
    from ferrum_b200.parts import ScaledPairMixer, ShapedAttention, TimeMixing
    td, E, eps = TD[dtype], 40, 1e-5
    for left, right in (((3, 1, 10, 14), (5, 6)), ((4, 2, 16, 16), (2, 32)), ((2, 2, 24, 8), (1, 8))):
        H, G, D, Dv = left
        att = ShapedAttention(E, H, G, D, Dv, td, 0.4, window=19, keep_first=3)
        mixer = ScaledPairMixer(E, att, TimeMixing(E, *right, eps, td, 4), left_scale, right_scale, td)
        need = mixer.cache_need()
        assert need.paged is not None and need.paged.keep_first == 3 and need.state is not None
        w = fill_part(mixer, 15, td, "p.")
        x = inputs(61, E, td, seed=16)
        c = {"left": {"heads": H, "kv_heads": G, "dim": D, "vdim": Dv, "scale": 0.4, "mask": {"size": 19, "keep_first": 3}},
             "right": {"heads": right[0], "dim": right[1]}, "left_scale": left_scale, "right_scale": right_scale}
        ref = P.parallel_mixer(x.double().cpu(), w, "p.", c, eps, rounding_of(dtype))
        check_mixers([mixer], [ref], [x], td, dtype)


# ================================================================= the walk and what surrounds it
@pytest.mark.parametrize("bonus", [False, True])
@pytest.mark.parametrize("H,D,Dv", [(2, 5, 7), (1, 32, 300), (3, 40, 24), (2, 64, 64), (1, 100, 33), (2, 128, 128), (1, 130, 20), (1, 256, 12)])
def test_walk_in_one_piece_and_in_segments(cuda, bonus, H, D, Dv):
    """Unequal portions in one batch (one of a single token, one that fills its last segment), each from a state of its own:
    in one piece, and cut into segments of several lengths that run side by side.  Channels that forget everything at
    once, that keep everything, and that decay so slowly that a token at the front still matters at the end."""
    from ferrum_b200.engine.batch import StepContext, StepEntry
    from ferrum_b200.ops import lib as ops
    lens, slots = [70, 1, 32, 129, 2], [3, 0, 4, 1, 2]
    T = sum(lens)
    g = torch.Generator(device="cuda").manual_seed(D)
    ctx = StepContext("cuda", 512, 6, [])
    ctx.fill([StepEntry(s, 0, [1] * n) for s, n in zip(slots, lens)], [])
    qkv = torch.randn(T, 2 * H * D + H * Dv + 8, device="cuda", generator=g)
    dec = torch.rand(T, H * D, device="cuda", generator=g)
    dec[:, 0::4], dec[:, 1::4] = 0.0, 1.0
    dec[:, 2::4] = 1.0 - 1e-3 * dec[:, 2::4]
    u = torch.randn(H, D, device="cuda", generator=g) if bonus else None
    start = torch.randn(6, H * D * Dv + 4, device="cuda", generator=g)
    q, k, v = qkv[:, :H * D], qkv[:, H * D:2 * H * D], qkv[:, 2 * H * D:2 * H * D + H * Dv]
    scale = D ** -0.5
    # float64, token by token
    ref, final, t = torch.zeros(T, H * Dv, dtype=F64), {}, 0
    for n, s in zip(lens, slots):
        S = start[s, :H * D * Dv].double().cpu().view(H, D, Dv)
        for i in range(t, t + n):
            qi, ki, ai = (m[i].double().cpu().view(H, D) for m in (q, k, dec))
            kv = ki[:, :, None] * v[i].double().cpu().view(H, 1, Dv)
            if bonus:
                o = torch.einsum("hdv,hd->hv", S + u.double().cpu()[:, :, None] * kv, qi)
                S = ai[:, :, None] * S + kv
            else:
                S = ai[:, :, None] * S + kv
                o = torch.einsum("hdv,hd->hv", S, qi)
            ref[i] = o.reshape(-1) * scale
        final[s] = S.reshape(-1)
        t += n
    for length in (None, 0, 1, 7, 16, 32, 43, 128, 500):
        state = start.clone()
        out = torch.full((T, H * Dv), float("nan"), device="cuda")
        cut = None if length is None else (length, sum(-(-n // length) for n in lens) if length else 0)
        ops.channel_decay(q, k, v, dec, T, ctx, H, D, Dv, state, out, bonus=u, out_scale=scale, segments=cut)
        assert (out.double().cpu() - ref).abs().max() < 3e-5 * ref.abs().max(), length
        for s in slots:
            assert (state[s, :H * D * Dv].double().cpu() - final[s]).abs().max() < 2e-5 * final[s].abs().max(), (length, s)
        assert torch.equal(state[5], start[5]) and torch.equal(state[:, H * D * Dv:], start[:, H * D * Dv:])     # nobody else's memory
    assert ops.channel_decay_segments(ctx, 16, 128, 128)[0] in (0, 32, 48)


def test_segments_are_chosen_from_the_sizes_of_the_batch(cuda):
    from ferrum_b200.engine.batch import StepContext, StepEntry
    from ferrum_b200.ops import lib as ops
    ctx = StepContext("cuda", 4096, 8, [])
    ctx.fill([StepEntry(i, 0, [1]) for i in range(8)], [])
    assert ops.channel_decay_segments(ctx, 16, 128, 128) == (0, 0)          # single tokens: never cut, so a captured step is not
    ctx.fill([StepEntry(0, 0, [1] * 2048)], [])
    length, n = ops.channel_decay_segments(ctx, 16, 128, 128)
    assert 32 <= length <= 512 and n == -(-2048 // length)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,N,rank", [(1, 40, 3), (9, 70, 16), (33, 128, 64), (100, 66, 130), (64, 8, 300), (8, 33, 257)])
def test_decays_from_a_low_rank_projection(cuda, dtype, T, N, rank):
    """Both maps at moderate and at extreme arguments (a decay of 0 or 1 and nothing undefined)."""
    from ferrum_b200.ops import lib as ops
    g = torch.Generator(device="cuda").manual_seed(N)
    rows = torch.randn(T, rank + 5, device="cuda", generator=g)
    w2 = (torch.randn(N, rank, device="cuda", generator=g) / rank ** 0.5).to(TD[dtype])
    bias = torch.linspace(-6.0, 6.0, N, device="cuda")
    bias[0], bias[-1] = -200.0, 200.0
    low = rows[:, :rank]
    for kind, tanh, tau in (("exp_exp", True, 1.0), ("exp_exp", False, 1.0), ("sigmoid_root", False, 16.0), ("sigmoid_root", True, 0.5)):
        out = torch.full((T, N), float("nan"), device="cuda")
        ops.channel_decay_gate(low, w2, bias, kind, T, out, tanh=tanh, tau=tau)
        z = (torch.tanh(low.double()) if tanh else low.double()) @ w2.double().T + bias.double()
        ref = torch.exp(-torch.exp(z)) if kind == "exp_exp" else torch.exp(-torch.nn.functional.softplus(-z) / tau)
        assert torch.isfinite(out).all() and (out.double() - ref).abs().max() < 2e-5, (kind, tanh)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E,n", [(52, 5), (33, 1), (640, 3)])
def test_blends_with_the_row_before(cuda, dtype, E, n):
    """Unequal portions in one batch; the row before a portion's first token is the request's own, and its last row is left."""
    from ferrum_b200.engine.batch import StepContext, StepEntry
    from ferrum_b200.ops import lib as ops
    td = TD[dtype]
    lens, slots = [4, 1, 9, 2], [2, 0, 3, 1]
    T = sum(lens)
    g = torch.Generator(device="cuda").manual_seed(E)
    ctx = StepContext("cuda", 64, 5, [])
    ctx.fill([StepEntry(s, 7, [1] * k) for s, k in zip(slots, lens)], [])
    x = torch.randn(T, E, device="cuda", generator=g).to(td)
    mu = torch.rand(n, E, device="cuda", generator=g)
    state = torch.randn(5, E + 12, device="cuda", generator=g)
    before = state.clone()
    out = torch.full((n, T, E), float("nan"), device="cuda", dtype=td)
    counts = torch.full((3,), -1, dtype=torch.int32, device="cuda")
    ops.token_shift_mix(x, mu, T, ctx, state[:, 12:], out, counts)
    t = 0
    for k, s in zip(lens, slots):
        rows = torch.cat([before[s, 12:][None].double(), x[t:t + k].double()])
        ref = rows[None, 1:] + (rows[None, :-1] - rows[None, 1:]) * mu.double()[:, None]
        assert (out[:, t:t + k].double() - ref).abs().max() < (1e-6 if dtype == "float32" else 2e-2)
        assert torch.equal(state[s, 12:], x[t + k - 1].float())
        t += k
    assert torch.equal(state[4], before[4]) and torch.equal(state[:, :12], before[:, :12]) and counts.tolist() == [T] * 3


# ================================================================= the feed-forward and the norms alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E,F,n_exp,top,T", [(52, 20, 5, 3, 37), (128, 64, 6, 2, 300), (40, 24, 1, 1, 9), (64, 32, 16, 4, 70), (72, 100, 4, 4, 11),
                                             (128, 128, 4, 2, 1000), (256, 80, 7, 1, 2), (64, 48, 40, 8, 16)])
def test_routed_feed_forward_alone(cuda, dtype, E, F, n_exp, top, T):
    """Biased logits choose and a softmax over the chosen ones weighs; the sum joins the residual rows, of which a copy in the
    compute type is left: sizes that take each of the product kernels and both routing kernels."""
    from ferrum_b200.engine.batch import StepContext, StepEntry
    from ferrum_b200.parts import RoutedFeedForward
    td = TD[dtype]
    ffn = RoutedFeedForward(E, F, n_exp, top, td, act="silu", scores="chosen_softmax", scale_input=False, router_bias=True)
    fixed = {"router.bias": torch.linspace(-2.0, 2.0, n_exp) if n_exp > 1 else torch.ones(1)}
    w = fill_part(ffn, 21, td, "f.", std=0.4, fixed=fixed)
    x = inputs(T, E, td, seed=22)
    margins = []
    ref = P.mixture(x.double().cpu(), w, "f.", {"router": {"experts": n_exp, "top": top}}, rounding_of(dtype), margins)
    ctx = StepContext("cuda", 1024, 4, [])
    ctx.fill([StepEntry(0, 0, list(range(T)))], [])
    g = torch.Generator(device="cuda").manual_seed(23)
    h0 = torch.randn(T, E, device="cuda", generator=g)
    h = h0.clone()
    copy = torch.full((T, E), float("nan"), device="cuda", dtype=td)
    ffn.forward(x, ctx, h, copy=copy)
    assert ctx.err.item() == 0 and torch.equal(copy, h.to(td))
    sure = (margins[0] > (1e-6 if dtype == "float32" else CLEAR_CALL)).numpy()
    assert sure.any() and sure.mean() >= min(0.5, 1.0 - 1.0 / T)
    got = (h - h0).double().cpu()
    assert (got - ref)[sure].abs().max() < (2e-4 if dtype == "float32" else 4e-2) * ref.abs().max()
    y = torch.full((T, E), float("nan"), device="cuda")
    ffn.forward(x, ctx, y, accumulate=False)
    assert (y - (h - h0)).abs().max() < 1e-4 * ref.abs().max()


@pytest.mark.parametrize("T", [2, 40])
def test_router_by_hand(cuda, T):
    """The bias enters before the choice and the weights; a tie goes to the lower index; rows are gathered by expert."""
    from ferrum_b200.ops import lib as ops
    logits = torch.tensor([[1.0, 0.0, 2.0], [0.5, 0.5, 0.5]] * (T // 2), device="cuda")
    bias = torch.tensor([0.0, 3.0, 0.0], device="cuda")
    x = torch.arange(T, device="cuda", dtype=torch.float32)[:, None].repeat(1, 8)
    expert_of, rank_of, row_of = (torch.full((T * 2,), -7, dtype=torch.int32, device="cuda") for _ in range(3))
    weight_of, counts, xg = torch.zeros(T * 2, device="cuda"), torch.full((3,), 9, dtype=torch.int32, device="cuda"), torch.zeros(T * 2, 8, device="cuda")
    ops.moe_route(logits, T, 3, 2, x, False, expert_of, rank_of, weight_of, counts, xg, row_of, scores="chosen_softmax", bias=bias)
    assert expert_of.view(T // 2, 4).tolist() == [[1, 2, 1, 0]] * (T // 2)
    a, b = torch.softmax(torch.tensor([3.0, 2.0]), 0), torch.softmax(torch.tensor([3.5, 0.5]), 0)
    assert torch.allclose(weight_of.cpu().view(T // 2, 4), torch.cat([a, b]).repeat(T // 2, 1), rtol=1e-5)
    assert counts.tolist() == [T // 2, T, T // 2] and sorted(row_of.tolist()) == list(range(2 * T))
    for pair in range(2 * T):
        e, row = expert_of[pair].item(), row_of[pair].item()
        assert sum(counts.tolist()[:e]) <= row < sum(counts.tolist()[:e + 1]) and xg[row, 0].item() == pair // 2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E,T", [(52, 9), (256, 70), (1030, 3), (2048, 80)])
def test_norms_alone(cuda, dtype, E, T):
    """The embedding's norm (and its copy into wider rows), the branch's sum that goes on to the next norm, and the gated norm
    of heads with silu and a factor."""
    from ferrum_b200.ops import lib as ops
    td, eps = TD[dtype], 1e-3
    g = torch.Generator(device="cuda").manual_seed(E)
    tol = 1e-5 if dtype == "float32" else 2e-2
    table = torch.randn(31, E, device="cuda", generator=g).to(td)
    ids = torch.randint(0, 31, (T,), device="cuda", generator=g).int()
    w, w2 = (1.0 + 0.3 * torch.randn(E, device="cuda", generator=g) for _ in range(2))
    err = torch.zeros(1, dtype=torch.int32, device="cuda")
    h, rows = torch.full((T, E), float("nan"), device="cuda"), torch.zeros(T, 2 * E, device="cuda", dtype=td)
    ops.embedding_norm(table, ids, w, eps, h, err, copy=rows[:, E:])
    ref = P.rms(table.double()[ids.long()], eps) * w.double()
    assert (h.double() - ref).abs().max() < 1e-5 and torch.equal(rows[:, E:], h.to(td)) and not rows[:, :E].any() and err.item() == 0
    y = torch.randn(T, E, device="cuda", generator=g) * 3.0
    want = h.double() + 0.5 * P.rms(y.double(), eps) * w2.double()
    h2, out = h.clone(), torch.full((T, E), float("nan"), device="cuda", dtype=td)
    if ops.norm_scaled_add_can_norm(h2, y, w2, w, out):
        ops.norm_scaled_add(h2, y, w2, 0.5, eps, T, norm=(w, 1e-5, out))
        assert (out.double() - P.rms(want, 1e-5) * w.double()).abs().max() < tol * 8
    else:
        assert E % 4
        ops.norm_scaled_add(h2, y, w2, 0.5, eps, T)
    assert (h2.double() - want).abs().max() < 2e-5
    H, Dv = 2, E // 2
    o, gate = torch.randn(T, H * Dv, device="cuda", generator=g), torch.randn(T, H * Dv + 4, device="cuda", generator=g) * 4.0
    for per_head in (False, True):
        wn = 1.0 + 0.3 * torch.randn(H * Dv if per_head else Dv, device="cuda", generator=g)
        got = torch.zeros(T, H * Dv + 8, device="cuda", dtype=td)
        ops.head_gate_norm(o, gate[:, 4:], wn, eps, T, H, Dv, got[:, 8:], gate_act="silu", out_scale=-0.7)
        z = gate[:, 4:].double().view(T, H, Dv)
        ref = -0.7 * P.rms(o.double().view(T, H, Dv), eps) * wn.double().view(H if per_head else 1, Dv) * z * torch.sigmoid(z)
        assert (got[:, 8:].double().view(T, H, Dv) - ref).abs().max() < tol * ref.abs().max() and not got[:, :8].any()


@pytest.mark.parametrize("dtype", ["bfloat16", "float16"])
@pytest.mark.parametrize("M,N,K", [(1, 3, 64), (8, 16, 2048), (13, 129, 264), (64, 64, 4096), (100, 7, 1032), (300, 16, 72), (16, 512, 128)])
def test_product_of_few_features(cuda, dtype, M, N, K):
    """Stored as float32, in the compute type, and through the token input's gate; rows may be parts of wider ones."""
    from ferrum_b200.ops import lib as ops
    td = TD[dtype]
    g = torch.Generator(device="cuda").manual_seed(K)
    wide = torch.randn(M, K + 8, device="cuda", generator=g).to(td)
    x, w = wide[:, 8:], torch.randn(N, K, device="cuda", generator=g).to(td)
    assert ops.thin_linear_supported(x, w, M)
    err = torch.zeros(1, dtype=torch.int32, device="cuda")
    ref = x.double() @ w.double().T
    f32, f16 = torch.full((M, N + 3), float("nan"), device="cuda"), torch.zeros(M, N, device="cuda", dtype=td)
    ops.thin_linear(x, w, f32, M, err)
    assert (f32[:, :N].double() - ref).abs().max() < 1e-5 * K ** 0.5 * 4 and torch.isnan(f32[:, N:]).all()
    ops.thin_linear(x, w, f16, M, err)
    assert torch.equal(f16, f32[:, :N].to(td))
    table = torch.randn(19, N + 6, device="cuda", generator=g).to(td)
    ids = torch.randint(0, 19, (M,), device="cuda", generator=g).int()
    ops.thin_linear(x * 0.01, w, f16, M, err, table=table, offset=5, token_ids=ids)
    ref = P.gelu_tanh((x * 0.01).double().cpu() @ w.double().cpu().T) * table[:, 5:5 + N].double().cpu()[ids.long().cpu()]
    assert (f16.double().cpu() - ref).abs().max() < 1e-2 * ref.abs().max() and err.item() == 0
    one = torch.zeros(1, N + 3, device="cuda")                  # a row alone gives the row of the batch, bit for bit
    if M <= 64:
        ops.thin_linear(x[M - 1:M], w, one, 1, err)
        assert torch.equal(one[:, :N], f32[M - 1:M, :N])


# ================================================================= whole models, every way of cutting the work
CASES = [(n, d) for n in ("A", "B") for d in ("float32", "bfloat16")]


@pytest.mark.parametrize("name,dtype", CASES + [("C", "float32"), ("C", "bfloat16"), ("D", "float32"), ("D", "bfloat16")])
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


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_residual_rows_after_every_layer_run(cuda, folders, name):
    toks = tokens_for(name, 25, 11, folders)
    cfg, w = P.load(folders[name])
    taps = []
    P.forward(cfg, w, toks, None, taps)
    s = session(folders[name], "float32", 64)
    got = []
    s.model.on_run = lambda k, h: got.append(h[:len(toks)].double().cpu())
    s.run_step({"step": 0, "entries": [{"id": "a", "tokens": toks, "want": []}], "end": ["a"]})
    assert len(got) == len(taps) == len(P.run_order(cfg))
    for k, (g, t) in enumerate(zip(got, taps)):
        assert (g - t).abs().max() < 1e-4 * t.abs().max(), k


@pytest.mark.parametrize("name,dtype", CASES + [("D", "float32")])
def test_prefill_then_long_decoding_past_every_window(cuda, folders, name, dtype):
    """30 tokens at once, then 120 one by one: windows pass over decoded tokens, pages behind them are given back while the
    first ones stay, the states are carried through a captured graph."""
    toks = tokens_for(name, 150, 12, folders)
    ref = plain(folders[name], dtype, toks)
    s = session(folders[name], dtype, 160, page_size=8)
    r = Replay(s)
    r.step([("a", toks[:30], "all")])
    for t in toks[30:]:
        r.step([("a", [t], "all")])
    close(r.logits("a", len(toks)), ref, dtype, f"{name} prefill+decode")
    assert s.runner.graph_replays > 0          # single tokens ran from a captured graph
    left = CONFIGS[name]["layers"][0]["mixer"].get("left") or CONFIGS[name]["layers"][1]["mixer"]["left"]
    table = s.cache.manager.table(0, s.slots["a"])
    kept, first = -(-left["mask"]["keep_first"] // 8), (150 - left["mask"]["size"] + 1) // 8
    assert [p >= 0 for p in table[:19]] == [lp < kept or lp >= first for lp in range(19)]


def test_token_by_token_from_the_first(cuda, folders):
    toks = tokens_for("A", 70, 17, folders)
    ref = plain(folders["A"], "float32", toks)
    r = Replay(session(folders["A"], "float32", 80, page_size=8))
    for t in toks:
        r.step([("a", [t], "all")])
    close(r.logits("a", len(toks)), ref, "float32", "A token by token")


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
    together: finished requests' pages and state rows go to later ones (which must start from zero)."""
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
    """700 tokens at once (the recurrences in segments) equal the same in portions and the plain run, and two prompts that
    differ in one early token still differ at the end."""
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
        assert d[5] > 1e-3 and d[-20:].min() > 1e-4


def plain_generate(cfg, w, prompt, n, rd=None):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(P.forward(cfg, w, seq, rd)[-1].argmax()))
    return seq[len(prompt):]


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("B", "float32"), ("B", "bfloat16"), ("D", "float32")])
def test_greedy_generation_through_the_engine(cuda, folders, name, dtype):
    """Engine.generate (scheduler, sampler, chunked prompts, several requests) against the plain
    implementation; in bfloat16 a token may differ only at a near-tie of the plain logits."""
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


def test_trace_run_program_and_command_line(cuda, folders, tmp_path):
    """bin/trace_run as a user runs it on a Tikunex folder (a subprocess, JSON lines in, .f32 files
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
    """The kernels with float16 storage (weights, activations, cached keys and values): a prompt, then
    single tokens, against the plain implementation rounding to float16 where the engine does."""
    toks = tokens_for("B", 150, 14, folders)
    ref, sure = plain(folders["B"], "float16", toks)
    r = Replay(session(folders["B"], "float16", 192))
    r.step([("a", toks[:100], "all")])
    for t in toks[100:]:
        r.step([("a", [t], "all")])
    assert_close_16bit(r.logits("a", len(toks))[sure], ref[sure], "B float16", "float16", c=C_MODEL["float16"])
