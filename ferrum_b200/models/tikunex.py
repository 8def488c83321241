"""The Tikunex decoder, built from parts, and its entry in the registry.

Token embedding through an RMS norm (every norm of the residual stream stores its weight around zero); layers
that are `PreNormBlock`s with a per-layer token input from a second embedding table, around one of two mixers
and a routed feed-forward:

  mixers         gated linear attention with one decay per head and key channel; or two mixers whose sum is
                 weighted by two fixed factors: attention without positions in a sliding window that keeps the
                 sequence's first keys, and an RWKV-style recurrence behind token shifts
  feed-forward   a mixture of silu-gated units, the largest biased logits choosing and a softmax over them
                 weighting

then a norm and an output matrix of its own.  A range of layers may run several times in a row with the same
weights: the schedule names those blocks once per pass, every pass has cache planes and state rows of its own
and starts by replacing the residual rows by W [x; embedding output] (`RestartInput`).

The checkpoint's tensor names are short (`embed`, `embed.norm`, `loop.in`, `side.embed`, `l<i>.norm1`, `l<i>.mix.q`,
`l<i>.mix.left.q`, `l<i>.mix.right.mu.r`, `l<i>.mlp.e<j>.gate`, `l<i>.side.gate`, `final.norm`, `head`); `file_names`
maps them onto the canonical names that the parts declare.
"""
from __future__ import annotations

from ..config.registry import Architecture, register
from ..config.tikunex import GlaSpec, TikunexConfig
from ..parts import (GatedLinearAttention, OutputHead, PreNormBlock, RestartInput, RMSNorm, RoutedFeedForward, ScaledPairMixer,
                     ShapedAttention, TimeMixing, TokenEmbedding, TokenSideInput, TokenSideTable)
from .decoder import DecoderModel, Run


def build_tikunex(config: TikunexConfig, dtype, device, max_positions=None):
    c = config
    E = c.n_embd

    def norm(out_dtype=dtype):
        return RMSNorm(E, c.norm_eps, out_dtype, zero_centred=True)

    side_table = TokenSideTable(c.n_vocab, c.n_layer * c.side_dim) if c.side_dim else None
    blocks = []
    for i, layer in enumerate(c.layers):
        m = layer.mixer
        if isinstance(m, GlaSpec):
            mixer = GatedLinearAttention(E, m.heads, m.dim, m.vdim, m.tau, c.norm_eps, dtype, m.decay_rank)
        else:
            a, r = m.left, m.right
            left = ShapedAttention(E, a.heads, a.kv_heads, a.dim, a.vdim, dtype, a.scale, eps=c.norm_eps, window=a.window,
                                   keep_first=a.keep_first)
            mixer = ScaledPairMixer(E, left, TimeMixing(E, r.heads, r.dim, c.norm_eps, dtype, r.decay_rank), m.left_scale,
                                    m.right_scale, dtype)
        ffn = norm2 = None
        p = layer.mlp
        if p is not None:
            norm2 = norm()
            ffn = RoutedFeedForward(E, p.ff, p.experts, p.top, dtype, act="silu", scores="chosen_softmax", scale_input=False,
                                    router_bias=True)
        side = TokenSideInput(E, c.side_dim, i * c.side_dim, side_table, c.norm_eps, dtype) if side_table is not None else None
        blocks.append(PreNormBlock(norm(), mixer, norm2, ffn, names=("norm1.", "mix.", "norm2.", "mlp.", "side."), side=side))
    entries = [("loop_in.", RestartInput(E, dtype))] if c.loop is not None else []
    schedule = [Run(i, before=0 if enters else None) for i, enters in c.run_order()]
    emb = TokenEmbedding(c.n_vocab, E, norm=norm(), restart_dtype=dtype if entries else None)
    head = OutputHead(c.n_vocab, E, tied=False)
    shared = [("side_embd.", side_table)] if side_table is not None else []
    return DecoderModel(c, dtype, emb, None, blocks, norm(), head, schedule=schedule, shared=shared, entries=entries)


_GLA = {"q": "q.weight", "k": "k.weight", "v": "v.weight", "g": "g.weight", "o": "o.weight", "norm": "norm.weight", "a1": "a1.weight",
        "a2": "a2.weight", "a2.b": "a2.bias"}
_LEFT = {"q": "q.weight", "k": "k.weight", "v": "v.weight", "o": "output.weight"}
_RIGHT = {"r": "r.weight", "k": "k.weight", "v": "v.weight", "g": "g.weight", "w1": "w1.weight", "w2": "w2.weight", "w0": "w0", "u": "u",
          "norm": "norm.weight", "o": "o.weight", **{"mu." + s: "mu." + s for s in TimeMixing.STREAMS}}
_UNIT = ("gate", "up", "down")
_SIDE = ("gate", "proj", "norm")


def file_names(config: TikunexConfig):
    """{name in the checkpoint: canonical name}, for the tensors this configuration has."""
    out = {"embed": "token_embd.weight", "embed.norm": "token_embd.norm.weight", "final.norm": "output_norm.weight", "head": "output.weight"}
    if config.loop is not None:
        out["loop.in"] = "loop_in.weight"
    if config.side_dim:
        out["side.embed"] = "side_embd.weight"
    for i, layer in enumerate(config.layers):
        names = {"norm1": "norm1.weight"}
        if isinstance(layer.mixer, GlaSpec):
            names.update({"mix." + k: "mix." + v for k, v in _GLA.items()})
        else:
            names.update({"mix.left." + k: "mix.left." + v for k, v in _LEFT.items()})
            names.update({"mix.right." + k: "mix.right." + v for k, v in _RIGHT.items()})
        if layer.mlp is not None:
            names.update({"norm2": "norm2.weight", "mlp.router": "mlp.router.weight", "mlp.router.b": "mlp.router.bias"})
            for e in range(layer.mlp.experts):
                names.update({f"mlp.e{e}.{k}": f"mlp.e{e}.{k}.weight" for k in _UNIT})
        if config.side_dim:
            names.update({"side." + k: f"side.{k}.weight" for k in _SIDE})
        for short, ours in names.items():
            out[f"l{i}.{short}"] = f"blk.{i}.{ours}"
    return out


register(Architecture("Tikunex", TikunexConfig.from_dict, build_tikunex, file_names), "tikunex")
