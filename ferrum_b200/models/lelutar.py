"""The Lelutar decoder, built from parts, and its entry in the registry.

Scaled token embedding plus a row of a hashed table of token pairs (the token before a portion is part of a request's
state); layers that are `PreNormBlock`s whose norms are a dynamic tanh, around one of three mixers and an ungated
feed-forward (the square of relu), dense or routed:

  mixers         grouped-query attention with biases and a rotation of neighbouring elements (frequencies and magnitude by
                 the YaRN rule); attention over a cached latent with a sink in the softmax and a gate per head, without
                 positions or with a rotated key part that all heads share
  feed-forward   one unit, or a mixture: sigmoid scores, a correction for the choice alone, choice limited to the best
                 groups of experts, weights renormalised

then a norm and an output matrix of its own.  A layer with `weights_of` is a further run of another layer's block with a
cache plane of its own.

The checkpoint's tensor names are short (`embed`, `bigram`, `l<i>.norm1`, `l<i>.norm1.alpha`, `l<i>.mix.q.b`,
`l<i>.mlp.e<j>.up`, `final.norm`, `head`); `file_names` maps them onto the canonical names that the parts declare.
"""
from __future__ import annotations

from ..config.lelutar import AttentionSpec, DenseMlpSpec, LelutarConfig
from ..config.registry import Architecture, register
from ..parts import (BigramTable, DynamicTanh, LatentAttention, OutputHead, PlainUnit, PreNormBlock, RotaryEmbedding, RoutedFeedForward,
                     ShapedAttention, TokenEmbedding)
from ..parts.rope import yarn
from .decoder import DecoderModel, Run

RENORM_EPS = 1e-20      # added to the sum that the routing weights are divided by


def build_lelutar(config: LelutarConfig, dtype, device, max_positions=None):
    c = config
    E = c.n_embd
    n_pos = int(max_positions or c.n_ctx_train)
    tables = {}     # (head size, rotation) -> rotary table, shared by the layers that turn alike

    def rotary(dim, r):
        if r is None:
            return None
        if (dim, r) not in tables:
            f, mag = None, 1.0
            if r.scaling is not None:
                s = r.scaling
                f, mag = yarn(r.dims, r.base, s.factor, s.original, s.fast, s.slow)
            tables[(dim, r)] = RotaryEmbedding(dim, r.dims, r.base, None, "adjacent", n_pos, device, frequencies=f, magnitude=mag)
        return tables[(dim, r)]

    blocks, index = [], {}
    for i in c.owners():
        m, p = c.layers[i].mixer, c.layers[i].mlp
        if isinstance(m, AttentionSpec):
            mixer = ShapedAttention(E, m.heads, m.kv_heads, m.dim, m.vdim, dtype, m.scale, rotary=rotary(m.dim, m.rot), qkv_bias=True,
                                    wide_weights=True)
        else:
            mixer = LatentAttention(E, m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.q_rank, c.norm_eps, m.scale, dtype,
                                    rotary=rotary(m.rot_dim, m.rot), sink=True, wide_weights=True)
        ffn = norm2 = None
        if isinstance(p, DenseMlpSpec):
            ffn = PlainUnit(E, p.ff, dtype, act="relu2")
        elif p is not None:
            ffn = RoutedFeedForward(E, p.ff, p.experts, p.top, dtype, act="relu2", gated=False, scores="sigmoid", renormalize=True,
                                    scale_input=False, correction=True, groups=p.groups, renorm_eps=RENORM_EPS, defer_sum=True)
        if ffn is not None:
            norm2 = DynamicTanh(E, dtype)
        index[i] = len(blocks)
        blocks.append(PreNormBlock(DynamicTanh(E, dtype), mixer, norm2, ffn, names=("norm1.", "mix.", "norm2.", "mlp.", "side.")))
    bigram = BigramTable(c.bigram.buckets, E, c.bigram.mul_prev, c.bigram.mul_cur) if c.bigram is not None else None
    emb = TokenEmbedding(c.n_vocab, E, scale=c.embedding_scale, bigram=bigram)
    head = OutputHead(c.n_vocab, E, tied=False)
    return DecoderModel(c, dtype, emb, None, blocks, DynamicTanh(E, dtype, scale=c.logit_scale), head,
                        schedule=[Run(index[c.owner(i)]) for i in range(c.n_layer)])


_NORM = {"": "weight", ".b": "bias", ".alpha": "alpha"}
_ATTENTION = {"q": "q.weight", "k": "k.weight", "v": "v.weight", "q.b": "q.bias", "k.b": "k.bias", "v.b": "v.bias", "o": "output.weight"}
_LATENT = {"dq": "dq.weight", "dq.norm": "dq_norm.weight", "uq": "uq.weight", "dkv": "dkv.weight", "dkv.norm": "dkv_norm.weight",
           "uk": "uk.weight", "uv": "uv.weight", "sink": "sink", "g": "g.weight", "o": "o.weight"}
_UNIT = ("up", "down")


def file_names(config: LelutarConfig):
    """{name in the checkpoint: canonical name}, for the tensors this configuration has."""
    out = {"embed": "token_embd.weight", "head": "output.weight"}
    out.update({"final.norm" + s: "output_norm." + ours for s, ours in _NORM.items()})
    if config.bigram is not None:
        out["bigram"] = "token_embd.bigram.weight"
    for k, i in enumerate(config.owners()):
        layer = config.layers[i]
        names = {"norm1" + s: "norm1." + ours for s, ours in _NORM.items()}
        names.update({"mix." + s: "mix." + ours for s, ours in (_ATTENTION if isinstance(layer.mixer, AttentionSpec) else _LATENT).items()})
        if layer.mlp is not None:
            names.update({"norm2" + s: "norm2." + ours for s, ours in _NORM.items()})
            if isinstance(layer.mlp, DenseMlpSpec):
                names.update({"mlp." + u: f"mlp.{u}.weight" for u in _UNIT})
            else:
                names.update({"mlp.router": "mlp.router.weight", "mlp.correction": "mlp.correction"})
                for e in range(layer.mlp.experts):
                    names.update({f"mlp.e{e}.{u}": f"mlp.e{e}.{u}.weight" for u in _UNIT})
        for short, ours in names.items():
            out[f"l{i}.{short}"] = f"blk.{k}.{ours}"
    return out


register(Architecture("Lelutar", LelutarConfig.from_dict, build_lelutar, file_names), "lelutar")
