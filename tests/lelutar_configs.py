"""Small Lelutar configurations for the tests, and the folder writer they share.

A: sizes that share no factor with the kernels' tiles; key and value heads of different sizes, a rotation over a part of the
head; groups of two experts of which three are kept; a layer without feed-forward; layers that run again with the tensors of
an earlier one (their caches differ), one of them twice; one rotation without scaling.
B: everything a multiple of 8, so that 16-bit runs take the tensor-core products, latents that take the tensor-core attention
(more heads than a row tile in one layer, rotated and not); groups of four experts; an entry that uses the tensors of a later one.
C: the smallest of everything: one head, keys of two, a latent of one, one expert in one group, no table of pairs.
D: many experts in groups of one, negative scales, values above the keys' size, an unrotated attention, a mixture without
groups, a scale of the embedding below one.
E: attention heads of the sizes that the tensor-core attention takes (values as long as the keys, and longer), in a model
without experts but for one layer, so that long requests compare row by row in 16 bits too.
"""
import os

_MOE_A = {"kind": "moe", "expert": {"ff": 20}, "router": {"experts": 10, "top": 3, "groups": {"count": 5, "keep": 3}}}
_ROT_A = {"base": 700.0, "dims": 6, "scaling": {"factor": 3.0, "original": 48, "fast": 9.0, "slow": 0.5}}
_LATENT_A = {"type": "latent_attention", "mixer": {"heads": 3, "dim": 7, "vdim": 9, "kv_rank": 11, "q_rank": 13, "scale": 0.6}, "mlp": _MOE_A}
_TURNED_A = {"type": "latent_attention_2", "mixer": {"heads": 5, "dim": 6, "rot_dim": 4, "vdim": 10, "kv_rank": 18, "q_rank": 17, "scale": 0.5,
                                                     "rot": {"base": 300.0, "dims": 4, "scaling": {"factor": 5.0, "original": 64, "fast": 4.0, "slow": 1.0}}},
             "mlp": None}
LELUTAR_A = {
    "architecture": "Lelutar", "vocab": 197, "width": 52, "norm": {"eps": 1e-4}, "logit_scale": 1.7,
    "embedding": {"scale": 3.5, "bigram": {"buckets": 61, "mul_prev": 31, "mul_cur": 7}},
    "layers": [
        {"type": "attention", "mixer": {"heads": 6, "kv_heads": 2, "dim": 10, "vdim": 14, "scale": 0.45, "rot": _ROT_A}, "mlp": {"kind": "dense", "ff": 36}},
        _LATENT_A, _TURNED_A, dict(_TURNED_A, weights_of=2), dict(_LATENT_A, weights_of=1), dict(_TURNED_A, weights_of=3),
        {"type": "attention", "mixer": {"heads": 3, "kv_heads": 3, "dim": 6, "vdim": 5, "scale": 0.5, "rot": {"base": 100.0, "dims": 6}}, "mlp": _MOE_A},
    ],
}
_MOE_B = {"kind": "moe", "expert": {"ff": 40}, "router": {"experts": 16, "top": 4, "groups": {"count": 4, "keep": 2}}}
_ATT_B = {"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 24, "scale": 0.2,
                                         "rot": {"base": 10000.0, "dims": 32, "scaling": {"factor": 2.0, "original": 128, "fast": 16.0, "slow": 1.0}}}, "mlp": _MOE_B}
LELUTAR_B = {
    "architecture": "Lelutar", "vocab": 256, "width": 128, "norm": {"eps": 3e-6}, "logit_scale": 0.8,
    "embedding": {"scale": 5.0, "bigram": {"buckets": 100, "mul_prev": 1013, "mul_cur": 2027}},
    "layers": [
        dict(_ATT_B, weights_of=3),
        {"type": "latent_attention", "mixer": {"heads": 20, "dim": 16, "vdim": 8, "kv_rank": 64, "q_rank": 48, "scale": 0.3}, "mlp": {"kind": "dense", "ff": 96}},
        {"type": "latent_attention_2", "mixer": {"heads": 2, "dim": 24, "rot_dim": 32, "vdim": 40, "kv_rank": 96, "q_rank": 56, "scale": 0.17,
                                                 "rot": {"base": 2000.0, "dims": 32, "scaling": {"factor": 16.0, "original": 32, "fast": 32.0, "slow": 2.0}}},
         "mlp": _MOE_B},
        _ATT_B,
    ],
}
LELUTAR_C = {
    "architecture": "Lelutar", "vocab": 64, "width": 32, "norm": {"eps": 1e-6}, "logit_scale": 1.0, "embedding": {"scale": 1.0},
    "layers": [
        {"type": "attention", "mixer": {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 1, "scale": 0.9, "rot": {"base": 50.0, "dims": 2}},
         "mlp": {"kind": "moe", "expert": {"ff": 24}, "router": {"experts": 1, "top": 1, "groups": {"count": 1, "keep": 1}}}},
        {"type": "latent_attention", "mixer": {"heads": 1, "dim": 1, "vdim": 3, "kv_rank": 1, "q_rank": 1, "scale": 1.0}, "mlp": None},
    ],
}
LELUTAR_D = {
    "architecture": "Lelutar", "vocab": 90, "width": 40, "norm": {"eps": 1e-3}, "logit_scale": -0.6,
    "embedding": {"scale": 0.7, "bigram": {"buckets": 1, "mul_prev": 5, "mul_cur": 3}},
    "layers": [
        {"type": "latent_attention_2", "mixer": {"heads": 8, "dim": 4, "rot_dim": 6, "vdim": 20, "kv_rank": 40, "q_rank": 9, "scale": -0.4,
                                                 "rot": {"base": 90.0, "dims": 6}},
         "mlp": {"kind": "moe", "expert": {"ff": 12}, "router": {"experts": 36, "top": 5, "groups": {"count": 36, "keep": 7}}}},
        {"type": "attention", "mixer": {"heads": 4, "kv_heads": 1, "dim": 6, "vdim": 20, "scale": 0.5},
         "mlp": {"kind": "moe", "expert": {"ff": 16}, "router": {"experts": 7, "top": 2}}},
    ],
}
_ROT_E = {"base": 4000.0, "dims": 64, "scaling": {"factor": 6.0, "original": 96, "fast": 12.0, "slow": 1.0}}
LELUTAR_E = {
    "architecture": "Lelutar", "vocab": 144, "width": 96, "norm": {"eps": 1e-5}, "logit_scale": 0.9,
    "embedding": {"scale": 2.0, "bigram": {"buckets": 77, "mul_prev": 13, "mul_cur": 29}},
    "layers": [
        {"type": "attention", "mixer": {"heads": 8, "kv_heads": 2, "dim": 64, "vdim": 64, "scale": 0.12, "rot": _ROT_E}, "mlp": {"kind": "dense", "ff": 120}},
        {"type": "attention", "mixer": {"heads": 6, "kv_heads": 1, "dim": 40, "vdim": 128, "scale": 0.16, "rot": {"base": 100.0, "dims": 24}}, "mlp": None},
        {"type": "latent_attention_2", "mixer": {"heads": 3, "dim": 16, "rot_dim": 16, "vdim": 24, "kv_rank": 32, "q_rank": 40, "scale": 0.25,
                                                 "rot": {"base": 500.0, "dims": 16}},
         "mlp": {"kind": "moe", "expert": {"ff": 32}, "router": {"experts": 6, "top": 2, "groups": {"count": 2, "keep": 1}}}},
        {"type": "attention", "mixer": {"heads": 8, "kv_heads": 2, "dim": 64, "vdim": 64, "scale": 0.12, "rot": _ROT_E}, "mlp": {"kind": "dense", "ff": 120},
         "weights_of": 0},
    ],
}
LELUTAR = {"A": (LELUTAR_A, 3), "B": (LELUTAR_B, 4), "C": (LELUTAR_C, 5), "D": (LELUTAR_D, 6), "E": (LELUTAR_E, 7)}


def write_model(cfg, folder, seed, std=0.12):
    """config.json + model.safetensors (bfloat16 matrices, short tensor names) from the engine's
    random-weights mode; the plain implementation reads the folder with its own reader."""
    from ferrum_b200.weights import write_random_model
    write_random_model(cfg, folder, seed, dtype="bfloat16", std=std)
    assert os.path.exists(os.path.join(folder, "model.safetensors"))
    return folder
