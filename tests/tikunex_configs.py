"""Small Tikunex configurations for the tests, and the folder writer they share.

A: sizes that share no factor with the kernels' tiles; key and value heads of different sizes; a window that is no
multiple of a page and keeps three first keys; three of five experts; a layer without feed-forward; a loop of two layers
that runs three times, with a layer before and one behind it.
B: everything a multiple of 8, so that 16-bit runs take the tensor-core products; key size 64; a window longer than two
pages that keeps more than a page of first keys; a loop that starts at layer 0 and runs twice.
C: the smallest of everything: one head, a window of one key and one kept key, one expert, no loop and no token input.
D: values above keys' size, a window without kept keys and one attention without a mask, the two scales of a pair far apart,
one of them negative, every expert chosen, a loop of one pass around the last layer.
"""
import os

_MLP_A = {"kind": "moe", "expert": {"ff": 20}, "router": {"experts": 5, "top": 3}}
_GLA_A = {"type": "gla", "mixer": {"heads": 3, "dim": 10, "vdim": 14, "tau": 4.0, "decay_rank": 5}}
_PAIR_A = {"type": "parallel", "mixer": {"left": {"heads": 3, "kv_heads": 1, "dim": 10, "vdim": 14, "scale": 0.4, "mask": {"size": 19, "keep_first": 3}},
                                         "right": {"heads": 5, "dim": 6, "decay_rank": 3}, "left_scale": 0.7, "right_scale": 1.6}}
TIKUNEX_A = {
    "architecture": "Tikunex", "vocab": 197, "width": 52, "norm": {"eps": 1e-5}, "token_side": {"dim": 6},
    "loop": {"start": 1, "stop": 3, "times": 3},
    "layers": [dict(_PAIR_A, mlp=_MLP_A), dict(_GLA_A, mlp=None), dict(_PAIR_A, mlp=_MLP_A), dict(_GLA_A, mlp=_MLP_A)],
}
_MLP_B = {"kind": "moe", "expert": {"ff": 64}, "router": {"experts": 6, "top": 2}}
TIKUNEX_B = {
    "architecture": "Tikunex", "vocab": 256, "width": 128, "norm": {"eps": 3e-6}, "token_side": {"dim": 32},
    "loop": {"start": 0, "stop": 2, "times": 2},
    "layers": [
        {"type": "gla", "mixer": {"heads": 2, "dim": 64, "vdim": 32, "tau": 8.0, "decay_rank": 16}, "mlp": _MLP_B},
        {"type": "parallel", "mixer": {"left": {"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 32, "scale": 0.2, "mask": {"size": 36, "keep_first": 18}},
                                       "right": {"heads": 2, "dim": 64, "decay_rank": 8}, "left_scale": 1.3, "right_scale": 0.6}, "mlp": _MLP_B},
        {"type": "gla", "mixer": {"heads": 4, "dim": 32, "vdim": 64, "tau": 2.0, "decay_rank": 24}, "mlp": _MLP_B},
    ],
}
TIKUNEX_C = {
    "architecture": "Tikunex", "vocab": 64, "width": 32, "norm": {"eps": 1e-6},
    "layers": [
        {"type": "parallel", "mixer": {"left": {"heads": 1, "kv_heads": 1, "dim": 8, "vdim": 8, "scale": 0.35, "mask": {"size": 1, "keep_first": 1}},
                                       "right": {"heads": 1, "dim": 4, "decay_rank": 1}, "left_scale": 1.0, "right_scale": 1.0},
         "mlp": {"kind": "moe", "expert": {"ff": 24}, "router": {"experts": 1, "top": 1}}},
        {"type": "gla", "mixer": {"heads": 1, "dim": 5, "vdim": 33, "tau": 1.0, "decay_rank": 2}, "mlp": None},
    ],
}
TIKUNEX_D = {
    "architecture": "Tikunex", "vocab": 90, "width": 40, "norm": {"eps": 1e-4}, "token_side": {"dim": 5},
    "loop": {"start": 2, "stop": 3, "times": 1},
    "layers": [
        {"type": "parallel", "mixer": {"left": {"heads": 4, "kv_heads": 4, "dim": 6, "vdim": 20, "scale": 0.5, "mask": {"size": 7, "keep_first": 0}},
                                       "right": {"heads": 2, "dim": 12, "decay_rank": 4}, "left_scale": 2.5, "right_scale": 0.1},
         "mlp": {"kind": "moe", "expert": {"ff": 12}, "router": {"experts": 4, "top": 4}}},
        {"type": "parallel", "mixer": {"left": {"heads": 2, "kv_heads": 1, "dim": 16, "vdim": 8, "scale": 0.3},
                                       "right": {"heads": 3, "dim": 9, "decay_rank": 7}, "left_scale": 0.8, "right_scale": -0.9}, "mlp": None},
        {"type": "gla", "mixer": {"heads": 2, "dim": 7, "vdim": 9, "tau": 32.0, "decay_rank": 3},
         "mlp": {"kind": "moe", "expert": {"ff": 16}, "router": {"experts": 7, "top": 1}}},
    ],
}
TIKUNEX = {"A": (TIKUNEX_A, 3), "B": (TIKUNEX_B, 4), "C": (TIKUNEX_C, 5), "D": (TIKUNEX_D, 6)}


def write_model(cfg, folder, seed, std=0.12):
    """config.json + model.safetensors (bfloat16 matrices, short tensor names) from the engine's
    random-weights mode; the plain implementation reads the folder with its own reader."""
    from ferrum_b200.weights import write_random_model
    write_random_model(cfg, folder, seed, dtype="bfloat16", std=std)
    assert os.path.exists(os.path.join(folder, "model.safetensors"))
    return folder
