"""Typed configuration of the Tikunex decoder.

Its config.json is nested: `architecture`, `vocab`, `width`, `norm.eps`, optionally `token_side.dim` (the
columns of the second embedding table that each layer reads) and `loop` {start, stop, times} (layers start ..
stop - 1 run that many times in a row), and `layers`, a list whose entries give the layer's `type` (which
mixer), the mixer's sizes under `mixer` and its feed-forward under `mlp` (null: none).  Every size and every
constant that can differ between two models of the design is read here and nowhere else; what an entry does
not mention does not exist.

Mixers:
  `gla`        heads, dim, vdim, tau: gated linear attention, one decay per head and key channel
  `parallel`   `left`: heads, kv_heads, dim, vdim, scale, mask.{size, keep_first} (a query sees itself, the
               size - 1 keys before it and the sequence's first keep_first keys); `right`: heads, dim: an
               RWKV-style recurrence; left_scale, right_scale: the factors of their sum
The inner sizes of the decays' low-rank pairs are read off the tensors (optional keys `decay_rank` fix them,
e.g. for random weights).

Feed-forward (`mlp.kind` = `moe`): expert.ff, router.{experts, top}.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import List, Optional, Tuple, Union

from ..errors import ConfigError


@dataclass(frozen=True)
class GlaSpec:
    heads: int
    dim: int
    vdim: int
    tau: float
    decay_rank: Optional[int] = None


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0                 # 0: every earlier key
    keep_first: int = 0             # with a window: first keys of the sequence that every query sees


@dataclass(frozen=True)
class TimeMixingSpec:
    heads: int
    dim: int
    decay_rank: Optional[int] = None


@dataclass(frozen=True)
class PairSpec:
    left: AttentionSpec
    right: TimeMixingSpec
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class MoeSpec:
    ff: int
    experts: int
    top: int
    kind: str = "moe"


@dataclass(frozen=True)
class LayerSpec:
    type: str
    mixer: Union[GlaSpec, PairSpec]
    mlp: Optional[MoeSpec]


@dataclass(frozen=True)
class LoopSpec:
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class TikunexConfig:
    architecture: str
    n_vocab: int
    n_embd: int
    norm_eps: float
    layers: Tuple[LayerSpec, ...]
    loop: Optional[LoopSpec] = None
    side_dim: int = 0               # 0: no second embedding table
    n_ctx_train: int = 8192         # the engine's default of the longest sequence (nothing in the model depends on it)
    eos_token_ids: Tuple[int, ...] = ()
    stored_dtype: str = "bfloat16"
    extra: dict = field(default_factory=dict, compare=False)

    @property
    def n_layer(self):
        return len(self.layers)

    def run_order(self) -> List[Tuple[int, bool]]:
        """(layer, whether a pass of the loop starts with it) in the order in which the layers run."""
        n, loop = len(self.layers), self.loop
        if loop is None:
            return [(i, False) for i in range(n)]
        once = [(i, i == loop.start) for i in range(loop.start, loop.stop)]
        return [(i, False) for i in range(loop.start)] + once * loop.times + [(i, False) for i in range(loop.stop, n)]

    def __post_init__(self):
        for k in ("n_vocab", "n_embd"):
            v = getattr(self, k)
            if not isinstance(v, int) or v <= 0:
                raise ConfigError(f"tikunex: {k} must be a positive integer, found {v!r}")
        if not (math.isfinite(self.norm_eps) and self.norm_eps > 0.0):
            raise ConfigError("tikunex: invalid norm.eps")
        if not self.layers:
            raise ConfigError("tikunex: no layers")
        if self.side_dim < 0:
            raise ConfigError("tikunex: token_side.dim must not be negative")
        loop = self.loop
        if loop is not None and not (0 <= loop.start < loop.stop <= len(self.layers) and loop.times >= 1):
            raise ConfigError(f"tikunex: loop {loop.start}..{loop.stop} x {loop.times} does not fit {len(self.layers)} layers")
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            if isinstance(m, GlaSpec):
                if min(m.heads, m.dim, m.vdim) <= 0 or not (math.isfinite(m.tau) and m.tau > 0):
                    raise ConfigError(f"tikunex: layer {i}: invalid sizes or tau of the gla mixer")
            else:
                a, r = m.left, m.right
                if min(a.heads, a.kv_heads, a.dim, a.vdim) <= 0 or a.heads % a.kv_heads:
                    raise ConfigError(f"tikunex: layer {i}: invalid sizes of the left mixer (kv_heads must divide heads)")
                if not all(math.isfinite(v) for v in (a.scale, m.left_scale, m.right_scale)):
                    raise ConfigError(f"tikunex: layer {i}: invalid scale")
                if a.window < 0 or a.keep_first < 0:
                    raise ConfigError(f"tikunex: layer {i}: invalid mask")
                if min(r.heads, r.dim) <= 0:
                    raise ConfigError(f"tikunex: layer {i}: invalid sizes of the right mixer")
            p = layer.mlp
            if p is not None and (p.ff <= 0 or p.experts <= 0 or not 0 < p.top <= p.experts):
                raise ConfigError(f"tikunex: layer {i}: {p.top} of {p.experts} experts of {p.ff} per token")

    @staticmethod
    def from_dict(d: dict) -> "TikunexConfig":
        def need(obj, key, where=""):
            if not isinstance(obj, dict) or key not in obj or obj[key] is None:
                raise ConfigError(f"config.json: missing required key {where}{key!r}")
            return obj[key]

        def rank(m):
            return int(m["decay_rank"]) if m.get("decay_rank") is not None else None

        layers = []
        for i, L in enumerate(need(d, "layers")):
            where = f"layers[{i}]."
            kind = need(L, "type", where)
            m = need(L, "mixer", where)
            mw = where + "mixer."
            if kind == "gla":
                spec = GlaSpec(heads=int(need(m, "heads", mw)), dim=int(need(m, "dim", mw)), vdim=int(need(m, "vdim", mw)),
                               tau=float(need(m, "tau", mw)), decay_rank=rank(m))
            elif kind == "parallel":
                a, r = need(m, "left", mw), need(m, "right", mw)
                aw, rw = mw + "left.", mw + "right."
                window = keep = 0
                if a.get("mask") is not None:
                    window = int(need(a["mask"], "size", aw + "mask."))
                    keep = int(a["mask"].get("keep_first") or 0)
                    if window <= 0:
                        raise ConfigError(f"config.json: {aw}mask.size must be positive")
                left = AttentionSpec(heads=int(need(a, "heads", aw)), kv_heads=int(need(a, "kv_heads", aw)), dim=int(need(a, "dim", aw)),
                                     vdim=int(need(a, "vdim", aw)), scale=float(need(a, "scale", aw)), window=window, keep_first=keep)
                spec = PairSpec(left=left, right=TimeMixingSpec(heads=int(need(r, "heads", rw)), dim=int(need(r, "dim", rw)), decay_rank=rank(r)),
                                left_scale=float(need(m, "left_scale", mw)), right_scale=float(need(m, "right_scale", mw)))
            else:
                raise ConfigError(f"config.json: {where}type {kind!r} is not a mixer of this design")
            mlp = L.get("mlp")
            if mlp is not None:
                pw = where + "mlp."
                if mlp.get("kind", "moe") != "moe":
                    raise ConfigError(f"config.json: {pw}kind {mlp['kind']!r} is not a feed-forward of this design")
                router = need(mlp, "router", pw)
                mlp = MoeSpec(ff=int(need(need(mlp, "expert", pw), "ff", pw + "expert.")),
                              experts=int(need(router, "experts", pw + "router.")), top=int(need(router, "top", pw + "router.")))
            layers.append(LayerSpec(kind, spec, mlp))
        loop = d.get("loop")
        if loop is not None:
            loop = LoopSpec(*(int(need(loop, k, "loop.")) for k in ("start", "stop", "times")))
        side = d.get("token_side")
        return TikunexConfig(
            architecture=str(d.get("architecture") or (d.get("architectures") or ["Tikunex"])[0]),
            n_vocab=int(need(d, "vocab")), n_embd=int(need(d, "width")), norm_eps=float(need(need(d, "norm"), "eps", "norm.")),
            layers=tuple(layers), loop=loop, side_dim=int(need(side, "dim", "token_side.")) if side is not None else 0,
            n_ctx_train=int(d.get("max_positions", 8192)), stored_dtype=str(d.get("torch_dtype", "bfloat16")), extra={})
