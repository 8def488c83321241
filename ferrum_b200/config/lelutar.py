"""Typed configuration of the Lelutar decoder.

Its config.json is nested: `architecture`, `vocab`, `width`, `norm.eps` (the latents' RMS norms), `logit_scale`,
`embedding.scale`, optionally `embedding.bigram` {buckets, mul_prev, mul_cur} (a hashed table of token pairs), and
`layers`, a list whose entries give the layer's `type` (which mixer), the mixer's sizes under `mixer` and its
feed-forward under `mlp` (null: none).  An entry with `weights_of`: j runs with layer j's tensors and a cache of its
own.  Every size and every constant that can differ between two models of the design is read here and nowhere
else; what an entry does not mention does not exist.

Mixers:
  `attention`           heads, kv_heads, dim, vdim, scale, rot
  `latent_attention`    heads, dim, vdim, kv_rank, q_rank, scale: no positions
  `latent_attention_2`  heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, rot (over the rot_dim part)
  rot: base, dims, optionally scaling {factor, original, fast, slow} (YaRN)

Feed-forwards (`mlp.kind`), all with the square of relu and without gates:
  `dense`        ff
  `moe`          expert.ff, router.{experts, top}, optionally router.groups.{count, keep}
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import List, Optional, Tuple, Union

from ..errors import ConfigError


@dataclass(frozen=True)
class YarnSpec:
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class RotarySpec:
    base: float
    dims: int
    scaling: Optional[YarnSpec] = None


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[RotarySpec] = None


@dataclass(frozen=True)
class LatentSpec:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    rot_dim: int = 0                        # 0: no rotated part
    rot: Optional[RotarySpec] = None


@dataclass(frozen=True)
class DenseMlpSpec:
    ff: int
    kind: str = "dense"


@dataclass(frozen=True)
class RoutedMlpSpec:
    ff: int
    experts: int
    top: int
    groups: Optional[Tuple[int, int]] = None        # (count, keep)
    kind: str = "moe"


@dataclass(frozen=True)
class LayerSpec:
    type: str
    mixer: Union[AttentionSpec, LatentSpec]
    mlp: Optional[Union[DenseMlpSpec, RoutedMlpSpec]]
    weights_of: Optional[int] = None


@dataclass(frozen=True)
class BigramSpec:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class LelutarConfig:
    architecture: str
    n_vocab: int
    n_embd: int
    norm_eps: float
    layers: Tuple[LayerSpec, ...]
    embedding_scale: float = 1.0
    bigram: Optional[BigramSpec] = None
    logit_scale: float = 1.0
    n_ctx_train: int = 8192                 # positions the rotary tables cover unless the caller asks for more or fewer
    eos_token_ids: Tuple[int, ...] = ()
    stored_dtype: str = "bfloat16"
    extra: dict = field(default_factory=dict, compare=False)

    @property
    def n_layer(self):
        return len(self.layers)

    def owner(self, i) -> int:
        """The layer whose tensors layer i runs with (itself, or where its chain of `weights_of` ends)."""
        seen = set()
        while self.layers[i].weights_of is not None:
            if i in seen:
                raise ConfigError(f"lelutar: layer {i}: weights_of runs in a circle")
            seen.add(i)
            i = self.layers[i].weights_of
        return i

    def owners(self) -> List[int]:
        """The layers that have tensors of their own, in order."""
        return [i for i, layer in enumerate(self.layers) if layer.weights_of is None]

    def __post_init__(self):
        for k in ("n_vocab", "n_embd"):
            v = getattr(self, k)
            if not isinstance(v, int) or v <= 0:
                raise ConfigError(f"lelutar: {k} must be a positive integer, found {v!r}")
        if not (math.isfinite(self.norm_eps) and self.norm_eps > 0.0):
            raise ConfigError("lelutar: invalid norm.eps")
        if not (math.isfinite(self.embedding_scale) and math.isfinite(self.logit_scale)):
            raise ConfigError("lelutar: invalid embedding.scale or logit_scale")
        if self.bigram is not None and self.bigram.buckets <= 0:
            raise ConfigError("lelutar: embedding.bigram.buckets must be positive")
        if not self.layers:
            raise ConfigError("lelutar: no layers")
        n = len(self.layers)
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            names = ("heads", "kv_heads", "dim", "vdim") if isinstance(m, AttentionSpec) else ("heads", "dim", "vdim", "kv_rank", "q_rank")
            for k in names:
                if getattr(m, k) <= 0:
                    raise ConfigError(f"lelutar: layer {i}: {k} must be positive")
            turned = m.dim
            if isinstance(m, AttentionSpec):
                if m.heads % m.kv_heads:
                    raise ConfigError(f"lelutar: layer {i}: kv_heads does not divide heads")
            else:
                turned = m.rot_dim
                if m.rot_dim < 0:
                    raise ConfigError(f"lelutar: layer {i}: rot_dim must not be negative")
            if not math.isfinite(m.scale):
                raise ConfigError(f"lelutar: layer {i}: invalid scale")
            r = m.rot
            if r is not None:
                if r.dims % 2 or not 0 < r.dims <= turned:
                    raise ConfigError(f"lelutar: layer {i}: rot.dims must be even and at most {turned}")
                if not (math.isfinite(r.base) and r.base > 0.0):
                    raise ConfigError(f"lelutar: layer {i}: invalid rot.base")
                s = r.scaling
                if s is not None and (r.base == 1.0 or not all(math.isfinite(v) and v > 0.0 for v in (s.factor, s.original, s.fast, s.slow))):
                    raise ConfigError(f"lelutar: layer {i}: invalid rot.scaling")
            p = layer.mlp
            if p is not None:
                if p.ff <= 0:
                    raise ConfigError(f"lelutar: layer {i}: ff must be positive")
                if isinstance(p, RoutedMlpSpec):
                    if not 0 < p.top <= p.experts:
                        raise ConfigError(f"lelutar: layer {i}: {p.top} of {p.experts} experts per token")
                    if p.groups is not None:
                        count, keep = p.groups
                        if not (0 < keep <= count and p.experts % count == 0 and p.top <= p.experts // count * keep):
                            raise ConfigError(f"lelutar: layer {i}: {p.top} of {p.experts} experts cannot come from {keep} of {count} groups")
            j = layer.weights_of
            if j is not None:
                if not 0 <= j < n or j == i:
                    raise ConfigError(f"lelutar: layer {i}: weights_of names layer {j}, which does not exist or is itself")
                o = self.layers[self.owner(i)]
                if (o.type, o.mixer, o.mlp) != (layer.type, layer.mixer, layer.mlp):
                    raise ConfigError(f"lelutar: layer {i} differs from layer {self.owner(i)}, whose weights it uses")

    @staticmethod
    def from_dict(d: dict) -> "LelutarConfig":
        def need(obj, key, where=""):
            if not isinstance(obj, dict) or key not in obj or obj[key] is None:
                raise ConfigError(f"config.json: missing required key {where}{key!r}")
            return obj[key]

        def rotary(m, where):
            r = m.get("rot")
            if not r or not r.get("dims"):
                return None
            s = r.get("scaling")
            if s:
                s = YarnSpec(*(float(need(s, k, where + "rot.scaling.")) for k in ("factor", "original", "fast", "slow")))
            return RotarySpec(float(need(r, "base", where + "rot.")), int(r["dims"]), s or None)

        layers = []
        for i, L in enumerate(need(d, "layers")):
            where = f"layers[{i}]."
            kind = need(L, "type", where)
            m = need(L, "mixer", where)
            mw = where + "mixer."
            if kind == "attention":
                spec = AttentionSpec(*(int(need(m, k, mw)) for k in ("heads", "kv_heads", "dim", "vdim")), float(need(m, "scale", mw)), rotary(m, mw))
            elif kind in ("latent_attention", "latent_attention_2"):
                sizes = (int(need(m, k, mw)) for k in ("heads", "dim", "vdim", "kv_rank", "q_rank"))
                rot_dim = int(need(m, "rot_dim", mw)) if kind == "latent_attention_2" else 0
                spec = LatentSpec(*sizes, float(need(m, "scale", mw)), rot_dim, rotary(m, mw) if rot_dim else None)
            else:
                raise ConfigError(f"config.json: {where}type {kind!r} is not a mixer of this design")
            mlp = L.get("mlp")
            if mlp is not None:
                pw = where + "mlp."
                mk = need(mlp, "kind", pw)
                if mk == "dense":
                    mlp = DenseMlpSpec(ff=int(need(mlp, "ff", pw)))
                elif mk == "moe":
                    router = need(mlp, "router", pw)
                    rw = pw + "router."
                    groups = router.get("groups")
                    if groups is not None:
                        groups = tuple(int(need(groups, k, rw + "groups.")) for k in ("count", "keep"))
                    mlp = RoutedMlpSpec(ff=int(need(need(mlp, "expert", pw), "ff", pw + "expert.")), experts=int(need(router, "experts", rw)),
                                        top=int(need(router, "top", rw)), groups=groups)
                else:
                    raise ConfigError(f"config.json: {pw}kind {mk!r} is not a feed-forward of this design")
            of = L.get("weights_of")
            layers.append(LayerSpec(kind, spec, mlp, int(of) if of is not None else None))
        emb = d.get("embedding") or {}
        bigram = emb.get("bigram")
        if bigram is not None:
            bigram = BigramSpec(*(int(need(bigram, k, "embedding.bigram.")) for k in ("buckets", "mul_prev", "mul_cur")))

        def number(obj, key):
            return float(obj[key]) if obj.get(key) is not None else 1.0
        return LelutarConfig(
            architecture=str(d.get("architecture") or (d.get("architectures") or ["Lelutar"])[0]),
            n_vocab=int(need(d, "vocab")), n_embd=int(need(d, "width")), norm_eps=float(need(need(d, "norm"), "eps", "norm.")),
            layers=tuple(layers), embedding_scale=number(emb, "scale"), bigram=bigram, logit_scale=number(d, "logit_scale"),
            n_ctx_train=int(d.get("max_positions", 8192)), stored_dtype=str(d.get("torch_dtype", "bfloat16")), extra={})
