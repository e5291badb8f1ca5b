"""Typed configuration of the Gedilorn decoder, read from its own config.json keys.

config.json gives every size and every constant that differs between models of the design:

    architecture "Gedilorn"; vocab, width; norm.eps; streams (optional); logit_scale (optional)
    embedding {scale (optional), bigram {buckets, mul_prev, mul_cur} (optional)}
    layers[i]: type "latent_attention" | "latent_attention_2" (the second with an element-wise output gate)
               mixer {heads, dim, rot_dim, vdim, kv_rank, scale, rot {dims, base, scaling {factor, original, fast, slow}
               (optional)}}
               mlp null | {kind "dense", ff}
               weights_of (optional): the layer whose tensors this one uses (its entry equals that layer's)

What the design fixes (the feed-forward's activation, where norms sit, how rotated pairs lie) is in the parts and in the
builder.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Dict, List, Optional

from .errors import InvalidValue, MissingKey
from .rifizen import _get


@dataclass
class LatentMixerConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot_base: Optional[float]
    rot_scaling: Optional[Dict[str, float]]
    gated: bool


@dataclass
class PairTableConfig:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass
class GedilornLayer:
    type: str
    mixer: LatentMixerConfig
    ff: Optional[int]              # width of the dense feed-forward; None: the layer has none
    weights_of: Optional[int]      # the layer that owns the tensors; None: this one


@dataclass
class GedilornConfig:
    architecture: str
    vocab: int
    width: int
    eps: float
    streams: Optional[int]         # None: one residual stream, added to in the ordinary way
    embedding_scale: float
    pairs: Optional[PairTableConfig]
    logit_scale: float
    layers: List[GedilornLayer]
    raw: dict = field(default_factory=dict, repr=False)

    ARCHITECTURE = "Gedilorn"
    GATED = {"latent_attention": False, "latent_attention_2": True}

    @classmethod
    def from_dict(cls, raw: dict) -> "GedilornConfig":
        layers_raw = raw.get("layers")
        if layers_raw is None:
            raise MissingKey("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise InvalidValue("layers", layers_raw, "must be a non-empty list")
        layers = [cls._layer(layers_raw, i) for i in range(len(layers_raw))]
        for i, L in enumerate(layers):
            if L.weights_of is None:
                continue
            src = layers[L.weights_of]
            if (src.type, src.mixer, src.ff) != (L.type, L.mixer, L.ff):
                raise InvalidValue(f"layers[{i}].weights_of", L.weights_of, "the two layers' entries must be equal")
        pairs = None
        if isinstance(raw.get("embedding"), dict) and raw["embedding"].get("bigram") is not None:
            pairs = PairTableConfig(buckets=_get(raw, "embedding.bigram.buckets", int, minimum=1),
                                    mul_prev=_get(raw, "embedding.bigram.mul_prev", int),
                                    mul_cur=_get(raw, "embedding.bigram.mul_cur", int))
            if pairs.buckets >= 1 << 31:
                raise InvalidValue("embedding.bigram.buckets", pairs.buckets, "must be below 2^31")
        scale = _get(raw, "embedding.scale", float, optional=True)
        logit_scale = _get(raw, "logit_scale", float, optional=True)
        return cls(architecture=str(raw.get("architecture") or cls.ARCHITECTURE),
                   vocab=_get(raw, "vocab", int, minimum=1), width=_get(raw, "width", int, minimum=1),
                   eps=_get(raw, "norm.eps", float, positive=True), streams=_get(raw, "streams", int, optional=True, minimum=1),
                   embedding_scale=1.0 if scale is None else scale, pairs=pairs,
                   logit_scale=1.0 if logit_scale is None else logit_scale, layers=layers, raw=copy.deepcopy(raw))

    @classmethod
    def _layer(cls, layers_raw, i: int) -> GedilornLayer:
        p = f"layers[{i}]"
        L = layers_raw[i]
        if not isinstance(L, dict):
            raise InvalidValue(p, L, "must be an object")

        def g(path, k, **kw):
            return _get(L, path, k, where=p + ".", **kw)
        kind = L.get("type")
        if kind not in cls.GATED:
            raise InvalidValue(f"{p}.type", kind, "this design has layers of type 'latent_attention' and 'latent_attention_2'")
        src = g("weights_of", int, optional=True, minimum=0)
        if src is not None:
            seen = [i]
            while True:                               # a layer may name one that borrows itself: follow it to the owner
                if src >= len(layers_raw) or src in seen or not isinstance(layers_raw[src], dict):
                    raise InvalidValue(f"{p}.weights_of", src, "must name a layer that has tensors of its own")
                nxt = _get(layers_raw[src], "weights_of", int, optional=True, minimum=0, where=f"layers[{src}].")
                if nxt is None:
                    break
                seen.append(src)
                src = nxt
        rot_dim = g("mixer.rot_dim", int, optional=True, minimum=0) or 0
        base = scaling = None
        if rot_dim:
            if rot_dim % 2:
                raise InvalidValue(f"{p}.mixer.rot_dim", rot_dim, "must be even")
            dims = g("mixer.rot.dims", int)
            if dims != rot_dim:
                raise InvalidValue(f"{p}.mixer.rot.dims", dims, f"the rotated part turns as a whole: must equal rot_dim = {rot_dim}")
            base = g("mixer.rot.base", float, positive=True)
            if not base > 1:
                raise InvalidValue(f"{p}.mixer.rot.base", base, "must be larger than 1")
            if L["mixer"]["rot"].get("scaling") is not None:
                scaling = {k: g(f"mixer.rot.scaling.{k}", float, positive=True) for k in ("factor", "original", "fast", "slow")}
        m = LatentMixerConfig(heads=g("mixer.heads", int, minimum=1), dim=g("mixer.dim", int, minimum=1), rot_dim=rot_dim,
                              vdim=g("mixer.vdim", int, minimum=1), kv_rank=g("mixer.kv_rank", int, minimum=1),
                              scale=g("mixer.scale", float, positive=True), rot_base=base, rot_scaling=scaling, gated=cls.GATED[kind])
        mlp = L.get("mlp")
        ff = None
        if mlp is not None:
            mk = mlp.get("kind") if isinstance(mlp, dict) else None
            if mk != "dense":
                raise InvalidValue(f"{p}.mlp.kind", mk, "must be 'dense' (or mlp null)")
            ff = g("mlp.ff", int, minimum=1)
        return GedilornLayer(kind, m, ff, src)

    def to_dict(self) -> dict:
        return copy.deepcopy(self.raw)
