"""Typed configuration of the Dubodra decoder, read from its own config.json keys.

config.json gives every size and every constant that differs between models of the design:

    architecture "Dubodra"; vocab, width; norm.eps; embedding.scale, logit_softcap, token_side.dim (each optional)
    layers[i]: type "attention":  mixer {heads, kv_heads, dim, vdim, scale, softcap (optional), rot {dims, base} (optional)}
               type "lightning":  mixer {heads, dim, vdim, decay[heads]}
               type "delta":      mixer {heads, kv_heads, dim, vdim, conv}
               mlp null | {kind "dense", ff}
                        | {kind "moe", expert {ff, limit}, router {experts, top, identity, scale, groups {count, keep}},
                           shared {ff, limit} (optional)}

Absent ``router.groups`` means one group, absent ``identity`` none, absent ``scale`` 1.  What the design fixes (activation
functions, where norms sit, how rotated pairs lie, the 1e-6 of the unit vectors, the 1.702 of the clamped unit) is in the
parts and in the builder.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import List, Optional

from .errors import InvalidValue, MissingKey
from .rifizen import _get


@dataclass
class CappedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: Optional[float]
    rot_dims: int
    rot_base: Optional[float]


@dataclass
class LightningConfig:
    heads: int
    dim: int
    vdim: int
    decay: List[float]


@dataclass
class DeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int


@dataclass
class UnitConfig:
    ff: int
    limit: float


@dataclass
class DubodraMlp:
    kind: str                      # "dense" | "moe"
    ff: int = 0                    # of the dense layer
    expert: Optional[UnitConfig] = None
    shared: Optional[UnitConfig] = None
    experts: int = 0
    identity: int = 0
    top: int = 0
    scale: float = 1.0
    groups: int = 1
    keep: int = 1


@dataclass
class DubodraLayer:
    type: str                      # "attention" | "lightning" | "delta"
    mixer: object
    mlp: Optional[DubodraMlp]


@dataclass
class DubodraConfig:
    architecture: str
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    logit_softcap: Optional[float]
    side_dim: Optional[int]
    layers: List[DubodraLayer]
    raw: dict = field(default_factory=dict, repr=False)

    ARCHITECTURE = "Dubodra"

    @classmethod
    def from_dict(cls, raw: dict) -> "DubodraConfig":
        layers_raw = raw.get("layers")
        if layers_raw is None:
            raise MissingKey("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise InvalidValue("layers", layers_raw, "must be a non-empty list")
        layers: List[DubodraLayer] = []
        mixers = {"attention": cls._attention, "lightning": cls._lightning, "delta": cls._delta}
        for i, L in enumerate(layers_raw):
            p = f"layers[{i}]"
            if not isinstance(L, dict):
                raise InvalidValue(p, L, "must be an object")
            kind = L.get("type")
            if kind not in mixers:
                raise InvalidValue(f"{p}.type", kind, "this design has layers of type 'attention', 'lightning' and 'delta'")

            def g(path, k, L=L, p=p, **kw):
                return _get(L, path, k, where=p + ".", **kw)
            layers.append(DubodraLayer(kind, mixers[kind](L, g, p), cls._mlp(L, g, p)))
        scale = _get(raw, "embedding.scale", float, optional=True)
        return cls(architecture=str(raw.get("architecture") or cls.ARCHITECTURE),
                   vocab=_get(raw, "vocab", int, minimum=1), width=_get(raw, "width", int, minimum=1),
                   eps=_get(raw, "norm.eps", float, positive=True), embedding_scale=1.0 if scale is None else scale,
                   logit_softcap=_get(raw, "logit_softcap", float, optional=True, positive=True),
                   side_dim=_get(raw, "token_side.dim", int, optional=raw.get("token_side") is None, minimum=1),
                   layers=layers, raw=copy.deepcopy(raw))

    @staticmethod
    def _shared_heads(p, heads: int, kv_heads: int) -> None:
        if heads % kv_heads:
            raise InvalidValue(f"{p}.mixer.kv_heads", kv_heads, f"must divide heads = {heads}")

    @classmethod
    def _attention(cls, L, g, p) -> CappedAttentionConfig:
        rot_dims = g("mixer.rot.dims", int, optional=True, minimum=0) or 0
        m = CappedAttentionConfig(
            heads=g("mixer.heads", int, minimum=1), kv_heads=g("mixer.kv_heads", int, minimum=1),
            dim=g("mixer.dim", int, minimum=1), vdim=g("mixer.vdim", int, minimum=1),
            scale=g("mixer.scale", float, positive=True), softcap=g("mixer.softcap", float, optional=True, positive=True),
            rot_dims=rot_dims, rot_base=g("mixer.rot.base", float, positive=True) if rot_dims else None)
        cls._shared_heads(p, m.heads, m.kv_heads)
        if m.rot_dims % 2 or m.rot_dims > m.dim:
            raise InvalidValue(f"{p}.mixer.rot.dims", m.rot_dims, f"must be even and at most dim = {m.dim}")
        return m

    @staticmethod
    def _lightning(L, g, p) -> LightningConfig:
        heads = g("mixer.heads", int, minimum=1)
        decay = L["mixer"].get("decay")
        if decay is None:
            raise MissingKey(f"{p}.mixer.decay")
        if (not isinstance(decay, list) or len(decay) != heads
                or any(isinstance(d, bool) or not isinstance(d, (int, float)) or not 0 <= d <= 1 for d in decay)):
            raise InvalidValue(f"{p}.mixer.decay", decay, f"must hold heads = {heads} numbers from 0 to 1")
        m = LightningConfig(heads, g("mixer.dim", int, minimum=1), g("mixer.vdim", int, minimum=1), [float(d) for d in decay])
        if m.dim > 256:
            raise InvalidValue(f"{p}.mixer.dim", m.dim, "the recurrence kernel holds at most 256 rows of a state column")
        return m

    @classmethod
    def _delta(cls, L, g, p) -> DeltaConfig:
        m = DeltaConfig(heads=g("mixer.heads", int, minimum=1), kv_heads=g("mixer.kv_heads", int, minimum=1),
                        dim=g("mixer.dim", int, minimum=1), vdim=g("mixer.vdim", int, minimum=1),
                        taps=g("mixer.conv", int, minimum=1))
        cls._shared_heads(p, m.heads, m.kv_heads)
        if m.dim > 256:
            raise InvalidValue(f"{p}.mixer.dim", m.dim, "the recurrence kernel holds at most 256 rows of a state column")
        if m.taps > 16:
            raise InvalidValue(f"{p}.mixer.conv", m.taps, "the convolution kernel takes up to 16 taps")
        return m

    @staticmethod
    def _mlp(L, g, p) -> Optional[DubodraMlp]:
        raw = L.get("mlp")
        if raw is None:
            return None
        kind = raw.get("kind") if isinstance(raw, dict) else None
        if kind == "dense":
            return DubodraMlp("dense", ff=g("mlp.ff", int, minimum=1))
        if kind != "moe":
            raise InvalidValue(f"{p}.mlp.kind", kind, "must be 'dense' or 'moe' (or mlp null)")
        router = raw.get("router") if isinstance(raw.get("router"), dict) else {}
        grouped = router.get("groups") is not None
        scale = g("mlp.router.scale", float, optional=True)
        mlp = DubodraMlp(
            "moe", expert=UnitConfig(g("mlp.expert.ff", int, minimum=1), g("mlp.expert.limit", float, positive=True)),
            shared=(UnitConfig(g("mlp.shared.ff", int, minimum=1), g("mlp.shared.limit", float, positive=True))
                    if raw.get("shared") is not None else None),
            experts=g("mlp.router.experts", int, minimum=1), identity=g("mlp.router.identity", int, optional=True, minimum=0) or 0,
            top=g("mlp.router.top", int, minimum=1), scale=1.0 if scale is None else scale,
            groups=g("mlp.router.groups.count", int, minimum=1) if grouped else 1,
            keep=g("mlp.router.groups.keep", int, minimum=1) if grouped else 1)
        outputs = mlp.experts + mlp.identity
        if mlp.top > outputs:
            raise InvalidValue(f"{p}.mlp.router.top", mlp.top, f"there are only {outputs} experts")
        if mlp.top > 16 or outputs > 1024:
            raise InvalidValue(f"{p}.mlp.router", router, "the routing kernels take up to 16 of up to 1024 experts")
        if outputs % mlp.groups:
            raise InvalidValue(f"{p}.mlp.router.groups.count", mlp.groups, f"must divide experts + identity = {outputs}")
        if mlp.keep > mlp.groups or mlp.keep * (outputs // mlp.groups) < mlp.top:
            raise InvalidValue(f"{p}.mlp.router.groups.keep", mlp.keep, f"must be at most count = {mlp.groups} and leave room for top = {mlp.top}")
        return mlp

    def to_dict(self) -> dict:
        return copy.deepcopy(self.raw)
