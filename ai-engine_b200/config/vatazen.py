"""VatazenConfig: the typed configuration of a Vatazen model.

config.json names the architecture under `architecture`, the sizes `vocab` and `width`, `norm.eps`,
`embedding.scale`, `token_side.dim` and a list `layers`.  A layer has a `type` (latent_attention | attention), the
sizes and constants of its mixer under `mixer`, and its feed-forward under `mlp` (null: none; kind moe).  Every size
and constant of a model is read here; a missing or ill-typed key is a ConfigError that names it.  Keys that may be
absent mean "none": no mask but causality, no rotation, no scaling of the frequencies, no per-layer token input, an
embedding that is not scaled.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional, Tuple

from .base import ConfigError, get_float, get_int, get_object, named

LAYER_TYPES = ("latent_attention", "attention")


@dataclass(frozen=True)
class YarnScaling:
    """Rotation frequencies stretched by `factor` where a pair turns less than `slow` times within `original`
    positions, kept where it turns more than `fast` times, blended between."""
    factor: float
    original: float
    fast: float
    slow: float

    @classmethod
    def from_dict(cls, s: dict) -> "YarnScaling":
        out = cls(*(get_float(s, k) for k in ("factor", "original", "fast", "slow")))
        for k in ("factor", "original", "fast", "slow"):
            if getattr(out, k) <= 0:
                raise ConfigError(f"config.json: `{k}` must be positive, got {getattr(out, k)}")
        return out

    def to_dict(self) -> dict:
        return dict(factor=self.factor, original=self.original, fast=self.fast, slow=self.slow)


@dataclass(frozen=True)
class VatazenMixer:
    """Sizes of a mixer.  latent_attention: heads with `dim` unrotated and `rot_dim` rotated query/key elements, values
    of `vdim`, a latent of kv_rank, the score's scale, the window `mask_size` (0: all keys), the rotation over the
    first rot_dims rotated elements (0: none) with its base and scaling.  attention: `heads` query heads and kv_heads
    key/value heads of two maps with queries and keys of `dim` each and a value of `vdim`, the scale, the chunk
    `mask_size` (0: all keys) and `diff`, the constant of the second map's weight."""
    heads: int
    dim: int
    vdim: int
    scale: float
    mask_size: int = 0
    kv_heads: int = 0
    diff: float = 0.0
    rot_dim: int = 0
    kv_rank: int = 0
    rot_dims: int = 0
    rot_base: float = 10000.0
    rot_scaling: Optional[YarnScaling] = None

    @classmethod
    def from_dict(cls, kind: str, m: dict) -> "VatazenMixer":
        heads, dim, vdim = get_int(m, "heads"), get_int(m, "dim"), get_int(m, "vdim")
        scale = get_float(m, "scale")
        mask = get_object(m, "mask", required=False)
        size = named(lambda: get_int(mask, "size"), "mask.") if mask else 0
        if kind == "attention":
            kv_heads = get_int(m, "kv_heads", heads)
            if heads % kv_heads:
                raise ConfigError(f"config.json: heads = {heads} is not a multiple of kv_heads = {kv_heads}")
            return cls(heads, dim, vdim, scale, size, kv_heads=kv_heads, diff=get_float(m, "diff"))
        rot_dim = get_int(m, "rot_dim", 0, minimum=0)
        rot = get_object(m, "rot", required=False)
        dims, base, scaling = 0, 10000.0, None
        if rot and rot_dim:
            dims = named(lambda: get_int(rot, "dims", rot_dim, minimum=0), "rot.")
            base = named(lambda: get_float(rot, "base"), "rot.")
            sc = named(lambda: get_object(rot, "scaling", required=False), "rot.")
            scaling = named(lambda: YarnScaling.from_dict(sc), "rot.scaling.") if sc else None
            if dims % 2 or dims > rot_dim:
                raise ConfigError(f"config.json: rot.dims = {dims} must be even and at most rot_dim = {rot_dim}")
        return cls(heads, dim, vdim, scale, size, rot_dim=rot_dim, kv_rank=get_int(m, "kv_rank"), rot_dims=dims,
                   rot_base=base, rot_scaling=scaling)

    def to_dict(self, kind: str) -> dict:
        d = dict(heads=self.heads, dim=self.dim, vdim=self.vdim, scale=self.scale)
        if self.mask_size:
            d["mask"] = dict(size=self.mask_size)
        if kind == "attention":
            d.update(kv_heads=self.kv_heads, diff=self.diff)
            return d
        d.update(rot_dim=self.rot_dim, kv_rank=self.kv_rank)
        if self.rot_dims:
            d["rot"] = dict(base=self.rot_base, dims=self.rot_dims)
            if self.rot_scaling:
                d["rot"]["scaling"] = self.rot_scaling.to_dict()
        return d


@dataclass(frozen=True)
class VatazenFF:
    """`experts` experts without a gate of width `ff`, of which a token uses `top`."""
    ff: int
    experts: int
    top: int

    @classmethod
    def from_dict(cls, f: dict) -> "VatazenFF":
        if f.get("kind") != "moe":
            raise ConfigError(f"config.json: kind `{f.get('kind')}` is not known (moe)")
        expert, router = get_object(f, "expert"), get_object(f, "router")
        out = cls(named(lambda: get_int(expert, "ff"), "expert."), *named(
            lambda: (get_int(router, "experts"), get_int(router, "top")), "router."))
        if out.top > out.experts:
            raise ConfigError(f"config.json: router.top = {out.top} exceeds router.experts = {out.experts}")
        return out

    def to_dict(self) -> dict:
        return dict(kind="moe", expert=dict(ff=self.ff), router=dict(experts=self.experts, top=self.top))


@dataclass(frozen=True)
class VatazenLayer:
    type: str
    mixer: VatazenMixer
    mlp: Optional[VatazenFF] = None

    def to_dict(self) -> dict:
        return dict(type=self.type, mixer=self.mixer.to_dict(self.type), mlp=self.mlp.to_dict() if self.mlp else None)


@dataclass(frozen=True)
class VatazenConfig:
    vocab: int
    width: int
    norm_eps: float
    embed_scale: float = 1.0
    side_dim: int = 0                               # 0: layers have no token input of their own
    layers: Tuple[VatazenLayer, ...] = field(default_factory=tuple)
    max_position_embeddings: int = 1 << 20          # nothing in the design bounds a sequence; the cache does
    eos_token_ids: Tuple[int, ...] = ()

    ARCHITECTURE = "Vatazen"

    @classmethod
    def from_dict(cls, raw: dict) -> "VatazenConfig":
        ls = raw.get("layers")
        if not isinstance(ls, list) or not ls:
            raise ConfigError("config.json: `layers` must be a non-empty list")
        layers = []
        for i, l in enumerate(ls):
            where = f"layers[{i}]."
            if not isinstance(l, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            kind = l.get("type")
            if kind not in LAYER_TYPES:
                raise ConfigError(f"config.json: {where}type `{kind}` is not known ({', '.join(LAYER_TYPES)})")
            m = named(lambda: get_object(l, "mixer"), where)
            mixer = named(lambda: VatazenMixer.from_dict(kind, m), where + "mixer.")
            f = named(lambda: get_object(l, "mlp", required=False), where)
            layers.append(VatazenLayer(kind, mixer, named(lambda: VatazenFF.from_dict(f), where + "mlp.") if f else None))
        norm = get_object(raw, "norm")
        embedding = get_object(raw, "embedding", required=False) or {}
        side = get_object(raw, "token_side", required=False)
        eos = raw.get("eos_token_id")
        eos = () if eos is None else tuple(eos) if isinstance(eos, list) else (eos,)
        return cls(get_int(raw, "vocab"), get_int(raw, "width"), named(lambda: get_float(norm, "eps"), "norm."),
                   named(lambda: get_float(embedding, "scale", 1.0), "embedding."),
                   named(lambda: get_int(side, "dim"), "token_side.") if side else 0, tuple(layers),
                   get_int(raw, "max_position_embeddings", 1 << 20), eos)

    def to_dict(self) -> dict:
        d = dict(architecture=self.ARCHITECTURE, vocab=self.vocab, width=self.width, norm=dict(eps=self.norm_eps),
                 embedding=dict(scale=self.embed_scale), layers=[l.to_dict() for l in self.layers])
        if self.side_dim:
            d["token_side"] = dict(dim=self.side_dim)
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d
