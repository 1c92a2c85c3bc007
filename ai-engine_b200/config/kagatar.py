"""KagatarConfig: the typed configuration of a Kagatar model.

config.json names the architecture under `architecture`, the sizes `vocab` and `width`, `norm.eps`, `embedding.scale`,
`logit_softcap`, a group of layers that runs several times (`loop`: start, stop, times) and a list `layers`.  A layer
has a `type` (attention | attention_2 | attention_3), the sizes and constants of its mixer under `mixer`, and its
feed-forward under `mlp` (null: none; kind dense).  Every size and constant of a model is read here; a missing or
ill-typed key is a ConfigError that names it.  Keys that may be absent mean "none": no window, no rotation, no scaling
of the frequencies, no bound on scores or logits, no loop, an embedding that is not scaled.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import List, Optional, Tuple

from .base import ConfigError, get_float, get_int, get_object, named
from .vatazen import YarnScaling

TIED, GATED, CAPPED = "attention", "attention_2", "attention_3"
LAYER_TYPES = (TIED, GATED, CAPPED)


@dataclass(frozen=True)
class WavelengthScaling:
    """Rotation frequencies kept where the wavelength is under original / high, divided by `factor` where it is over
    original / low, blended between."""
    factor: float
    low: float
    high: float
    original: float

    @classmethod
    def from_dict(cls, s: dict) -> "WavelengthScaling":
        out = cls(*(get_float(s, k) for k in ("factor", "low", "high", "original")))
        for k in ("factor", "low", "high", "original"):
            if getattr(out, k) <= 0:
                raise ConfigError(f"config.json: `{k}` must be positive, got {getattr(out, k)}")
        if out.high <= out.low:
            raise ConfigError(f"config.json: high = {out.high} must exceed low = {out.low}")
        return out

    def to_dict(self) -> dict:
        return dict(factor=self.factor, low=self.low, high=self.high, original=self.original)


@dataclass(frozen=True)
class KagatarMixer:
    """Sizes of a mixer: `heads` query heads of `dim`, kv_heads key/value heads with values of `vdim`, the score's scale
    and the window (0: all keys).  attention: the values are the keys, no rotation.  attention_2: rotation with yarn
    scaling, a gate on every output element.  attention_3: rotation with wavelength scaling, unit heads, scores within
    +-softcap (0: no bound)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0
    rot_dims: int = 0                    # 0: no rotation
    rot_base: float = 10000.0
    rot_scaling: Optional[object] = None
    softcap: float = 0.0

    @classmethod
    def from_dict(cls, kind: str, m: dict) -> "KagatarMixer":
        heads, dim = get_int(m, "heads"), get_int(m, "dim")
        kv_heads, vdim = get_int(m, "kv_heads", heads), get_int(m, "vdim", dim)
        if heads % kv_heads:
            raise ConfigError(f"config.json: heads = {heads} is not a multiple of kv_heads = {kv_heads}")
        if kind == TIED and vdim != dim:
            raise ConfigError(f"config.json: the values are the keys: vdim = {vdim} must equal dim = {dim}")
        mask = get_object(m, "mask", required=False)
        window = named(lambda: get_int(mask, "size"), "mask.") if mask else 0
        dims, base, scaling, cap = 0, 10000.0, None, 0.0
        rot = get_object(m, "rot", required=False) if kind != TIED else None
        if rot:
            dims = named(lambda: get_int(rot, "dims", dim, minimum=0), "rot.")
            base = named(lambda: get_float(rot, "base"), "rot.")
            sc = named(lambda: get_object(rot, "scaling", required=False), "rot.")
            reader = YarnScaling if kind == GATED else WavelengthScaling
            scaling = named(lambda: reader.from_dict(sc), "rot.scaling.") if sc else None
            if dims % 2 or dims > dim:
                raise ConfigError(f"config.json: rot.dims = {dims} must be even and at most dim = {dim}")
        if kind == CAPPED:
            cap = get_float(m, "softcap", 0.0)
            if cap < 0:
                raise ConfigError(f"config.json: `softcap` must not be negative, got {cap}")
        return cls(heads, kv_heads, dim, vdim, get_float(m, "scale"), window, dims, base, scaling, cap)

    def to_dict(self) -> dict:
        d = dict(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, scale=self.scale)
        if self.window:
            d["mask"] = dict(size=self.window)
        if self.rot_dims:
            d["rot"] = dict(base=self.rot_base, dims=self.rot_dims)
            if self.rot_scaling:
                d["rot"]["scaling"] = self.rot_scaling.to_dict()
        if self.softcap:
            d["softcap"] = self.softcap
        return d


@dataclass(frozen=True)
class KagatarFF:
    """A gated feed-forward of width `ff` whose gate is kept under `limit` and whose up branch within +-limit."""
    ff: int
    limit: float = math.inf

    @classmethod
    def from_dict(cls, f: dict) -> "KagatarFF":
        if f.get("kind") != "dense":
            raise ConfigError(f"config.json: kind `{f.get('kind')}` is not known (dense)")
        out = cls(get_int(f, "ff"), get_float(f, "limit", math.inf))
        if not out.limit > 0:
            raise ConfigError(f"config.json: `limit` must be positive, got {out.limit}")
        return out

    def to_dict(self) -> dict:
        d = dict(kind="dense", ff=self.ff)
        if math.isfinite(self.limit):
            d["limit"] = self.limit
        return d


@dataclass(frozen=True)
class KagatarLayer:
    type: str
    mixer: KagatarMixer
    mlp: Optional[KagatarFF] = None

    def to_dict(self) -> dict:
        return dict(type=self.type, mixer=self.mixer.to_dict(), mlp=self.mlp.to_dict() if self.mlp else None)


@dataclass(frozen=True)
class KagatarConfig:
    vocab: int
    width: int
    norm_eps: float
    embed_scale: float = 1.0
    logit_softcap: float = 0.0           # 0: the logits are not bounded
    layers: Tuple[KagatarLayer, ...] = field(default_factory=tuple)
    loop_start: int = 0                  # layers loop_start .. loop_stop - 1 run loop_times times in a row;
    loop_stop: int = 0                   # loop_times 0: the model has no loop
    loop_times: int = 0
    max_position_embeddings: int = 1 << 20          # nothing in the design bounds a sequence; the cache does
    eos_token_ids: Tuple[int, ...] = ()

    ARCHITECTURE = "Kagatar"

    @classmethod
    def from_dict(cls, raw: dict) -> "KagatarConfig":
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
            mixer = named(lambda: KagatarMixer.from_dict(kind, m), where + "mixer.")
            f = named(lambda: get_object(l, "mlp", required=False), where)
            layers.append(KagatarLayer(kind, mixer, named(lambda: KagatarFF.from_dict(f), where + "mlp.") if f else None))
        norm = get_object(raw, "norm")
        embedding = get_object(raw, "embedding", required=False) or {}
        loop = get_object(raw, "loop", required=False)
        start = stop = times = 0
        if loop:
            start, stop, times = (named(lambda k=k, n=n: get_int(loop, k, minimum=n), "loop.")
                                  for k, n in (("start", 0), ("stop", 0), ("times", 1)))
            if not start < stop <= len(layers):
                raise ConfigError(f"config.json: loop.start = {start} and loop.stop = {stop} must name layers "
                                  f"(0 <= start < stop <= {len(layers)})")
        cap = get_float(raw, "logit_softcap", 0.0)
        if cap < 0:
            raise ConfigError(f"config.json: `logit_softcap` must not be negative, got {cap}")
        eos = raw.get("eos_token_id")
        eos = () if eos is None else tuple(eos) if isinstance(eos, list) else (eos,)
        return cls(get_int(raw, "vocab"), get_int(raw, "width"), named(lambda: get_float(norm, "eps"), "norm."),
                   named(lambda: get_float(embedding, "scale", 1.0), "embedding."), cap, tuple(layers), start, stop, times,
                   get_int(raw, "max_position_embeddings", 1 << 20), eos)

    def to_dict(self) -> dict:
        d = dict(architecture=self.ARCHITECTURE, vocab=self.vocab, width=self.width, norm=dict(eps=self.norm_eps),
                 embedding=dict(scale=self.embed_scale), layers=[l.to_dict() for l in self.layers])
        if self.logit_softcap:
            d["logit_softcap"] = self.logit_softcap
        if self.loop_times:
            d["loop"] = dict(start=self.loop_start, stop=self.loop_stop, times=self.loop_times)
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

    def run_order(self) -> List[Tuple[int, int]]:
        """(layer, pass) in the order they run: the loop's layers `loop_times` times in a row, the others once (as
        pass 0)."""
        n = len(self.layers)
        if not self.loop_times:
            return [(i, 0) for i in range(n)]
        return ([(i, 0) for i in range(self.loop_start)]
                + [(i, t) for t in range(self.loop_times) for i in range(self.loop_start, self.loop_stop)]
                + [(i, 0) for i in range(self.loop_stop, n)])
