"""Rotary position encoding: the frequencies.

Default (crates/ai-engine-runtime/src/arch/rope.rs:34-36): inv_freq[i] =
1 / theta^(2i/d) in float32.  The reference precomputes cos/sin tables up to
max_position_embeddings; here only inv_freq is kept and kernels compute
cos/sin(float(pos) * inv_freq[i]) in float32, so no table bounds the context.

`linear` scaling divides every frequency by `factor`.  `llama3` scaling is not in the reference (it reads no rope_scaling); it follows
the rule the config keys name: with wavelength = 2*pi / inv_freq, frequencies
whose wavelength is below original/high_freq_factor are kept, above
original/low_freq_factor are divided by `factor`, and between the two are
blended linearly in original/wavelength.

`yarn` scaling: with turns(t) = d * ln(original / (2 pi t)) / (2 ln theta), the pair index at which a rotation makes t
turns within `original` positions, lo = max(floor(turns(fast)), 0) and hi = min(ceil(turns(slow)), d - 1), pair i keeps
its frequency up to lo, has it divided by `factor` from hi on, and takes a linear blend in i between; cosines and
sines are multiplied by 0.1 ln(factor) + 1 (`rotary_magnitude`).
"""
from __future__ import annotations

import math

import numpy as np
import torch

from .base import PositionEncoding


def rotary_inv_freq(rot_dim: int, theta: float, scaling=None) -> np.ndarray:
    i = np.arange(rot_dim // 2, dtype=np.float32)
    base = (np.float32(1.0) / np.power(np.float32(theta), (np.float32(2.0) * i) / np.float32(rot_dim)))
    base = base.astype(np.float32)
    if not scaling:
        return base
    kind = scaling.get("rope_type", scaling.get("type"))
    if kind == "linear":         # every frequency divided by the factor: positions stretched evenly
        return (base.astype(np.float64) / float(scaling["factor"])).astype(np.float32)
    if kind not in ("llama3", "yarn"):
        raise ValueError(f"rotary scaling `{kind}` is not supported (supported: llama3, linear, yarn)")
    factor = float(scaling["factor"])
    if kind == "yarn":
        pair = np.arange(rot_dim // 2, dtype=np.float64)
        f = np.power(float(theta), -2.0 * pair / rot_dim)
        turns = lambda t: rot_dim * math.log(float(scaling["original"]) / (2.0 * math.pi * t)) / (2.0 * math.log(theta))
        lo = max(math.floor(turns(float(scaling["fast"]))), 0)
        hi = min(math.ceil(turns(float(scaling["slow"]))), rot_dim - 1)
        ramp = np.clip((pair - lo) / max(hi - lo, 0.001), 0.0, 1.0)
        return (f / factor * ramp + f * (1.0 - ramp)).astype(np.float32)
    low, high = float(scaling["low_freq_factor"]), float(scaling["high_freq_factor"])
    original = float(scaling["original_max_position_embeddings"])
    f = base.astype(np.float64)
    wavelength = 2.0 * math.pi / f
    smooth = (original / wavelength - low) / (high - low)
    blended = (1.0 - smooth) * f / factor + smooth * f
    out = np.where(wavelength < original / high, f,
                   np.where(wavelength > original / low, f / factor, blended))
    return out.astype(np.float32)


def rotary_magnitude(scaling=None) -> float:
    """What cosines and sines are multiplied by (1 but for yarn scaling)."""
    if scaling and scaling.get("rope_type", scaling.get("type")) == "yarn":
        return 0.1 * math.log(float(scaling["factor"])) + 1.0
    return 1.0


class RotaryEncoding(PositionEncoding):
    """params: rot_dim (elements of each head that are rotated; the full head for
    Llama), theta, scaling (None, the llama3 dict, {"type": "linear", "factor": f}, or {"type": "yarn", factor,
    original, fast, slow}, whose `magnitude` a mixer multiplies cosines and sines by), layout ("halves", the default: element i turns with
    element i + rot_dim / 2; "interleaved": element 2i with 2i + 1; a mixer reads `interleaved`).  Holds
    inv_freq [rot_dim / 2] float32 on the device."""

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.rot_dim = int(spec.params["rot_dim"])
        if self.rot_dim % 2:
            raise ValueError(f"rotary encoding needs an even rot_dim, got {self.rot_dim}")
        self.inv_freq_host = rotary_inv_freq(self.rot_dim, float(spec.params["theta"]),
                                             spec.params.get("scaling"))
        self.magnitude = rotary_magnitude(spec.params.get("scaling"))
        self.inv_freq = None
        layout = spec.params.get("layout") or "halves"
        if layout not in ("halves", "interleaved"):
            raise ValueError(f"rotary encoding: layout `{layout}` is not known (halves, interleaved)")
        self.interleaved = layout == "interleaved"

    def load(self, source):
        self.inv_freq = torch.from_numpy(self.inv_freq_host.copy()).to(self.env.device)

    def rotation(self):
        return self.inv_freq, self.rot_dim
