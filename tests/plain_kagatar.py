"""A plain, slow restatement of the Kagatar design, one function per mechanism, in torch on the CPU.

It shares nothing with the engine: it reads a dict of tensors by name and the raw config.json dict, runs a whole
sequence from its first token, and returns logits for every token.  Everything is computed in the dtype the caller
asks for (float64 by default).

Notation: T tokens, D = width; H query heads, G key/value heads, d per-head query/key size, e per-head value size.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch

GLU_SLOPE, GLU_SHIFT = 1.702, 1.0


# ---------------------------------------------------------------------------------------------------
# token-local pieces
def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def clamped_ff(h, w_gate, w_up, w_down, limit: float):
    """down(g sigmoid(1.702 g) (u + 1)) with g = min(gate, limit) and u = up kept within +-limit."""
    g = torch.minimum(h @ w_gate.T, torch.tensor(limit, dtype=h.dtype))
    u = torch.clamp(h @ w_up.T, min=-limit, max=limit)
    return (g / (1.0 + torch.exp(-GLU_SLOPE * g)) * (u + GLU_SHIFT)) @ w_down.T


def bounded(z, cap: Optional[float]):
    return z if not cap else cap * torch.tanh(z / cap)


# ---------------------------------------------------------------------------------------------------
# rotation
def yarn_frequencies(dims: int, base: float, s: dict) -> List[float]:
    """Pair i keeps base^(-2i/dims) below the pair that turns `fast` times within `original` positions, has it divided
    by the factor above the pair that turns `slow` times, and takes a mixture in between."""
    pair_of = lambda t: dims * math.log(s["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo = max(math.floor(pair_of(s["fast"])), 0)
    hi = min(math.ceil(pair_of(s["slow"])), dims - 1)
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * r + f * (1.0 - r))
    return out


def yarn_magnitude(s: dict) -> float:
    return 0.1 * math.log(s["factor"]) + 1.0


def wavelength_frequencies(dims: int, base: float, s: dict) -> List[float]:
    """A frequency is kept where its wavelength is short, divided by the factor where it is long, mixed in between."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        wave = 2 * math.pi / f
        if wave < s["original"] / s["high"]:
            out.append(f)
        elif wave > s["original"] / s["low"]:
            out.append(f / s["factor"])
        else:
            m = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
            out.append((1.0 - m) * f / s["factor"] + m * f)
    return out


def rotate_neighbours(x: torch.Tensor, positions, freqs: List[float], magnitude: float = 1.0) -> torch.Tensor:
    """x [T, heads, d]: elements 2i and 2i + 1 of every head turned by position * freqs[i], the turned ones scaled by
    `magnitude`; what lies behind the last pair stays."""
    y = x.clone()
    p = torch.tensor([float(t) for t in positions], dtype=torch.float64)
    for i, f in enumerate(freqs):
        c, s = ((fn(p * f) * magnitude).to(x.dtype)[:, None] for fn in (torch.cos, torch.sin))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i], y[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


# ---------------------------------------------------------------------------------------------------
# attention
def window_of(m: dict) -> int:
    return int((m.get("mask") or {}).get("size") or 0)


def first_key(i: int, size: int) -> int:
    """The first place that the token at place i reads (size 0: no window)."""
    return max(0, i - size + 1) if size > 0 else 0


def softmax_over_sight(q, k, v, scale: float, size: int, cap: Optional[float] = None) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, e] of one sequence -> [T, H, e]: the token at place i reads the places
    first_key(i) .. i; head h reads key/value head h // (H / G)."""
    T, H = q.shape[:2]
    k, v = (t.repeat_interleave(H // t.shape[1], dim=1) for t in (k, v))       # one key/value head per query head
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        seen = slice(first_key(i, size), i + 1)
        s = bounded((k[seen] * q[i]).sum(dim=-1) * scale, cap)                 # [keys seen, H]
        p = torch.exp(s - s.max(dim=0).values)
        out[i] = (p[..., None] * v[seen]).sum(dim=0) / p.sum(dim=0)[:, None]
    return out


def tied_attention(h, w, m: dict, eps: float, positions) -> torch.Tensor:
    """Values are the keys; no positions in the scores."""
    T = h.shape[0]
    q = (h @ w["q"].T + w["q.b"]).view(T, m["heads"], m["dim"])
    k = (h @ w["k"].T + w["k.b"]).view(T, m["kv_heads"], m["dim"])
    o = softmax_over_sight(q, k, k, m["scale"], window_of(m))
    return o.reshape(T, -1) @ w["o"].T


def _qkv(h, w, m):
    T = h.shape[0]
    return ((h @ w["q"].T + w["q.b"]).view(T, m["heads"], m["dim"]), (h @ w["k"].T + w["k.b"]).view(T, m["kv_heads"], m["dim"]),
            (h @ w["v"].T + w["v.b"]).view(T, m["kv_heads"], m["vdim"]))


def gated_attention(h, w, m: dict, eps: float, positions) -> torch.Tensor:
    """Rotated with yarn frequencies, causal, every output element times the sigmoid of its own gate."""
    q, k, v = _qkv(h, w, m)
    rot = m.get("rot")
    if rot:
        s = rot.get("scaling")
        f = yarn_frequencies(rot["dims"], rot["base"], s) if s else [rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)]
        mag = yarn_magnitude(s) if s else 1.0
        q, k = rotate_neighbours(q, positions, f, mag), rotate_neighbours(k, positions, f, mag)
    o = softmax_over_sight(q, k, v, m["scale"], window_of(m)).reshape(h.shape[0], -1)
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def capped_attention(h, w, m: dict, eps: float, positions) -> torch.Tensor:
    """Rotated with stretched frequencies, then every head of q and k divided by its root mean square; scores within
    +-softcap; a window."""
    q, k, v = _qkv(h, w, m)
    rot = m.get("rot")
    if rot:
        s = rot.get("scaling")
        f = wavelength_frequencies(rot["dims"], rot["base"], s) if s else [rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)]
        q, k = rotate_neighbours(q, positions, f), rotate_neighbours(k, positions, f)
    q, k = rms(q, eps), rms(k, eps)
    o = softmax_over_sight(q, k, v, m["scale"], window_of(m), m.get("softcap"))
    return o.reshape(h.shape[0], -1) @ w["o"].T


MIXERS = {"attention": tied_attention, "attention_2": gated_attention, "attention_3": capped_attention}


# ---------------------------------------------------------------------------------------------------
# the whole model
def run_order(cfg: dict) -> List[Tuple[int, Optional[int]]]:
    """[(layer, the pass it opens or None)]: the layers of `loop` run `times` times in a row, the rest once."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    order = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None) for i in range(loop["stop"], n)]


def sub(w: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def open_pass(x, x0, steps, t: int):
    """What happens to the stream ahead of pass t: the embedding's output joins from the second pass on, then the
    pass's own vector."""
    return (x + x0 if t > 0 else x) + steps[t]


def layer_update(x, L: dict, w: Dict[str, torch.Tensor], eps: float, positions):
    """mixer(norm1(x)) + ff(norm2(x)), both of the same x."""
    y = MIXERS[L["type"]](rms(x, eps) * w["norm1"], sub(w, "mix."), L["mixer"], eps, positions)
    if L.get("mlp"):
        y = y + clamped_ff(rms(x, eps) * w["norm2"], w["mlp.gate"], w["mlp.up"], w["mlp.down"],
                           L["mlp"].get("limit", math.inf))
    return y


def forward(weights: Dict[str, torch.Tensor], cfg: dict, tokens, dtype=torch.float64, streams: Optional[list] = None):
    """Logits [T, vocab] of one sequence from its first token.  `streams`: receives the residual stream after every
    layer run."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    ids = torch.as_tensor(tokens, dtype=torch.long)
    x0 = w["embed"][ids] * (cfg.get("embedding") or {}).get("scale", 1.0)
    x = x0
    for i, t in run_order(cfg):
        if t is not None:
            x = open_pass(x, x0, w["loop.step"], t)
        x = x + layer_update(x, cfg["layers"][i], sub(w, f"l{i}."), eps, range(len(ids)))
        if streams is not None:
            streams.append(x.clone())
    return bounded((rms(x, eps) * w["final.norm"]) @ w["embed"].T, cfg.get("logit_softcap"))


def greedy(weights, cfg, prompt, n_new: int, dtype=torch.float64):
    """(tokens, margins): greedy continuation of `prompt`, and at each new token the best logit's lead over the
    second."""
    toks, margins = list(prompt), []
    for _ in range(n_new):
        top = forward(weights, cfg, toks, dtype)[-1].topk(2)
        margins.append(float(top.values[0] - top.values[1]))
        toks.append(int(top.indices[0]))
    return toks, margins
