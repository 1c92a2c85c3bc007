"""A plain, slow restatement of the Vatazen design, one function per mechanism, whole sequences only, on the CPU.

It shares no code with the engine: weights come as a dict name -> tensor, the configuration as the parsed
config.json.  Everything is computed in `dtype` (float64 by default), so it is the yardstick for both of the
engine's precisions.

    layer:    y = mixer(shifted(x)) * gate1(x);   x = x + norm1(y);   y = ff(x) * gate2(x);   x = x + norm2(y)
              x = x + side(x, token)
    mixers:   latent attention with a window, a sink and YaRN positions | differential attention in chunks
    ff:       experts without a gate, chosen by a router with a bias
"""
from __future__ import annotations

import math

import torch


def rms(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def token_shift(x, s):
    """Every channel moves from this token's value towards the one before it (zero before the first) by s."""
    before = torch.cat([torch.zeros_like(x[:1]), x[:-1]], dim=0)
    return x + (before - x) * s


def residual_gate(x, W, name):
    return torch.sigmoid(x @ W[name].T + W[name + ".b"])


def yarn_frequencies(dims, base, scaling, dtype=torch.float64):
    """(frequencies [dims / 2], factor of cos and sin)."""
    i = torch.arange(dims // 2, dtype=dtype)
    f = base ** (-2.0 * i / dims)
    if not scaling:
        return f, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def turns_at(t):
        return dims * math.log(original / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo = max(math.floor(turns_at(float(scaling["fast"]))), 0)
    hi = min(math.ceil(turns_at(float(scaling["slow"]))), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate_interleaved(x, pos, rot):
    """x [T, heads, n]: element 2i turns with element 2i + 1, 2i + 1 < dims; the rest passes."""
    dims = rot["dims"]
    f, m = yarn_frequencies(dims, float(rot["base"]), rot.get("scaling"), x.dtype)
    a = pos.to(x.dtype)[:, None] * f[None, :]
    c, s = (torch.cos(a) * m)[:, None, :], (torch.sin(a) * m)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def sink_softmax(s, sink):
    """softmax over the last axis of s [H, i, j] with exp(sink[h]) added to the denominator."""
    top = torch.maximum(s.max(dim=-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(s - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink[:, None, None] - top))


def latent_attention(h, W, p, m, eps):
    T = h.shape[0]
    H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    q = (h @ W[p + "q"].T).view(T, H, d + r)
    kv = h @ W[p + "dkv"].T
    c = rms(kv[:, :rank], W[p + "dkv.norm"], eps)
    q_rot, k_rot = q[..., d:], kv[:, rank:].view(T, 1, r)
    if m.get("rot"):
        q_rot, k_rot = rotate_interleaved(q_rot, pos, m["rot"]), rotate_interleaved(k_rot, pos, m["rot"])
    k = (c @ W[p + "uk"].T).view(T, H, d)
    v = (c @ W[p + "uv"].T).view(T, H, dv)
    s = (torch.einsum("ihd,jhd->hij", q[..., :d], k) + torch.einsum("ihd,jd->hij", q_rot, k_rot[:, 0])) * m["scale"]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    size = (m.get("mask") or {}).get("size", 0)
    if size:
        seen = seen & (i - j < size)
    pr = sink_softmax(s.masked_fill(~seen, float("-inf")), W[p + "sink"])
    return torch.einsum("hij,jhd->ihd", pr, v).reshape(T, H * dv) @ W[p + "o"].T


def differential_lambda(W, p, m):
    return (torch.exp((W[p + "lq1"] * W[p + "lk1"]).sum()) - torch.exp((W[p + "lq2"] * W[p + "lk2"]).sum()) + m["diff"])


def differential_attention(h, W, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m["vdim"]
    proj = lambda n: h @ W[p + n].T + W[p + n + ".b"]
    q = rms(proj("q").view(T, H, 2, d), W[p + "q.norm"], eps)
    k = rms(proj("k").view(T, G, 2, d), W[p + "k.norm"], eps).repeat_interleave(H // G, dim=1)
    v = proj("v").view(T, G, dv).repeat_interleave(H // G, dim=1)
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    size = (m.get("mask") or {}).get("size", 0)
    if size:
        seen = seen & (i // size == j // size)
    maps = []
    for n in range(2):
        s = torch.einsum("ihd,jhd->hij", q[:, :, n], k[:, :, n]) * m["scale"]
        maps.append(torch.einsum("hij,jhd->ihd", torch.softmax(s.masked_fill(~seen, float("-inf")), dim=-1), v))
    o = maps[0] - differential_lambda(W, p, m) * maps[1]
    o = rms(o, 1.0, eps) * (1.0 - m["diff"])
    return o.reshape(T, H * dv) @ W[p + "o"].T + W[p + "o.b"]


def route(h, W, p, router, margins_out=None):
    """(chosen experts [T, top], their weights [T, top]).  margins_out: a list that receives, per token, the lead of
    the last chosen logit over the first one left out."""
    top = router["top"]
    z = h @ W[p + "router"].T + W[p + "router.b"]
    val, ids = z.topk(top, dim=-1)
    if margins_out is not None:
        s = z.sort(dim=-1, descending=True).values
        margins_out.append(s[:, top - 1] - s[:, top] if top < z.shape[1] else torch.full((z.shape[0],), float("inf"), dtype=z.dtype))
    return ids, torch.softmax(val, dim=-1)


def moe_ff(h, W, p, f, margins_out=None):
    ids, w = route(h, W, p, f["router"], margins_out)
    out = torch.zeros(h.shape[0], W[p + "e0.down"].shape[0], dtype=h.dtype)
    for t in range(h.shape[0]):
        for e, we in zip(ids[t].tolist(), w[t]):
            a = torch.relu(W[f"{p}e{e}.up"] @ h[t])
            out[t] += we * (W[f"{p}e{e}.down"] @ (a * a))
    return out


def token_side(x, W, p, tokens, i, dim, eps):
    e = W["side.embed"][tokens][:, i * dim:(i + 1) * dim]
    g = gelu_tanh(x @ W[p + "side.gate"].T) * e
    return rms(g @ W[p + "side.proj"].T, W[p + "side.norm"], eps)


def forward(cfg, weights, tokens, dtype=torch.float64, margins_out=None):
    """(logits [T, vocab], the stream behind every layer [L, T, width]).  margins_out: see `route`, one entry a
    layer."""
    W = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    ids = torch.as_tensor(tokens, dtype=torch.long)
    x = W["embed"][ids] * cfg.get("embedding", {}).get("scale", 1.0)
    streams = []
    mixers = {"latent_attention": latent_attention, "attention": differential_attention}
    for i, l in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = mixers[l["type"]](token_shift(x, W[p + "shift"]), W, p + "mix.", l["mixer"], eps)
        x = x + rms(y * residual_gate(x, W, p + "rg1"), 1.0 + W[p + "norm1"], eps)
        if l.get("mlp"):
            y = moe_ff(x, W, p + "mlp.", l["mlp"], margins_out)
            x = x + rms(y * residual_gate(x, W, p + "rg2"), 1.0 + W[p + "norm2"], eps)
        if cfg.get("token_side"):
            x = x + token_side(x, W, p, ids, i, cfg["token_side"]["dim"], eps)
        streams.append(x)
    h = rms(x, 1.0 + W["final.norm"], eps)
    return h @ W["embed"].T, torch.stack(streams)
