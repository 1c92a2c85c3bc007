"""Differential attention: two softmax maps over the same values, one taken from the other.

    q = W_q h + b_q,  k = W_k h + b_k,  v = W_v h + b_v
        H query heads and G key/value heads; every head of q and k has two maps of d elements, every value e elements
    every map of every head of q and k is divided by its root mean square, times a weight [d]
    s_m(i, j) = (q_i,m . k_j,m) * scale over the keys j <= i of the same chunk: i / chunk == j / chunk (chunk 0: all)
    a_m = sum_j softmax_j(s_m(i, j)) v_j
    o = a_1 - lambda a_2,   lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff       (one number per layer)
    out = W_o concat_h(o / rms(o) * (1 - diff)) + b_o

Query head h reads key/value head h / (H / G).  Positions enter through the mask only.  A token's two keys and its
value lie side by side in one cache row.  Norms, scores, weights and the difference are float32.
"""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights.loader import TensorSpec
from .attention import ATTENTION_WORK
from .base import KVRequest, Mixer

MAPS = 2


class DifferentialAttention(Mixer):
    """params: hidden_size, num_heads, num_kv_heads, head_dim (of one map), value_dim, scale, chunk (0: all keys), eps,
    diff.  tensors: q [H 2 d, hidden], k [G 2 d, hidden], v [G e, hidden], o [hidden, H e], their biases q_bias,
    k_bias, v_bias, o_bias, q_norm [d], k_norm [d], lq1, lk1, lq2, lk2 [d]."""

    leaves_bias = True

    def __init__(self, spec, env):
        super().__init__(spec, env)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.H, self.G = int(p["num_heads"]), int(p["num_kv_heads"])
        self.d, self.e = int(p["head_dim"]), int(p["value_dim"])
        if self.H % self.G:
            raise ValueError(f"attention: {self.H} heads are not a multiple of {self.G} kv heads")
        if not (0 < self.d <= 256 and 0 < self.e <= 256):
            raise ValueError(f"attention: head sizes {self.d} / {self.e} must be within 1 .. 256")
        self.scale = float(p["scale"]) if p.get("scale") is not None else float(self.d) ** -0.5
        self.chunk, self.eps, self.diff = int(p.get("chunk") or 0), float(p["eps"]), float(p["diff"])
        self.w_in = self.w_o = self.bias = self.output_bias = self.q_w = self.k_w = None
        self.lam = 0.0

    def tensor_specs(self):
        t, Hd, Gd, Ge, He = (self.spec.tensors, self.H * MAPS * self.d, self.G * MAPS * self.d, self.G * self.e,
                             self.H * self.e)
        return [TensorSpec(t["q"], (Hd, self.hidden)), TensorSpec(t["k"], (Gd, self.hidden)),
                TensorSpec(t["v"], (Ge, self.hidden)), TensorSpec(t["o"], (self.hidden, He)),
                TensorSpec(t["q_bias"], (Hd,), std=0.1), TensorSpec(t["k_bias"], (Gd,), std=0.1),
                TensorSpec(t["v_bias"], (Ge,), std=0.1), TensorSpec(t["o_bias"], (self.hidden,), std=0.1),
                TensorSpec(t["q_norm"], (self.d,), init="ones"), TensorSpec(t["k_norm"], (self.d,), init="ones"),
                *(TensorSpec(t[n], (self.d,), std=0.1) for n in ("lq1", "lk1", "lq2", "lk2"))]

    def load(self, source):
        t = self.spec.tensors
        ws = [source.get(t[n]) for n in ("q", "k", "v")]
        dt = torch.float32 if any(w.dtype == torch.float32 for w in ws) else ws[0].dtype
        self.w_in = torch.cat([w.to(dt) for w in ws], dim=0).contiguous()        # [q | k | v]
        self.w_o = source.get(t["o"])
        f32 = lambda name: source.get(t[name]).float().contiguous()
        self.bias = torch.cat([f32("q_bias"), f32("k_bias"), f32("v_bias")]).contiguous()
        self.output_bias, self.q_w, self.k_w = f32("o_bias"), f32("q_norm"), f32("k_norm")
        dot = lambda a, b: (source.get(t[a]).double() * source.get(t[b]).double()).sum()
        self.lam = float(torch.exp(dot("lq1", "lk1")) - torch.exp(dot("lq2", "lk2"))) + self.diff

    def weight_bytes(self):
        return sum(w.numel() * w.element_size() for w in (self.w_in, self.w_o))

    def flops(self, tokens, keys=0.0):
        if self.chunk > 0:
            keys = min(keys, self.chunk / 2.0)
        proj = 2.0 * tokens * self.hidden * (self.w_in.shape[0] + self.H * self.e)
        return proj + 2.0 * tokens * keys * self.H * MAPS * (self.d + self.e)

    def cache_request(self):
        return KVRequest(self.G, MAPS * self.d + self.e, planes=1, chunk=self.chunk)

    def step_planner(self):
        return ATTENTION_WORK

    def forward(self, h, ctx, cache, leave_bias=False):
        """leave_bias: the caller adds `output_bias` (where it reads the output anyway)."""
        proj = ops.linear(h, self.w_in, torch.float32, ctx.err)
        q, _ = ops.normed_attn_prepare(proj, self.bias, self.q_w, self.k_w, self.eps, None, 0, False, cache.k_pages, ctx,
                                       cache.block_table, self.H * MAPS, self.G, self.d, self.e, write=cache.writes,
                                       maps=MAPS, per_head=True)
        a = ops.sink_attention(q, cache.k_pages, None, None, None, None, ctx, ctx.plan(ATTENTION_WORK), cache.block_table,
                               self.e, self.scale, 0, 0, chunk=self.chunk, maps=MAPS, out_dtype=torch.float32)
        a = ops.map_difference(a, self.lam, self.eps, 1.0 - self.diff, self.env.dtype)
        y = ops.linear_parts(a, self.w_o, ctx.err)
        return y if leave_bias else ops.add_bias_(y, self.output_bias)
