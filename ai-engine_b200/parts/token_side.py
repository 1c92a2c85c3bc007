"""A learned input per layer and token: every layer has a slice e of `size` numbers in one table row per token, and
adds norm(W_proj (gelu_tanh(W_gate x) * e)) to the stream.  This part makes W_proj (gelu_tanh(W_gate x) * e); the
block norms and adds it."""
from __future__ import annotations

from ..kernels import ops
from ..weights.loader import TensorSpec
from .base import FeedForward


class TokenSide(FeedForward):
    """params: hidden_size, size (numbers per layer), vocab_size, layers (of the table), index (this layer's slice).
    tensors: table [vocab, layers * size] (one for all layers), gate [size, hidden], proj [hidden, size]."""

    def __init__(self, spec, env):
        super().__init__(spec, env)
        p = spec.params
        self.hidden, self.n, self.vocab = int(p["hidden_size"]), int(p["size"]), int(p["vocab_size"])
        self.levels, self.index = int(p["layers"]), int(p["index"])
        if not 0 <= self.index < self.levels:
            raise ValueError(f"token side input: slice {self.index} of a table of {self.levels}")
        self.table = self.w_gate = self.w_proj = None

    def tensor_specs(self):
        t = self.spec.tensors
        return [TensorSpec(t["table"], (self.vocab, self.levels * self.n)), TensorSpec(t["gate"], (self.n, self.hidden)),
                TensorSpec(t["proj"], (self.hidden, self.n))]

    def load(self, source):
        t = self.spec.tensors
        self.table, self.w_gate, self.w_proj = (source.get(t[n]) for n in ("table", "gate", "proj"))

    def weight_bytes(self):
        return sum(w.numel() * w.element_size() for w in (self.w_gate, self.w_proj))

    def flops(self, tokens, keys=0.0):
        return 4.0 * tokens * self.n * self.hidden

    def forward(self, h, ctx):
        z = ops.linear_parts(h, self.w_gate, ctx.err)
        g = ops.side_gate(z, ctx.token_ids, self.table, self.index * self.n, self.n, self.env.dtype, ctx.err)
        return ops.linear_parts(g, self.w_proj, ctx.err)
