"""Token embedding and output projection
(crates/ai-engine-runtime/src/arch/embedding.rs:14-20,33-35; tied head:
crates/ai-engine-runtime/src/arch/model.rs:130-134)."""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights.loader import TensorSpec
from .base import Part


class TokenEmbedding(Part):
    """params: vocab_size, hidden_size, alternatives (names that may stand in), scale (absent or 1: none).
    tensors: weight [vocab, hidden].  forward(ctx) -> float32 residual stream [T, hidden] of the
    step's tokens, the table's rows times `scale` (`ctx.token_ids`; an embedding that depends on the place reads `ctx.positions`)."""

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.vocab, self.hidden = int(spec.params["vocab_size"]), int(spec.params["hidden_size"])
        self.scale = float(spec.params["scale"]) if spec.params.get("scale") is not None else 1.0
        self.weight = None

    def tensor_specs(self):
        return [TensorSpec(self.spec.tensors["weight"], (self.vocab, self.hidden),
                           alternatives=tuple(self.spec.params.get("alternatives", ())))]

    def load(self, source):
        self.weight = source.get(self.spec.tensors["weight"])

    def forward(self, ctx):
        return ops.embed_gather(ctx.token_ids, self.weight, ctx.err, scale=self.scale)


class LMHead(Part):
    """params: vocab_size, hidden_size, alternatives, stored, softcap (0 or absent: none; c > 0: the logits
    become c * tanh(logits / c)), scale (absent or 1: none; the logits are multiplied by it, before a softcap).  tensors: weight [vocab, hidden] (the embedding's name when tied).
    forward(h [N, hidden]) -> float32 logits [N, vocab]."""

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.vocab, self.hidden = int(spec.params["vocab_size"]), int(spec.params["hidden_size"])
        self.softcap = float(spec.params.get("softcap") or 0.0)
        self.scale = float(spec.params.get("scale") or 1.0)
        if self.softcap < 0:
            raise ValueError(f"head: softcap must be positive, got {self.softcap}")
        self.weight = None

    def tensor_specs(self):
        return [TensorSpec(self.spec.tensors["weight"], (self.vocab, self.hidden),
                           alternatives=tuple(self.spec.params.get("alternatives", ())),
                           stored=bool(self.spec.params.get("stored", True)))]

    def load(self, source):
        self.weight = source.get(self.spec.tensors["weight"])

    def weight_bytes(self):
        return self.weight.numel() * self.weight.element_size()

    def flops(self, tokens, keys=0.0):
        return 2.0 * tokens * self.vocab * self.hidden

    def forward(self, h, err=None):
        logits = ops.linear(h, self.weight, torch.float32, err)
        if self.scale != 1.0:
            logits = ops.scale_(logits, self.scale)
        return ops.softcap(logits, self.softcap) if self.softcap else logits
