"""What a mixer reads, moved towards the token before: h_t + (h_(t-1) - h_t) * s element by element, zeros before the
sequence's first token.  The last h of a request, as it was before the shift, is state of the request; a portion of a
prompt or a single decoded token continues from it."""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights.loader import TensorSpec
from .base import StateRequest, TokenFilter


class TokenShift(TokenFilter):
    """params: size (channels).  tensors: weight [size].  Input float32 rows, output in the compute dtype; with
    `plain` it returns (shifted, the input in the compute dtype).  `ahead(cache)` hands (weight, state) to a kernel
    that makes a step's input of this part itself (steps in which every request brings one token)."""

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.size = int(spec.params["size"])
        self.weight = None

    def tensor_specs(self):
        return [TensorSpec(self.spec.tensors["weight"], (self.size,), mean=0.5, std=0.3)]

    def load(self, source):
        self.weight = source.get(self.spec.tensors["weight"]).float().contiguous()

    def weight_bytes(self):
        return self.weight.numel() * 4

    def state_request(self):
        return StateRequest((self.size,), torch.float32)

    def ahead(self, cache):
        return self.weight, cache.state

    def forward(self, h, ctx, cache, plain=False):
        return ops.token_shift(h, self.weight, cache.state, ctx, self.env.dtype, plain=plain)
