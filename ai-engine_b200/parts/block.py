"""The pre-norm residual block (crates/ai-engine-runtime/src/arch/block.rs:13-27):
x = x + mixer(norm(x)); x = x + ffn(norm(x)).

The residual stream stays float32.  A branch's output is not added by a kernel
of its own: it travels as `pending` into the next norm, which adds it in
float32, stores the sum and normalises it in one pass over the row.
"""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights.loader import TensorSpec
from .base import Block


class PreNormBlock(Block):
    """x = x + mixer(norm(x)); x = x + ffn(norm(x)).  The feed-forward with its norm is optional.

    With the tensor `input_mix` [hidden, 2 hidden], the block first replaces the stream by a projection of the
    stream and the embedding's output side by side, x <- W [x ; x0] (a layer that opens a pass over a group of
    layers which is run several times: every pass starts from the running stream and the embedding together).  The
    projection reads both in the compute dtype and writes the new float32 stream."""

    roles = {"mixer_norm": "norm", "mixer": "mixer", "ffn_norm": "norm", "ffn": "feed_forward"}
    optional_roles = ("ffn_norm", "ffn")

    def __init__(self, spec, env, parts):
        super().__init__(spec, env)
        self.mixer_norm, self.mixer = parts["mixer_norm"], parts["mixer"]
        self.ffn_norm, self.ffn = parts.get("ffn_norm"), parts.get("ffn")
        if (self.ffn is None) != (self.ffn_norm is None):
            raise ValueError("pre-norm block: a feed-forward comes with its norm")
        self.hidden = env.hidden_size
        self.w_mix = None
        self.needs_embedding_output = self.replaces_stream = "input_mix" in spec.tensors

    def tensor_specs(self):
        name = self.spec.tensors.get("input_mix")
        return [TensorSpec(name, (self.hidden, 2 * self.hidden))] if name else []

    def load(self, source):
        name = self.spec.tensors.get("input_mix")
        if name:
            self.w_mix = source.get(name)

    def weight_bytes(self):
        return self.w_mix.numel() * self.w_mix.element_size() if self.w_mix is not None else 0

    def flops(self, tokens, keys=0.0):
        return 4.0 * tokens * self.hidden * self.hidden if self.w_mix is not None else 0.0

    def forward(self, x, pending, ctx, caches):
        if self.w_mix is not None:
            both = ops.join_streams(x, pending, ctx.embedding_output, self.env.dtype)
            x, pending = ops.linear(both, self.w_mix, torch.float32, ctx.err), None
        h = self.mixer_norm.forward(x, pending)
        if self.mixer.adds_in_place:      # a large step's output projection adds to the stream itself: a is None then
            a = self.mixer.forward(h, ctx, caches.get("mixer"), add_to=x)
        else:
            a = self.mixer.forward(h, ctx, caches.get("mixer"))
        if self.ffn is None:
            return x, a
        h = self.ffn_norm.forward(x, a)
        if self.ffn.adds_in_place:
            return x, self.ffn.forward(h, ctx, add_to=x)
        return x, self.ffn.forward(h, ctx)


class DepthAveragedBlock(Block):
    """A pre-norm block whose sublayers read their input through a filter over time, and whose result is
    averaged with the results of all earlier layers:

        h = filter(norm(x));  x = x + mixer(h);  h = filter(norm(x));  x = x + ffn(h)          -> X_(depth + 1)
        x = sum_{j = 0 .. depth + 1} coef[j] * X_j        (X_0: the stream the first layer received)

    The filters and the feed-forward (with its norm) are optional roles.  params: depth (number of layers
    before this one), levels (layers of the model + 1).  tensors: coef [depth + 2] (absent: no averaging).
    The streams X_j of a step live in one float32 buffer [levels, T, hidden] that the first layer makes
    and hangs on the step context; norms hand float32 rows to the filters."""

    roles = {"mixer_norm": "norm", "mixer_filter": "filter", "mixer": "mixer",
             "ffn_norm": "norm", "ffn_filter": "filter", "ffn": "feed_forward"}
    optional_roles = ("mixer_filter", "ffn_norm", "ffn_filter", "ffn")

    def __init__(self, spec, env, parts):
        super().__init__(spec, env)
        self.p = parts
        self.depth, self.levels = int(spec.params["depth"]), int(spec.params["levels"])
        if "ffn" in parts and "ffn_norm" not in parts:
            raise ValueError("depth-averaged block: a feed-forward needs its norm")
        self.coef = None

    def tensor_specs(self):
        name = self.spec.tensors.get("coef")
        n = self.depth + 2
        return [TensorSpec(name, (n,), mean=1.0 / n, std=0.1 / n)] if name else []

    def load(self, source):
        name = self.spec.tensors.get("coef")
        if name:
            self.coef = source.get(name).float().contiguous()

    def _filtered(self, role, h, ctx, caches):
        f = self.p.get(role)
        if f is None:
            return ops.cast(h, self.env.dtype)
        return f.forward(h, ctx, caches[role])

    def forward(self, x, pending, ctx, caches):
        h = self.p["mixer_norm"].forward(x, pending)
        if self.coef is not None:
            if self.depth == 0:
                ctx.depth_history = torch.empty((self.levels,) + tuple(x.shape), dtype=torch.float32, device=x.device)
                ctx.depth_history[0].copy_(x)
            history = ctx.depth_history
        h = self._filtered("mixer_filter", h, ctx, caches)
        mixer = self.p["mixer"]
        if mixer.adds_in_place:
            a = mixer.forward(h, ctx, caches.get("mixer"), add_to=x)
        else:
            a = mixer.forward(h, ctx, caches.get("mixer"))
        ffn = self.p.get("ffn")
        if ffn is not None:
            h = self.p["ffn_norm"].forward(x, a)
            h = self._filtered("ffn_filter", h, ctx, caches)
            a = ffn.forward(h, ctx, add_to=x) if ffn.adds_in_place else ffn.forward(h, ctx)
        if self.coef is None:
            return x, a
        ops.depth_average(x, a, history, self.coef, self.depth + 1)
        return x, None


class SandwichNormBlock(Block):
    """A block that normalises each sublayer's input and its output:

        x = x + post_norm(mixer(norm(x)));   x = x + ffn_post_norm(ffn(ffn_norm(x)))

    The feed-forward with its two norms is optional.  A post-norm reads the branch in float32 and hands its
    float32 result on as the pending branch, which the next norm adds to the stream."""

    roles = {"mixer_norm": "norm", "mixer": "mixer", "mixer_post_norm": "norm",
             "ffn_norm": "norm", "ffn": "feed_forward", "ffn_post_norm": "norm"}
    optional_roles = ("ffn_norm", "ffn", "ffn_post_norm")

    def __init__(self, spec, env, parts):
        super().__init__(spec, env)
        self.p = parts
        if ("ffn" in parts) != ("ffn_norm" in parts) or ("ffn" in parts) != ("ffn_post_norm" in parts):
            raise ValueError("sandwich block: a feed-forward comes with both of its norms")

    @staticmethod
    def _normed(norm, y):
        """norm(y) in float32 for a branch y [T, D] (any dtype) or float32 [parts, T, D] (summed first)."""
        if y.dim() == 3:
            return norm.forward(y[0], y[1:] if y.shape[0] > 1 else None, write_back=False)
        return norm.forward(ops.cast(y, torch.float32), None, write_back=False)

    def forward(self, x, pending, ctx, caches):
        h = self.p["mixer_norm"].forward(x, pending)
        pending = self._normed(self.p["mixer_post_norm"], self.p["mixer"].forward(h, ctx, caches.get("mixer")))
        ffn = self.p.get("ffn")
        if ffn is not None:
            h = self.p["ffn_norm"].forward(x, pending)
            pending = self._normed(self.p["ffn_post_norm"], ffn.forward(h, ctx))
        return x, pending


class ParallelBlock(Block):
    """A block whose mixer and feed-forward read the same normed input and are added together:

        h = norm(x);   X = x + mult * (mixer(h) + ffn(h))                                 -> X_(depth + 1)
        x = sum_{j = 0 .. depth + 1} coef[j] * X_j        (X_0: the stream the first layer received)

    The feed-forward is optional, and so is the averaging (no tensor `coef`: x = X).  params: mult (default 1),
    depth (number of layers before this one), levels (layers of the model + 1).  tensors: coef [depth + 2].
    The two branch outputs, the stream and the earlier streams meet in one kernel.  `norm_ahead` (set by the model
    builder's order of layers through `set_next_norm`): when the norm that reads the stream next is one without
    statistics, that kernel writes its output too and hangs it on the step for the next block to pick up."""

    roles = {"norm": "norm", "mixer": "mixer", "ffn": "feed_forward"}
    optional_roles = ("ffn",)

    def __init__(self, spec, env, parts):
        super().__init__(spec, env)
        self.norm, self.mixer, self.ffn = parts["norm"], parts["mixer"], parts.get("ffn")
        self.mult = float(spec.params.get("mult", 1.0))
        self.depth, self.levels = int(spec.params.get("depth") or 0), int(spec.params.get("levels") or 0)
        self.coef = None
        self.next_norm = None

    def tensor_specs(self):
        name = self.spec.tensors.get("coef")
        n = self.depth + 2
        return [TensorSpec(name, (n,), mean=1.0 / n, std=0.1 / n)] if name else []

    def load(self, source):
        name = self.spec.tensors.get("coef")
        if name:
            self.coef = source.get(name).float().contiguous()

    def first_norm(self):
        return self.norm

    def set_next_norm(self, norm) -> None:
        """The norm that reads the stream after this block (the next block's, or the model's last); used only if it
        can be made ahead (`ahead()`) and hands on the compute dtype."""
        self.next_norm = norm if hasattr(norm, "ahead") else None

    def forward(self, x, pending, ctx, caches):
        ahead = getattr(ctx, "normed_ahead", None)
        if pending is None and ahead is not None and ahead[0] is self.norm:
            h = ahead[1]
        else:
            h = self.norm.forward(x, pending)
        ctx.normed_ahead = None
        history = None
        if self.coef is not None:
            if self.depth == 0:
                ctx.depth_history = torch.empty((self.levels,) + tuple(x.shape), dtype=torch.float32, device=x.device)
                ctx.depth_history[0].copy_(x)
            history = ctx.depth_history
        a = self.mixer.forward(h, ctx, caches.get("mixer"))
        b = self.ffn.forward(h, ctx) if self.ffn is not None else None
        a, b = ops.cast(a, torch.float32), (ops.cast(b, torch.float32) if b is not None else None)
        nxt = self.next_norm
        made = ops.parallel_residual(x, a, b, self.mult, history, self.coef, self.depth + 1,
                                     norm_ahead=nxt.ahead() if nxt is not None else None,
                                     out_dtype=nxt.out_dtype if nxt is not None else None)
        if made is not None:
            ctx.normed_ahead = (nxt, made)
        return x, None


class TwoNormParallelBlock(Block):
    """A block whose mixer and feed-forward read the same stream, each behind a norm of its own, and are added together:

        x = x + (mixer(mixer_norm(x)) + ffn(ffn_norm(x)))

    The feed-forward with its norm is optional.  With the tensor `pass_steps` [passes, hidden] the layer opens a pass over
    a group of layers that runs several times (params: passes): what it reads, and what its branches are added to, is

        x + steps[0] in the first pass,     (x + x0) + steps[t] in pass t > 0,     x0 the embedding's output

    with t = ctx.pass_index.  One kernel adds what the branches before left, opens the pass and makes both norms' outputs
    (a row has one root mean square).  Where both branches can leave their last product to the block, the two products
    of a small step write their parts side by side into one buffer, which is the next norm's pending branch; in larger
    steps both add to the stream in place."""

    roles = {"mixer_norm": "norm", "mixer": "mixer", "ffn_norm": "norm", "ffn": "feed_forward"}
    optional_roles = ("ffn_norm", "ffn")

    def __init__(self, spec, env, parts):
        super().__init__(spec, env)
        self.mixer_norm, self.mixer = parts["mixer_norm"], parts["mixer"]
        self.ffn_norm, self.ffn = parts.get("ffn_norm"), parts.get("ffn")
        if (self.ffn is None) != (self.ffn_norm is None):
            raise ValueError("two-norm block: a feed-forward comes with its norm")
        if not self.mixer_norm.pairs_with(self.ffn_norm):
            raise ValueError("two-norm block: both norms divide by the same root mean square")
        for part in (self.mixer, self.ffn):
            if part is not None and not part.leaves_projection:
                raise ValueError("two-norm block: both branches leave their last product to the block")
        self.hidden = env.hidden_size
        self.needs_embedding_output = "pass_steps" in spec.tensors and int(spec.params["passes"]) > 1
        self.steps = None

    def tensor_specs(self):
        name = self.spec.tensors.get("pass_steps")
        return [TensorSpec(name, (int(self.spec.params["passes"]), self.hidden), std=0.5)] if name else []

    def load(self, source):
        name = self.spec.tensors.get("pass_steps")
        if name:
            self.steps = source.get(name).float().contiguous()

    def forward(self, x, pending, ctx, caches):
        step = extra = None
        if self.steps is not None:
            step = self.steps[ctx.pass_index]
            extra = ctx.embedding_output if ctx.pass_index > 0 else None
        h, h2 = self.mixer_norm.forward_pair(self.ffn_norm, x, pending, extra, step)
        branches = [self.mixer.forward(h, ctx, caches.get("mixer"), leave_projection=True)]
        if self.ffn is not None:
            branches.append(self.ffn.forward(h2, ctx, leave_projection=True))
        if all(ops.linear_adds(x, a, w) for a, w in branches):
            for a, w in branches:
                ops.linear_add(x, a, w)
            return x, None
        return x, ops.linear_parts_together(branches, ctx.err)


class GatedPostNormBlock(Block):
    """A block whose sublayers read the stream as it is and whose results are gated and normed before they join it:

        y = mixer(shift(x)) * sigmoid(W_g1 x + b_g1);   x = x + mixer_norm(y)
        y = ffn(x) * sigmoid(W_g2 x + b_g2);            x = x + ffn_norm(y)
        x = x + side_norm(side(x))

    Roles: `shift` (a filter over time in front of the mixer) is optional, so are the feed-forward with its norm, and
    `side` (a token-local part that closes the layer) with its norm.  tensors: mixer_gate [hidden, hidden] with
    mixer_gate_bias [hidden], ffn_gate with ffn_gate_bias (each pair optional: no gate).

    The stream changes in one kernel a sublayer, which joins the parts of the products (or the expert rows), adds the
    projection's bias, gates, norms, adds, and hands on the new stream in the compute dtype.  A router whose weight the
    feed-forward hands out is a product with the feed-forward's gate.  In steps in which every request brings one
    token the layer's last kernel makes the next layer's shift too (`set_next_block`) and hangs it on the step."""

    roles = {"shift": "filter", "mixer": "mixer", "mixer_norm": "norm", "ffn": "feed_forward", "ffn_norm": "norm",
             "side": "feed_forward", "side_norm": "norm"}
    optional_roles = ("shift", "ffn", "ffn_norm", "side", "side_norm")

    def __init__(self, spec, env, parts):
        super().__init__(spec, env)
        self.p = parts
        self.hidden = env.hidden_size
        if ("ffn" in parts) != ("ffn_norm" in parts) or ("side" in parts) != ("side_norm" in parts):
            raise ValueError("post-norm block: a feed-forward and a side input come with their norms")
        self.gated = [n for n in ("mixer_gate", "ffn_gate") if n in spec.tensors]
        if "ffn_gate" in self.gated and "ffn" not in parts:
            raise ValueError("post-norm block: a gate without a feed-forward")
        self.gate, self.gate_bias = {}, {}
        self.joined = False            # the feed-forward's gate and its router are one weight
        self.next_block, self.next_run = None, -1

    def tensor_specs(self):
        t = self.spec.tensors
        return [s for n in self.gated for s in (TensorSpec(t[n], (self.hidden, self.hidden)),
                                                TensorSpec(t[n + "_bias"], (self.hidden,), std=0.3))]

    def load(self, source):
        t = self.spec.tensors
        for n in self.gated:
            self.gate[n] = source.get(t[n])
            self.gate_bias[n] = source.get(t[n + "_bias"]).float().contiguous()
        ffn = self.p.get("ffn")
        if ffn is not None and getattr(ffn, "leaves_rows", False) and "ffn_gate" in self.gate:
            router = ffn.router_weight()
            if router.dtype == self.gate["ffn_gate"].dtype:
                self.gate["ffn_gate"] = torch.cat([self.gate["ffn_gate"], router], dim=0).contiguous()
                self.joined = True

    def weight_bytes(self):
        return sum(w.numel() * w.element_size() for w in self.gate.values())

    def flops(self, tokens, keys=0.0):
        return 2.0 * tokens * self.hidden * self.hidden * len(self.gated)

    def set_next_block(self, block, run: int) -> None:
        """The block that runs after this one in every step, as entry `run` of the run order (only when every layer
        runs once)."""
        self.next_run = run
        self.next_block = block if isinstance(block, GatedPostNormBlock) and hasattr(block.p.get("shift"), "ahead") else None

    def forward(self, x, pending, ctx, caches):
        if pending is not None:
            raise RuntimeError("post-norm block: the block before it left a branch that no norm adds")
        p, dt = self.p, self.env.dtype
        ahead = getattr(ctx, "shifted_ahead", None)
        if ahead is not None and ahead[0] is self:
            h, shifted = ahead[1], ahead[2]
        elif "shift" in p:
            shifted, h = p["shift"].forward(x, ctx, caches["shift"], plain=True)
        else:
            h = shifted = ops.cast(x, dt)
        ctx.shifted_ahead = None
        z = ops.linear_parts(h, self.gate["mixer_gate"], ctx.err) if "mixer_gate" in self.gate else None
        mixer = p["mixer"]
        y = mixer.forward(shifted, ctx, caches.get("mixer"), **(dict(leave_bias=True) if mixer.leaves_bias else {}))
        bias = mixer.output_bias if mixer.leaves_bias else None
        last = "mixer" if "ffn" not in p and "side" not in p else ("ffn" if "side" not in p else "side")
        h = self._add("mixer_norm", x, y, ctx, last == "mixer", gate=z, gate_bias=self.gate_bias.get("mixer_gate"), bias=bias)
        if "ffn" in p:
            ffn = p["ffn"]
            z = ops.linear_parts(h, self.gate["ffn_gate"], ctx.err) if "ffn_gate" in self.gate else None
            options = dict(leave_rows=True) if getattr(ffn, "leaves_rows", False) else {}
            if self.joined:
                options["logits"] = z[..., self.hidden:]
            y = ffn.forward(h, ctx, **options)
            h = self._add("ffn_norm", x, y, ctx, last == "ffn", gate=z, gate_bias=self.gate_bias.get("ffn_gate"))
        if "side" in p:
            self._add("side_norm", x, p["side"].forward(h, ctx), ctx, True)
        return x, None

    def _add(self, norm, x, y, ctx, closes, **options):
        """x += norm(gated y); the new stream in the compute dtype.  `closes`: it is the layer's last addition, whose
        cast only the next layer's shift would read: it is made with that shift where that is possible."""
        if isinstance(y, torch.Tensor):
            y = ops.cast(y, torch.float32)
        if not closes:
            return self.p[norm].add_normed(x, y, out_dtype=self.env.dtype, **options)
        nxt = self.next_block
        if nxt is None or ctx.max_q_len != 1:
            return self.p[norm].add_normed(x, y, **options)
        cache = ctx.cache.part_cache(self.next_run, "shift", ctx)
        h, shifted = self.p[norm].add_normed(x, y, out_dtype=self.env.dtype, next_shift=nxt.p["shift"].ahead(cache), ctx=ctx,
                                             **options)
        ctx.shifted_ahead = (nxt, h, shifted)
        return h
