"""Kagatar as a ModelSpec: a decoder whose mixer and feed-forward run side by side behind norms of their own, both on
the same stream.  A layer mixes with one of three grouped softmax attentions, all with biases on their projections:
values that are the keys, without positions, behind a window; all keys, rotated with YaRN frequencies, a gate on every
output element; or heads rotated, then normed without a weight, scores bounded by a tanh, behind a window.  The
feed-forward is a gated unit whose two branches are clamped.  A group of neighbouring layers may run several times in a
row with the same weights, every pass with caches of its own; each pass opens with a vector of its own added to the
stream, and every pass but the first with the embedding's output too.  The embedding is scaled where it enters, serves
as the head unscaled, and the logits are bounded by a tanh.

Tensor names: `embed`, `loop.step`, `final.norm`, and per layer i `l<i>.norm1|norm2`, `l<i>.mix.q|k|v` with `.b`,
`l<i>.mix.g`, `l<i>.mix.o`, `l<i>.mlp.gate|up|down`.
"""
from __future__ import annotations

from ..config.kagatar import CAPPED, GATED, TIED, KagatarConfig
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, RunStep

GLU_SLOPE, GLU_SHIFT = 1.702, 1.0        # the feed-forward: gate * sigmoid(slope * gate) * (up + shift)


def _rotary(encodings: dict, kind: str, m):
    if not m.rot_dims:
        return None
    s = m.rot_scaling
    scaling = None
    if s and kind == GATED:
        scaling = dict(type="yarn", **s.to_dict())
    elif s:
        scaling = dict(type="llama3", factor=s.factor, low_freq_factor=s.low, high_freq_factor=s.high,
                       original_max_position_embeddings=s.original)
    name = f"rotary_{m.rot_dims}_{m.rot_base!r}_{s!r}"
    encodings[name] = PartSpec("rotary", dict(rot_dim=m.rot_dims, theta=m.rot_base, layout="interleaved", scaling=scaling))
    return name


def build_kagatar_spec(cfg: KagatarConfig) -> ModelSpec:
    D, V, eps = cfg.width, cfg.vocab, cfg.norm_eps
    encodings, layers, unread = {}, [], []
    norm = lambda name: PartSpec("rmsnorm", dict(size=D, eps=eps), dict(weight=name))
    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        q = p + "mix."
        tensors = dict(q=q + "q", k=q + "k", o=q + "o", q_bias=q + "q.b", k_bias=q + "k.b")
        if l.type != TIED:
            tensors.update(v=q + "v", v_bias=q + "v.b")
        if l.type == GATED:
            tensors["g"] = q + "g"
        mixer = PartSpec("normed_gated_attention", dict(
            hidden_size=D, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.vdim, scale=m.scale,
            window=m.window, eps=eps, qk_norm="unit" if l.type == CAPPED else False, bias=True, output_bias=False,
            gate=l.type == GATED, tied_values=l.type == TIED, softcap=m.softcap,
            position_encoding=_rotary(encodings, l.type, m)), tensors)
        parts = {"mixer_norm": norm(p + "norm1"), "mixer": mixer}
        if l.mlp is not None:
            parts["ffn_norm"] = norm(p + "norm2")
            parts["ffn"] = PartSpec("swiglu", dict(
                hidden_size=D, intermediate_size=l.mlp.ff, activation="clamped", limit=l.mlp.limit, slope=GLU_SLOPE,
                shift=GLU_SHIFT), dict(gate=p + "mlp.gate", up=p + "mlp.up", down=p + "mlp.down"))
        else:
            unread.append(p + "norm2")
        opens = cfg.loop_times > 0 and i == cfg.loop_start
        layers.append(LayerSpec("parallel_two_norms", parts, dict(passes=cfg.loop_times) if opens else {},
                                dict(pass_steps="loop.step") if opens else {}))
    if not cfg.loop_times:
        unread.append("loop.step")
    return ModelSpec(
        hidden_size=D, vocab_size=V, max_position=cfg.max_position_embeddings,
        embedding=PartSpec("token_embedding", dict(vocab_size=V, hidden_size=D, scale=cfg.embed_scale), dict(weight="embed")),
        layers=layers, order=[RunStep(i, pass_index=t) for i, t in cfg.run_order()], final_norm=norm("final.norm"),
        lm_head=PartSpec("lm_head", dict(vocab_size=V, hidden_size=D, stored=False, softcap=cfg.logit_softcap),
                         dict(weight="embed")),
        position_encodings=encodings, eos_token_ids=cfg.eos_token_ids, ignored_tensors=tuple(unread))


register_architecture(KagatarConfig.ARCHITECTURE, KagatarConfig, build_kagatar_spec)
