"""Vatazen as a ModelSpec: a decoder whose sublayers read the stream as it is and whose results are gated element by
element and normed before they join it.  A layer mixes with latent attention (a window, a softmax with a sink per head,
YaRN positions on a rotated key part shared by all heads) or with differential attention in chunks (two maps per head
over the same values, queries and keys normed per head, no positions), behind a shift of its input towards the token
before; it feeds forward through experts without a gate, chosen by a router with a bias, and takes a learned input per
token and layer.  The embedding is scaled where it enters and serves as the head unscaled.

Tensor names: `embed`, `side.embed`, `final.norm`, and per layer i `l<i>.norm1|norm2`, `l<i>.shift`,
`l<i>.rg1|rg2` with `.b`, `l<i>.mix.*`, `l<i>.mlp.router` with `.b`, experts `l<i>.mlp.e<k>.up|down`, and
`l<i>.side.gate|proj|norm`.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.vatazen import VatazenConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, RunStep


def _rotary(encodings: dict, m):
    if not m.rot_dims:
        return None
    s = m.rot_scaling
    name = f"rotary_{m.rot_dims}_{m.rot_base!r}_{s!r}"
    encodings[name] = PartSpec("rotary", dict(rot_dim=m.rot_dims, theta=m.rot_base, layout="interleaved",
                                              scaling=dict(type="yarn", **s.to_dict()) if s else None))
    return name


def build_vatazen_spec(cfg: VatazenConfig) -> ModelSpec:
    D, V, eps, n = cfg.width, cfg.vocab, cfg.norm_eps, len(cfg.layers)
    encodings, layers, unread = {}, [], []
    norm = lambda name, offset=1.0: PartSpec("rmsnorm", dict(size=D, eps=eps, offset=offset), dict(weight=name))
    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        q = p + "mix."
        parts = {"shift": PartSpec("token_shift", dict(size=D), dict(weight=p + "shift")), "mixer_norm": norm(p + "norm1")}
        if l.type == "latent_attention":
            parts["mixer"] = PartSpec("latent_attention", dict(
                hidden_size=D, num_heads=m.heads, head_dim=m.dim, rot_dim=m.rot_dim, value_dim=m.vdim, kv_rank=m.kv_rank,
                scale=m.scale, window=m.mask_size, eps=eps, sink=True, exact_weights=True, position_encoding=_rotary(encodings, m)),
                dict(q=q + "q", dkv=q + "dkv", dkv_norm=q + "dkv.norm", uk=q + "uk", uv=q + "uv", sink=q + "sink", o=q + "o"))
        else:
            parts["mixer"] = PartSpec("differential_attention", dict(
                hidden_size=D, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.vdim,
                scale=m.scale, chunk=m.mask_size, eps=eps, diff=m.diff),
                dict(q=q + "q", k=q + "k", v=q + "v", o=q + "o", q_bias=q + "q.b", k_bias=q + "k.b", v_bias=q + "v.b",
                     o_bias=q + "o.b", q_norm=q + "q.norm", k_norm=q + "k.norm",
                     **{name: q + name for name in ("lq1", "lk1", "lq2", "lk2")}))
        gates = dict(mixer_gate=p + "rg1", mixer_gate_bias=p + "rg1.b")
        f = l.mlp
        if f is not None:
            parts["ffn"] = PartSpec("routed_moe", dict(
                hidden_size=D, num_experts=f.experts, top=f.top, intermediate_size=f.ff, activation="relu_squared",
                score="softmax_chosen"),
                dict(router=p + "mlp.router", router_bias=p + "mlp.router.b", up=p + "mlp.e{e}.up", down=p + "mlp.e{e}.down"))
            parts["ffn_norm"] = norm(p + "norm2")
            gates.update(ffn_gate=p + "rg2", ffn_gate_bias=p + "rg2.b")
        else:
            unread += [p + "norm2", p + "rg2", p + "rg2.b"]
        if cfg.side_dim:
            parts["side"] = PartSpec("token_side", dict(hidden_size=D, size=cfg.side_dim, vocab_size=V, layers=n, index=i),
                                     dict(table="side.embed", gate=p + "side.gate", proj=p + "side.proj"))
            parts["side_norm"] = norm(p + "side.norm", offset=0.0)
        layers.append(LayerSpec("gated_post_norm", parts, {}, gates))
    return ModelSpec(
        hidden_size=D, vocab_size=V, max_position=cfg.max_position_embeddings,
        embedding=PartSpec("token_embedding", dict(vocab_size=V, hidden_size=D, scale=cfg.embed_scale), dict(weight="embed")),
        layers=layers, order=[RunStep(i) for i in range(n)], final_norm=norm("final.norm"),
        lm_head=PartSpec("lm_head", dict(vocab_size=V, hidden_size=D, stored=False), dict(weight="embed")),
        position_encodings=encodings, eos_token_ids=cfg.eos_token_ids, ignored_tensors=tuple(unread))


register_architecture(VatazenConfig.ARCHITECTURE, VatazenConfig, build_vatazen_spec)
