"""Kagatar without a GPU: config.json keys and their defaults, rejections that name the key, the run order of its passes,
the tensors a model of a configuration reads, random weights written and read back, what its layers ask of the cache, its
rotation frequencies, what the shared parts refuse, and the plain implementation's own mechanisms against closed forms."""
import copy
import json
import math
import os

import numpy as np
import pytest
import torch

import ai_engine_b200 as aie
import plain_kagatar as pk
from ai_engine_b200.config import ConfigError, load_config
from ai_engine_b200.parts import KVRequest, PartSpec, rotary_inv_freq, rotary_magnitude
from ai_engine_b200.parts.model import Model, tensor_specs_of
from kagatar_helpers import CONFIGS, ids_for, make_dir, read_tensors, waves, yarn


def test_every_key_is_read_and_written_back():
    for name, raw in CONFIGS.items():
        arch, cfg = load_config(raw)
        assert arch.name == "Kagatar"
        assert aie.KagatarConfig.from_dict(cfg.to_dict()) == cfg, name
    cfg = aie.KagatarConfig.from_dict(CONFIGS["A"])
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.embed_scale, cfg.logit_softcap) == (211, 96, 1e-4, 2.0, 9.0)
    assert (cfg.loop_start, cfg.loop_stop, cfg.loop_times) == (1, 3, 3)
    c, g, t = cfg.layers[0], cfg.layers[1], cfg.layers[2]
    m = c.mixer
    assert (c.type, m.heads, m.kv_heads, m.dim, m.vdim, m.scale, m.window, m.softcap) == ("attention_3", 6, 2, 20, 12, 0.35, 37, 6.0)
    s = m.rot_scaling
    assert (m.rot_dims, m.rot_base, s.factor, s.low, s.high, s.original) == (12, 3000.0, 4.0, 1.0, 4.0, 60)
    assert (c.mlp.ff, c.mlp.limit) == (80, 0.4)
    m, s = g.mixer, g.mixer.rot_scaling
    assert (g.type, m.dim, m.vdim, m.window, m.softcap) == ("attention_2", 12, 28, 0, 0.0)
    assert (m.rot_dims, m.rot_base, s.factor, s.original, s.fast, s.slow) == (6, 700.0, 8.0, 40, 8.0, 0.5)
    assert (t.type, t.mixer.dim, t.mixer.vdim, t.mixer.window, t.mixer.rot_dims, t.mlp) == ("attention", 36, 36, 21, 0, None)


def test_absent_keys_mean_none():
    cfg = aie.KagatarConfig.from_dict(CONFIGS["C"])
    assert cfg.embed_scale == 1.0 and cfg.logit_softcap == 0.0 and cfg.loop_times == 0
    assert cfg.layers[0].mlp.limit == math.inf and cfg.layers[1].mixer.rot_scaling is None
    assert cfg.layers[3].mixer.rot_dims == 0 and cfg.layers[3].mixer.softcap == 0.0 and cfg.layers[4].mlp is None
    raw = copy.deepcopy(CONFIGS["A"])
    for k in ("kv_heads", "vdim"):               # as many key/value heads as heads, values of the keys' size
        del raw["layers"][0]["mixer"][k]
    raw["layers"][0]["mixer"]["mask"] = None
    raw["layers"][2]["mixer"]["rot"] = dict(base=10.0, dims=4)        # nothing rotates where the values are the keys
    raw["loop"] = None
    cfg = aie.KagatarConfig.from_dict(raw)
    m = cfg.layers[0].mixer
    assert (m.kv_heads, m.vdim, m.window, cfg.layers[2].mixer.rot_dims, cfg.loop_times) == (6, 20, 0, 0, 0)


def test_the_passes_of_the_run_order():
    cfg = aie.KagatarConfig.from_dict(CONFIGS["A"])
    assert cfg.run_order() == [(0, 0), (1, 0), (2, 0), (1, 1), (2, 1), (1, 2), (2, 2), (3, 0)]
    assert [i for i, _ in pk.run_order(CONFIGS["A"])] == [i for i, _ in cfg.run_order()]
    assert [t for _, t in pk.run_order(CONFIGS["A"])] == [None, 0, None, 1, None, 2, None, None]
    arch, cfg = load_config(CONFIGS["A"])
    spec = arch.build_spec(cfg)
    assert [(s.layer, s.pass_index) for s in spec.order] == cfg.run_order()
    m = Model(spec, torch.float32, device="cpu")
    assert [l.block.needs_embedding_output for l in m.layers] == [False, True, False, False] and m.keeps_embedding_output
    arch, cfg = load_config(CONFIGS["D"])        # one pass: the embedding's output never joins again
    assert not Model(arch.build_spec(cfg), torch.float32, device="cpu").keeps_embedding_output


@pytest.mark.parametrize("edit,needle", [
    (lambda r: r.pop("vocab"), "vocab"),
    (lambda r: r["norm"].pop("eps"), "in norm: required key `eps`"),
    (lambda r: r.pop("norm"), "norm"),
    (lambda r: r.__setitem__("layers", []), "layers"),
    (lambda r: r.__setitem__("logit_softcap", -1.0), "logit_softcap"),
    (lambda r: r["loop"].__setitem__("stop", 1), "loop.start = 1"),
    (lambda r: r["loop"].__setitem__("stop", 5), "loop.stop = 5"),
    (lambda r: r["loop"].__setitem__("times", 0), "in loop: `times`"),
    (lambda r: r["loop"].pop("start"), "in loop: required key `start`"),
    (lambda r: r["layers"][0].__setitem__("type", "attention_4"), "attention_4"),
    (lambda r: r["layers"][0].pop("mixer"), "mixer"),
    (lambda r: r["layers"][0]["mixer"].__setitem__("kv_heads", 4), "in layers[0].mixer: heads = 6"),
    (lambda r: r["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda r: r["layers"][0]["mixer"].__setitem__("softcap", -2), "softcap"),
    (lambda r: r["layers"][0]["mixer"]["mask"].__setitem__("size", 0), "in layers[0].mixer: in mask: `size`"),
    (lambda r: r["layers"][0]["mixer"]["rot"].__setitem__("dims", 7), "rot.dims"),
    (lambda r: r["layers"][0]["mixer"]["rot"].__setitem__("dims", 22), "rot.dims"),
    (lambda r: r["layers"][0]["mixer"]["rot"]["scaling"].__setitem__("high", 0.5), "in rot.scaling: high = 0.5"),
    (lambda r: r["layers"][0]["mixer"]["rot"]["scaling"].pop("low"), "in rot.scaling: required key `low`"),
    (lambda r: r["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "in rot.scaling: required key `slow`"),
    (lambda r: r["layers"][1]["mixer"]["rot"]["scaling"].__setitem__("factor", 0), "factor"),
    (lambda r: r["layers"][2]["mixer"].__setitem__("vdim", 20), "vdim = 20"),
    (lambda r: r["layers"][3]["mlp"].__setitem__("kind", "moe"), "moe"),
    (lambda r: r["layers"][3]["mlp"].__setitem__("limit", 0), "in layers[3].mlp: `limit`"),
    (lambda r: r["layers"][3]["mlp"].pop("ff"), "ff"),
])
def test_rejections_name_the_key(edit, needle):
    raw = copy.deepcopy(CONFIGS["A"])
    edit(raw)
    with pytest.raises(ConfigError) as e:
        aie.KagatarConfig.from_dict(raw)
    assert needle in str(e.value), str(e.value)


def test_tensors_of_a_configuration():
    arch, cfg = load_config(CONFIGS["A"])
    specs = {s.name: tuple(s.shape) for s in tensor_specs_of(arch.build_spec(cfg)) if s.stored}
    assert specs["embed"] == (211, 96) and specs["loop.step"] == (3, 96) and specs["final.norm"] == (96,)
    assert specs["l0.mix.q"] == (120, 96) and specs["l0.mix.k"] == (40, 96) and specs["l0.mix.v"] == (24, 96)
    assert specs["l0.mix.q.b"] == (120,) and specs["l0.mix.k.b"] == (40,) and specs["l0.mix.v.b"] == (24,)
    assert specs["l0.mix.o"] == (96, 72) and specs["l0.norm1"] == (96,) and specs["l0.norm2"] == (96,)
    assert specs["l1.mix.g"] == (140, 96) and specs["l1.mix.o"] == (96, 140) and specs["l1.mix.v"] == (28, 96)
    assert specs["l2.mix.q"] == (144, 96) and specs["l2.mix.k"] == (72, 96) and specs["l2.mix.o"] == (96, 144)
    assert specs["l3.mlp.gate"] == specs["l3.mlp.up"] == (72, 96) and specs["l3.mlp.down"] == (96, 72)
    for gone in ("head", "l0.mix.g", "l0.mix.o.b", "l2.mix.v", "l2.mix.v.b", "l2.mix.g", "l2.norm2", "l2.mlp.gate", "l3.mix.g"):
        assert gone not in specs, gone
    arch, cfg = load_config(CONFIGS["C"])
    assert "loop.step" not in {s.name for s in tensor_specs_of(arch.build_spec(cfg))}


def test_random_weights_are_written_and_read_back(tmp_path):
    d = make_dir(tmp_path, "D")
    with open(os.path.join(d, "config.json")) as f:
        raw = json.load(f)
    assert raw["architecture"] == "Kagatar" and len(raw["layers"]) == 3
    t = read_tensors(d)
    arch, cfg = load_config(d)
    assert set(t) == {s.name for s in tensor_specs_of(arch.build_spec(cfg)) if s.stored}
    streams = []
    logits = pk.forward(t, CONFIGS["D"], ids_for(12, 97, 3), streams=streams)
    assert logits.shape == (12, 97) and len(streams) == 3 and bool(torch.isfinite(logits).all())
    assert float(logits.abs().max()) < 4.0       # the bound on the logits


def test_what_the_layers_ask_of_the_cache():
    arch, cfg = load_config(CONFIGS["A"])
    m = Model(arch.build_spec(cfg), torch.float32, device="cpu")
    needs = m.cache_requests()
    assert all(n.role == "mixer" and n.state is None and n.cache_from is None for n in needs)
    c0, g, t, c1 = (KVRequest(2, 32, 37, planes=1), KVRequest(1, 40, planes=1), KVRequest(2, 36, 21, planes=1),
                    KVRequest(3, 52, 50, planes=1))
    assert [n.kv for n in needs] == [c0, g, t, g, t, g, t, c1]        # every pass has pages of its own
    assert m.pads_decode_rows() and not m.has_host_parts()


@pytest.mark.parametrize("dims,base,scaling", [
    (16, 10000.0, yarn(8.0, 512)), (64, 500000.0, yarn(4.0, 4096)), (8, 100.0, yarn(16.0, 30, 64.0, 0.01)),
    (2, 50.0, yarn(3.0, 20, 4.0, 1.0)), (12, 10000.0, yarn(40.0, 1000000, 2.0, 2.0)),
    (16, 10000.0, waves(8.0, 64)), (48, 500000.0, waves(32.0, 8192)), (8, 100.0, waves(2.0, 100, 0.5, 20.0)),
    (20, 300.0, waves(1.0, 50)), (6, 1e6, waves(4.0, 10, 3.0, 3.5))])
def test_rotation_frequencies(dims, base, scaling):
    if "fast" in scaling:
        ref, kind = pk.yarn_frequencies(dims, base, scaling), dict(type="yarn", **scaling)
        assert abs(rotary_magnitude(kind) - pk.yarn_magnitude(scaling)) < 1e-12
    else:
        ref = pk.wavelength_frequencies(dims, base, scaling)
        kind = dict(type="llama3", factor=scaling["factor"], low_freq_factor=scaling["low"],
                    high_freq_factor=scaling["high"], original_max_position_embeddings=scaling["original"])
        assert rotary_magnitude(kind) == 1.0
    got = rotary_inv_freq(dims, base, kind).astype(np.float64)
    assert np.abs(got - np.array(ref)).max() <= 2e-7 * max(ref) and np.abs(got / np.array(ref) - 1).max() < 1e-5


def _attention_spec(**over):
    p = dict(hidden_size=16, num_heads=2, num_kv_heads=1, head_dim=8, value_dim=8, scale=0.3, eps=1e-5, qk_norm=False,
             output_bias=False, gate=False)
    p.update(over)
    return PartSpec("normed_gated_attention", p, {n: n for n in ("q", "k", "v", "o", "q_bias", "k_bias", "v_bias", "g", "q_norm", "k_norm")})


@pytest.mark.parametrize("over,needle", [
    (dict(tied_values=True, value_dim=4), "tied"), (dict(tied_values=True, qk_norm="unit"), "tied"),
    (dict(qk_norm="rms"), "qk_norm"), (dict(softcap=-1.0), "softcap"), (dict(qk_norm="unit", value_mix="mix"), "unit"),
    (dict(position_encoding="yarn", qk_norm=True), "magnitude"), (dict(position_encoding="halves", qk_norm="unit"), "unit"),
    (dict(position_encoding="halves", tied_values=True), "tied")])
def test_what_the_attention_refuses(over, needle):
    from ai_engine_b200.parts import BuildEnv, NormedGatedAttention, RotaryEncoding
    e = BuildEnv(16, torch.float32, torch.device("cpu"))
    e.position_encodings["yarn"] = RotaryEncoding(PartSpec("rotary", dict(
        rot_dim=4, theta=100.0, layout="interleaved", scaling=dict(type="yarn", **yarn(4.0, 100)))), e)
    e.position_encodings["halves"] = RotaryEncoding(PartSpec("rotary", dict(rot_dim=4, theta=100.0)), e)
    NormedGatedAttention(_attention_spec(), e)
    with pytest.raises(ValueError) as err:
        NormedGatedAttention(_attention_spec(**over), e)
    assert needle in str(err.value)


def test_what_the_block_and_the_unit_refuse():
    from ai_engine_b200.parts import BuildEnv, DynamicTanh, NormedGatedAttention, RMSNorm, SwiGLU, TwoNormParallelBlock
    e = BuildEnv(16, torch.float32, torch.device("cpu"))
    norm = lambda eps: RMSNorm(PartSpec("rmsnorm", dict(size=16, eps=eps), dict(weight="w")), e)
    mixer = NormedGatedAttention(_attention_spec(), e)
    ffn = SwiGLU(PartSpec("swiglu", dict(hidden_size=16, intermediate_size=8), dict(gate="g", up="u", down="d")), e)
    make = lambda **p: TwoNormParallelBlock(PartSpec("parallel_two_norms"), e, p)
    make(mixer_norm=norm(1e-5), mixer=mixer, ffn_norm=norm(1e-5), ffn=ffn)
    make(mixer_norm=norm(1e-5), mixer=mixer)
    for bad in (dict(mixer_norm=norm(1e-5), mixer=mixer, ffn_norm=norm(1e-6), ffn=ffn),       # one root mean square a row
                dict(mixer_norm=norm(1e-5), mixer=mixer, ffn=ffn),
                dict(mixer_norm=DynamicTanh(PartSpec("dynamic_tanh", dict(size=16)), e), mixer=mixer)):
        with pytest.raises(ValueError):
            make(**bad)
    with pytest.raises(ValueError):
        SwiGLU(PartSpec("swiglu", dict(hidden_size=16, intermediate_size=8, activation="clamped", limit=0.0)), e)


# ---------------------------------------------------------------------------------------------------
def test_the_oracles_rotation_keeps_lengths_and_depends_on_the_distance():
    gen = torch.Generator().manual_seed(3)
    x = torch.randn(1, 2, 10, generator=gen, dtype=torch.float64)
    f = [0.7, 0.02, 1.3]
    y = pk.rotate_neighbours(x, [5], f)
    assert torch.allclose(y.norm(dim=-1), x.norm(dim=-1)) and torch.equal(y[..., 6:], x[..., 6:])
    assert abs(float(y[0, 0, 0]) - float(x[0, 0, 0] * math.cos(3.5) - x[0, 0, 1] * math.sin(3.5))) < 1e-12
    a, b = x[:, :1], x[:, 1:]
    dot = lambda p, q: float((pk.rotate_neighbours(a, [p], f) * pk.rotate_neighbours(b, [q], f)).sum())
    assert abs(dot(9, 4) - dot(105, 100)) < 1e-9 and abs(dot(9, 4) - dot(9, 5)) > 1e-3
    assert torch.allclose(pk.rotate_neighbours(x, [5], f, 1.5)[..., :6], 1.5 * y[..., :6])      # the rest is not scaled
    assert torch.equal(pk.rotate_neighbours(x, [5], f, 1.5)[..., 6:], x[..., 6:])


def test_the_oracles_window_cap_and_clamp_in_closed_form():
    T, w = 9, 4
    zeros, v = torch.zeros(T, 1, 2, dtype=torch.float64), torch.arange(T, dtype=torch.float64).view(T, 1, 1)
    o = pk.softmax_over_sight(zeros, zeros, v, 1.0, w)[:, 0, 0]                  # equal scores: the mean of what is seen
    assert [float(x) for x in o] == [sum(range(max(0, i - 3), i + 1)) / min(i + 1, 4) for i in range(T)]
    q, k = torch.full((2, 1, 1), 100.0, dtype=torch.float64), torch.tensor([1.0, -1.0], dtype=torch.float64).view(2, 1, 1)
    p = pk.softmax_over_sight(q, k, torch.tensor([1.0, 0.0], dtype=torch.float64).view(2, 1, 1), 1.0, 0, 2.0)[1, 0, 0]
    assert abs(float(p) - 1 / (1 + math.exp(-4.0))) < 1e-12                      # both scores at the bound: 2 and -2
    one = torch.ones(1, 1, dtype=torch.float64)
    ff = lambda g, u, lim: float(pk.clamped_ff(one, g * one, u * one, one, lim))
    glu = lambda g, u: g / (1 + math.exp(-1.702 * g)) * (u + 1)
    for g, u, lim, g2, u2 in ((5.0, 9.0, 2.0, 2.0, 2.0), (-5.0, -9.0, 2.0, -5.0, -2.0), (1.0, -1.0, 2.0, 1.0, -1.0)):
        assert abs(ff(g, u, lim) - glu(g2, u2)) < 1e-12


def test_the_oracle_does_not_depend_on_later_tokens(tmp_path):
    d = make_dir(tmp_path, "A")
    t, ids = read_tensors(d), ids_for(60, 211, 5)
    a = pk.forward(t, CONFIGS["A"], ids)
    b = pk.forward(t, CONFIGS["A"], ids[:31])
    assert float((a[:31] - b).abs().max()) < 1e-10
