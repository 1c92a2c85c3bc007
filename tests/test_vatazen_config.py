"""Vatazen without a GPU: config.json keys and their defaults, rejections that name the key, the tensors a model of a
configuration reads, random weights written and read back, what its layers ask of the cache, the stretched rotation
frequencies, and the plain implementation's own mechanisms against closed forms."""
import copy
import json
import math
import os

import numpy as np
import pytest
import torch

import ai_engine_b200 as aie
import plain_vatazen as pv
from ai_engine_b200.config import ConfigError, load_config
from ai_engine_b200.parts import KVRequest, StateRequest, rotary_inv_freq, rotary_magnitude
from ai_engine_b200.parts.model import Model, tensor_specs_of
from vatazen_helpers import CONFIGS, ids_for, make_dir, read_tensors, yarn


def test_every_key_is_read_and_written_back():
    for name, raw in CONFIGS.items():
        arch, cfg = load_config(raw)
        assert arch.name == "Vatazen"
        assert aie.VatazenConfig.from_dict(cfg.to_dict()) == cfg, name
    cfg = aie.VatazenConfig.from_dict(CONFIGS["A"])
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.embed_scale, cfg.side_dim) == (211, 96, 1e-4, 0.7, 12)
    a, l = cfg.layers[0], cfg.layers[1]
    assert (a.type, a.mixer.heads, a.mixer.kv_heads, a.mixer.dim, a.mixer.vdim, a.mixer.scale, a.mixer.diff, a.mixer.mask_size) \
        == ("attention", 6, 2, 12, 20, 0.3, 0.4, 50)
    assert (a.mlp.ff, a.mlp.experts, a.mlp.top) == (40, 6, 2)
    m = l.mixer
    assert (l.type, m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.scale, m.mask_size) == ("latent_attention", 5, 12, 8, 20, 24, 0.25, 37)
    assert (m.rot_dims, m.rot_base, m.rot_scaling.factor, m.rot_scaling.original, m.rot_scaling.fast, m.rot_scaling.slow) \
        == (8, 3000.0, 4.0, 64, 8.0, 0.5)


def test_absent_keys_mean_none():
    cfg = aie.VatazenConfig.from_dict(CONFIGS["C"])
    assert cfg.embed_scale == 1.0 and cfg.layers[3].mlp is None and cfg.layers[1].mixer.rot_scaling is None
    cfg = aie.VatazenConfig.from_dict(CONFIGS["D"])
    assert cfg.side_dim == 0 and all(l.mixer.mask_size == 0 for l in cfg.layers) and cfg.layers[0].mixer.rot_dims == 0
    raw = copy.deepcopy(CONFIGS["A"])
    del raw["layers"][0]["mixer"]["kv_heads"]    # as many key/value heads as query heads
    raw["layers"][0]["mixer"]["mask"] = None
    raw["layers"][1]["mixer"]["rot"]["scaling"] = None
    cfg = aie.VatazenConfig.from_dict(raw)
    assert cfg.layers[0].mixer.kv_heads == 6 and cfg.layers[0].mixer.mask_size == 0 and cfg.layers[1].mixer.rot_scaling is None


@pytest.mark.parametrize("edit,needle", [
    (lambda r: r.pop("vocab"), "vocab"),
    (lambda r: r["norm"].pop("eps"), "in norm: required key `eps`"),
    (lambda r: r.pop("norm"), "norm"),
    (lambda r: r["token_side"].__setitem__("dim", 0), "in token_side: `dim`"),
    (lambda r: r["layers"][0].__setitem__("type", "conv"), "conv"),
    (lambda r: r["layers"][0]["mixer"].__setitem__("kv_heads", 4), "in layers[0].mixer: heads = 6"),
    (lambda r: r["layers"][0]["mixer"].pop("diff"), "diff"),
    (lambda r: r["layers"][0]["mixer"]["mask"].__setitem__("size", 0), "in layers[0].mixer: in mask: `size`"),
    (lambda r: r["layers"][1]["mixer"]["rot"].__setitem__("dims", 7), "rot.dims"),
    (lambda r: r["layers"][1]["mixer"]["rot"].__setitem__("dims", 10), "rot.dims"),
    (lambda r: r["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "in rot.scaling: required key `slow`"),
    (lambda r: r["layers"][1]["mixer"]["rot"]["scaling"].__setitem__("factor", -1), "factor"),
    (lambda r: r["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda r: r["layers"][1]["mlp"]["router"].__setitem__("top", 6), "router.top"),
    (lambda r: r["layers"][1]["mlp"].__setitem__("kind", "dense"), "dense"),
    (lambda r: r["layers"][4]["mixer"].__setitem__("heads", "four"), "heads"),
])
def test_rejections_name_the_key(edit, needle):
    raw = copy.deepcopy(CONFIGS["A"])
    edit(raw)
    with pytest.raises(ConfigError) as e:
        aie.VatazenConfig.from_dict(raw)
    assert needle in str(e.value), str(e.value)


def test_tensors_of_a_configuration():
    arch, cfg = load_config(CONFIGS["A"])
    specs = {s.name: tuple(s.shape) for s in tensor_specs_of(arch.build_spec(cfg)) if s.stored}
    assert specs["embed"] == (211, 96) and specs["side.embed"] == (211, 60) and specs["final.norm"] == (96,)
    assert specs["l0.mix.q"] == (144, 96) and specs["l0.mix.k"] == (48, 96) and specs["l0.mix.v"] == (40, 96)
    assert specs["l0.mix.q.b"] == (144,) and specs["l0.mix.o"] == (96, 120) and specs["l0.mix.o.b"] == (96,)
    assert specs["l0.mix.q.norm"] == (12,) and specs["l0.mix.lk2"] == (12,) and specs["l0.rg1"] == (96, 96) and specs["l0.rg2.b"] == (96,)
    assert specs["l1.mix.q"] == (100, 96) and specs["l1.mix.dkv"] == (32, 96) and specs["l1.mix.dkv.norm"] == (24,)
    assert specs["l1.mix.uk"] == (60, 24) and specs["l1.mix.uv"] == (100, 24) and specs["l1.mix.sink"] == (5,)
    assert specs["l1.mlp.router.b"] == (5,) and specs["l1.mlp.e4.up"] == (24, 96) and specs["l1.mlp.e4.down"] == (96, 24)
    assert specs["l4.side.gate"] == (12, 96) and specs["l4.side.proj"] == (96, 12) and specs["l4.side.norm"] == (96,)
    assert specs["l2.shift"] == (96,) and "l2.rg1" in specs
    for gone in ("l2.rg2", "l2.norm2", "l2.mlp.router", "l0.mlp.e0.gate", "l1.mix.o.b"):
        assert gone not in specs, gone


def test_random_weights_are_written_and_read_back(tmp_path):
    d = make_dir(tmp_path, "D")
    with open(os.path.join(d, "config.json")) as f:
        raw = json.load(f)
    assert raw["architecture"] == "Vatazen" and len(raw["layers"]) == 3
    t = read_tensors(d)
    arch, cfg = load_config(d)
    assert set(t) == {s.name for s in tensor_specs_of(arch.build_spec(cfg)) if s.stored}
    logits, streams = pv.forward(CONFIGS["D"], t, ids_for(12, 97, 3))
    assert logits.shape == (12, 97) and streams.shape == (3, 12, 48) and bool(torch.isfinite(logits).all())


def test_what_the_layers_ask_of_the_cache():
    arch, cfg = load_config(CONFIGS["A"])
    m = Model(arch.build_spec(cfg), torch.float32, device="cpu")
    needs = m.cache_requests()
    assert [n.state for n in needs if n.role == "shift"] == [StateRequest((96,), torch.float32)] * 5
    kv = [n.kv for n in needs if n.role == "mixer"]
    assert kv == [KVRequest(2, 44, planes=1, chunk=50), KVRequest(1, 32, 37, planes=1), KVRequest(1, 44, 21, planes=1),
                  KVRequest(4, 56, planes=1, chunk=23), KVRequest(1, 36, 70, planes=1)]
    assert not m.pads_decode_rows()              # a repeated row would move the shift's state twice


# ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dims,base,scaling", [
    (16, 10000.0, yarn(8.0, 512)), (64, 500000.0, yarn(4.0, 4096, 32.0, 1.0)), (8, 100.0, yarn(16.0, 30, 64.0, 0.01)),
    (2, 50.0, yarn(3.0, 20, 4.0, 1.0)), (32, 10000.0, yarn(1.0, 100)), (12, 10000.0, yarn(40.0, 1000000, 2.0, 2.0)), (24, 300.0, None)])
def test_stretched_frequencies(dims, base, scaling):
    ref, mag = pv.yarn_frequencies(dims, base, scaling)
    sc = dict(type="yarn", **scaling) if scaling else None
    got = rotary_inv_freq(dims, base, sc)
    assert got.dtype == np.float32 and np.allclose(got, ref.numpy(), rtol=3e-7, atol=0)
    assert rotary_magnitude(sc) == pytest.approx(mag, rel=1e-12)


def test_frequencies_are_kept_divided_or_blended():
    dims, base, s = 32, 10000.0, yarn(8.0, 2048, 16.0, 1.0)
    f = rotary_inv_freq(dims, base, dict(type="yarn", **s)).astype(np.float64)
    plain = base ** (-2.0 * np.arange(16) / dims)
    turns = 2048 * plain / (2 * math.pi)         # of pair i within the original positions
    assert np.allclose(f[turns > 16.0 * 2], plain[turns > 16.0 * 2]) and (turns > 32).any()
    assert np.allclose(f[turns < 0.5], plain[turns < 0.5] / 8.0) and (turns < 0.5).any()
    mid = (turns < 10) & (turns > 1.5)
    assert mid.any() and ((f < plain) & (f > plain / 8.0))[mid].all()
    assert rotary_magnitude(dict(type="yarn", **s)) == pytest.approx(1.0 + 0.1 * math.log(8.0))
    assert rotary_magnitude(dict(type="linear", factor=8.0)) == 1.0 and rotary_magnitude(None) == 1.0


def test_mixers_that_rotate_without_a_magnitude_refuse_a_stretched_encoding():
    from ai_engine_b200.parts import BuildEnv, GQAAttention, NormedGatedAttention, PartSpec, RotaryEncoding
    e = BuildEnv(32, torch.float32, torch.device("cpu"))
    for layout, cls, more in (("halves", GQAAttention, {}), ("interleaved", NormedGatedAttention, dict(value_dim=8, eps=1e-5))):
        e.position_encodings["r"] = RotaryEncoding(PartSpec("rotary", dict(
            rot_dim=8, theta=100.0, layout=layout, scaling=dict(type="yarn", **yarn(2.0, 64)))), e)
        with pytest.raises(ValueError, match="magnitude"):
            cls(PartSpec("m", dict(hidden_size=32, num_heads=2, num_kv_heads=1, head_dim=8, position_encoding="r", **more)), e)


def test_plain_shift_and_side_input():
    x = torch.arange(12, dtype=torch.float64).view(4, 3)
    s = torch.tensor([0.0, 1.0, 0.25], dtype=torch.float64)
    y = pv.token_shift(x, s)
    assert torch.equal(y[:, 0], x[:, 0]) and torch.equal(y[1:, 1], x[:-1, 1]) and float(y[0, 1]) == 0.0
    assert torch.allclose(y[1:, 2], x[1:, 2] - 0.25 * 3) and float(y[0, 2]) == 0.75 * 2
    W = {"side.embed": torch.tensor([[1.0, 2.0, 3.0, 4.0]], dtype=torch.float64), "side.gate": torch.eye(2, 3, dtype=torch.float64) * 100,
         "side.proj": torch.ones(3, 2, dtype=torch.float64), "side.norm": torch.tensor([1.0, 2.0, -1.0], dtype=torch.float64)}
    # gelu of a large positive number is that number: g = 100 x[:2] * e; the projection sums it into every column alike
    out = pv.token_side(x[1:2], W, "", [0], 1, 2, 0.0)
    assert torch.allclose(out, torch.tensor([[1.0, 2.0, -1.0]], dtype=torch.float64))


def test_plain_masks_sink_and_difference():
    """All scores zero: every visible key weighs alike, the sink takes exp(sink) of the denominator, and two equal maps
    leave (1 - lambda) times one of them, whose size the norm takes away."""
    torch.manual_seed(0)
    D, T = 8, 12
    eye = torch.eye(4, D, dtype=torch.float64)
    h = torch.randn(T, D, dtype=torch.float64)
    W = {"q": torch.zeros(6, D, dtype=torch.float64), "dkv": torch.cat([eye, torch.zeros(2, D, dtype=torch.float64)]),
         "dkv.norm": torch.ones(4, dtype=torch.float64), "uk": torch.zeros(4, 4, dtype=torch.float64),
         "uv": torch.eye(4, dtype=torch.float64), "sink": torch.tensor([math.log(2.0)], dtype=torch.float64),
         "o": torch.eye(D, 4, dtype=torch.float64)}
    m = dict(heads=1, dim=4, rot_dim=2, vdim=4, kv_rank=4, scale=1.0, mask=dict(size=3), rot=dict(base=10.0, dims=2))
    out = pv.latent_attention(h, W, "", m, 1e-9)
    c = pv.rms(h[:, :4], 1.0, 1e-9)
    for i in range(T):
        seen = list(range(max(0, i - 2), i + 1))
        assert torch.allclose(out[i, :4], c[seen].sum(0) / (2.0 + len(seen)))
    zeros = lambda *s: torch.zeros(*s, dtype=torch.float64)
    W = {"q": zeros(4, D), "k": zeros(4, D), "v": eye, "q.b": zeros(4), "k.b": zeros(4), "v.b": zeros(4), "o": torch.eye(D, 4, dtype=torch.float64),
         "o.b": zeros(D) + 0.5, "q.norm": zeros(2) + 1, "k.norm": zeros(2) + 1, "lq1": zeros(2), "lk1": zeros(2), "lq2": zeros(2), "lk2": zeros(2)}
    m = dict(heads=1, kv_heads=1, dim=2, vdim=4, scale=1.0, diff=0.3, mask=dict(size=5))
    out = pv.differential_attention(h, W, "", m, 1e-12)
    assert pv.differential_lambda(W, "", m) == pytest.approx(0.3)
    for i in range(T):
        a = h[i // 5 * 5:i + 1, :4].mean(0)
        assert torch.allclose(out[i, :4], pv.rms(a, 1.0, 1e-12) * 0.7 + 0.5) and torch.allclose(out[i, 4:], zeros(4) + 0.5)


def test_plain_router_weighs_the_chosen_only():
    z = torch.tensor([[1.0, 5.0, 3.0, 2.0]], dtype=torch.float64)
    W = {"router": torch.eye(4, dtype=torch.float64), "router.b": torch.tensor([4.5, 0.0, 0.0, 0.0], dtype=torch.float64)}
    ids, w = pv.route(z, W, "", dict(experts=4, top=2))
    assert ids[0].tolist() == [0, 1]             # 5.5 and 5.0: the bias enters the choice
    e = math.exp(-0.5)
    assert torch.allclose(w, torch.tensor([[1 / (1 + e), e / (1 + e)]], dtype=torch.float64))
