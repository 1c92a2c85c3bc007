"""Each mechanism of the Kagatar design alone, on a real cache and step context, against the plain implementation: the
pair of norms with what joins the stream ahead of them, the clamped gated unit, products whose parts join the stream
together, the prepare kernel (rotation with a magnitude, unit heads, tied values), and the three attentions (three
requests in unequal portions on pages used again; keys planted just inside and just outside the window, at a page's edges
and far back, as one prompt, decoded token by token and in portions of two; scores at their bound; the gate)."""
import pytest
import torch

import plain_kagatar as pk
from kagatar_helpers import DEV, Rig, capped, env, gated, load, rot, tied, waves, yarn
from test_fokisun_parts_gpu import DT, f64, near, rnd

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


# ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,T", [(36, 5), (97, 3), (128, 1), (512, 300), (1024, 64), (2048, 257), (4608, 7), (4608, 256), (6, 2)])
def test_two_norms_of_one_stream_and_what_joins_it_ahead(dtype, D, T):
    from ai_engine_b200.parts import PartSpec, RMSNorm
    gen = torch.Generator().manual_seed(D + T)
    e, eps = env(DT[dtype], D), 3e-2
    w = {n: rnd(gen, D, std=0.4, mean=1.0) for n in ("a", "b")}
    a, b = (load(RMSNorm(PartSpec("rmsnorm", dict(size=D, eps=eps), dict(weight=n)), e), {n: w[n]}, DT[dtype]) for n in ("a", "b"))
    assert a.pairs_with(b) and a.pairs_with(None)
    x, parts, extra, step = rnd(gen, T, D), rnd(gen, 7, T, D, std=0.3), rnd(gen, T, D), rnd(gen, D)
    for delta, ex, st, two in ((None, None, None, True), (parts, None, None, True), (parts[0], extra, step, True),
                               (parts[:5].contiguous(), None, step, False), (None, extra, step, True), (parts, extra, None, False)):
        s = x.double()
        for more in (None if delta is None else delta.sum(0) if delta.dim() == 3 else delta, ex, st):
            s = s if more is None else s + more.double()
        xd = x.to(DEV)
        put = lambda t: None if t is None else t.to(DEV)
        h1, h2 = a.forward_pair(b if two else None, xd, put(delta), put(ex), put(st))
        assert float((xd.cpu().double() - s).abs().max()) < 1e-5
        near(h1.cpu(), pk.rms(s, eps) * w["a"].double(), dtype, "first norm")
        assert h1.dtype == DT[dtype] and (h2 is None) == (not two)
        if two:
            near(h2.cpu(), pk.rms(s, eps) * w["b"].double(), dtype, "second norm")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,F,T,limit", [(64, 128, 5, 0.8), (128, 64, 64, 1.5), (128, 192, 70, 0.4), (40, 24, 9, 2.0),
                                         (36, 33, 130, 0.7), (64, 320, 17, None), (64, 40, 1, 0.3)])
def test_clamped_gated_unit(dtype, D, F, T, limit):
    from ai_engine_b200.parts import PartSpec, SwiGLU
    gen = torch.Generator().manual_seed(D * F)
    t = {n: rnd(gen, *s, std=0.25) for n, s in (("gate", (F, D)), ("up", (F, D)), ("down", (D, F)))}
    p = dict(hidden_size=D, intermediate_size=F, activation="clamped", slope=1.702, shift=1.0)
    if limit is not None:
        p["limit"] = limit
    part = load(SwiGLU(PartSpec("swiglu", p, dict(gate="gate", up="up", down="down")), env(DT[dtype], D)), t, DT[dtype])
    h = rnd(gen, T, D)
    ctx = type("C", (), {"err": torch.zeros(1, dtype=torch.int32, device=DEV)})()
    got = part.forward(h.to(DEV).to(DT[dtype]), ctx).double()
    got = (got.sum(0) if got.dim() == 3 else got).cpu()
    lim = limit if limit is not None else 1e30
    ref = pk.clamped_ff(h.double(), *(t[n].double() for n in ("gate", "up", "down")), lim)
    near(got, ref, dtype, "clamped unit")
    if limit is not None:        # the clamps bind on both sides, and the test tells a clamp left out
        g, u = h @ t["gate"].T, h @ t["up"].T
        assert bool((g > limit).any() and (u > limit).any() and (u < -limit).any())
        assert float((pk.clamped_ff(h.double(), *(t[n].double() for n in ("gate", "up", "down")), 1e30) - ref).abs().max()) > 0.3 * float(ref.std())
    a, w = part.forward(h.to(DEV).to(DT[dtype]), ctx, leave_projection=True)       # what it leaves is what it multiplies
    near((a.double() @ w.double().T).cpu(), ref, dtype, "clamped unit, the last product left")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("N,K1,K2,T", [(96, 64, 200, 3), (128, 1024, 40, 64), (2048, 2048, 6144, 8), (36, 20, 24, 7), (40, 13, 64, 5)])
def test_two_products_that_join_the_stream_together(dtype, N, K1, K2, T):
    from ai_engine_b200.kernels import ops
    gen = torch.Generator().manual_seed(N + T)
    x1, w1, x2, w2 = rnd(gen, T, K1), rnd(gen, N, K1, std=0.1), rnd(gen, T, K2), rnd(gen, N, K2, std=0.1)
    put = lambda t: t.to(DEV).to(DT[dtype])
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    y = ops.linear_parts_together([(put(x1), put(w1)), (put(x2), put(w2))], err)
    assert y.dtype == torch.float32 and y.shape[-2:] == (T, N)
    got = (y.double().sum(0) if y.dim() == 3 else y.double()).cpu()
    ref = x1.double() @ w1.double().T + x2.double() @ w2.double().T
    assert float((got - ref).abs().max()) < 1e-4 * float(ref.abs().max()) and int(err.item()) == 0


# ---------------------------------------------------------------------------------------------------
def attention_part(l, hidden, eps, dtype, gen, tie_keys=False):
    """The framework's attention part for a layer entry, with random weights; tie_keys: k reads the second half of the
    input as q reads the first, so q_i . k_j is large where h_j is h_i moved by half the width."""
    from ai_engine_b200.models.kagatar import _rotary
    from ai_engine_b200.config.kagatar import CAPPED, GATED, TIED, KagatarMixer
    from ai_engine_b200.parts import NormedGatedAttention, PartSpec, RotaryEncoding
    kind, m = l["type"], KagatarMixer.from_dict(l["type"], l["mixer"])
    H, G, d, e = m.heads, m.kv_heads, m.dim, m.vdim
    t = {"q": rnd(gen, H * d, hidden, std=0.25), "k": rnd(gen, G * d, hidden, std=0.25), "q.b": rnd(gen, H * d, std=0.3),
         "k.b": rnd(gen, G * d, std=0.3), "o": rnd(gen, hidden, H * e, std=0.2)}
    if kind != TIED:
        t.update({"v": rnd(gen, G * e, hidden, std=0.25), "v.b": rnd(gen, G * e, std=0.3)})
    if kind == GATED:
        t["g"] = rnd(gen, H * e, hidden, std=0.4)
    if tie_keys:
        t["k"] = torch.roll(t["q"][:G * d], hidden // 2, dims=1).contiguous()
        t["q.b"].zero_()
        t["k.b"].zero_()
    e_, encodings = env(DT[dtype], hidden), {}
    pe = _rotary(encodings, kind, m)
    for name, spec in encodings.items():
        e_.position_encodings[name] = RotaryEncoding(spec, e_)
        e_.position_encodings[name].load(None)
    spec = PartSpec("normed_gated_attention", dict(
        hidden_size=hidden, num_heads=H, num_kv_heads=G, head_dim=d, value_dim=e, scale=m.scale, window=m.window, eps=eps,
        qk_norm="unit" if kind == CAPPED else False, output_bias=False, gate=kind == GATED, tied_values=kind == TIED,
        softcap=m.softcap, position_encoding=pe), {n.replace(".b", "_bias"): n for n in t})
    return load(NormedGatedAttention(spec, e_), t, DT[dtype]), t


def plain(l, t, h, eps):
    return pk.MIXERS[l["type"]](h.double(), f64(t), l["mixer"], eps, range(h.shape[0]))


SHAPES = [          # the plain kernels, the tensor-core kernels at their own sizes, and at sizes that are filled up
    (tied(4, 2, 64, 0.09, 100), 96), (tied(6, 2, 40, 0.12, 37), 64), (tied(1, 1, 12, 0.3, 2), 36), (tied(8, 1, 128, 0.05), 128),
    (tied(9, 1, 32, 0.15, 130), 64), (tied(2, 2, 96, 0.06, 64), 80),
    (gated(4, 1, 64, 128, 0.1, rot(50000.0, 32, yarn(8.0, 64))), 96), (gated(5, 5, 12, 28, 0.3, rot(500.0, 6, yarn(4.0, 40, 8.0, 0.5))), 40),
    (gated(4, 2, 128, 64, 0.07, rot(1e4, 128, yarn(2.0, 300)), 130), 64), (gated(6, 3, 72, 24, 0.1, rot(300.0, 2)), 48),
    (gated(3, 1, 20, 30, 0.2), 36), (gated(16, 1, 32, 32, 0.2, rot(1e5, 30, yarn(16.0, 128))), 64),
    (capped(6, 2, 64, 40, 0.2, rot(30000.0, 48, waves(8.0, 60)), 100, 8.0), 96), (capped(4, 4, 10, 6, 0.5, rot(500.0, 10, waves(4.0, 100)), 37, 3.0), 40),
    (capped(4, 1, 128, 128, 0.1, rot(1e6, 128, waves(32.0, 256)), 1, 30.0), 64), (capped(2, 1, 144, 20, 0.1, rot(100.0, 6), 90, 20.0), 48),
    (capped(3, 3, 36, 44, 0.3, None, 64), 36), (capped(8, 2, 24, 104, 0.4, rot(2000.0, 24, waves(2.0, 30, 0.5, 9.0)), None, 50.0), 64),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", range(len(SHAPES)))
def test_attention_three_requests_in_unequal_portions(dtype, shape):
    l, hidden = SHAPES[shape]
    gen = torch.Generator().manual_seed(10 + shape)
    part, t = attention_part(l, hidden, 1e-2, dtype, gen)
    seqs = [rnd(gen, n, hidden) for n in (260, 41, 150)]
    refs = [plain(l, t, s, 1e-2) for s in seqs]
    rig = Rig(part, DT[dtype], page=8, pages=128)
    cuts = [[129, 2, 89, 1, 1, 38], [1, 2, 3, 35], [64, 1, 1, 1, 1, 1, 1, 80]]
    for got, ref, n in zip(rig.run([s.to(DT[dtype]) for s in seqs], cuts), refs, (260, 41, 150)):
        near(got, ref, dtype, f"{l['type']} shape {shape}, request of {n}")
    # once more on the pages and slots the first three gave back
    for got, ref in zip(rig.run([s.to(DT[dtype]) for s in seqs[1:]], [[41], [150]]), refs[1:]):
        near(got, ref, dtype, f"{l['type']} shape {shape}, pages used again")
    rig.cache.book.check_invariants()


def value_size(d, other):
    """Keys and values of 64 or of 128 take the tcgen05 prompt kernel in bfloat16, other sizes the mma.sync or the plain one."""
    return d if d in (64, 128) else other


KINDS = {      # the window is put in by the test
    "tied": lambda d: tied(4, 4, d, 0.35),
    "gated": lambda d: gated(4, 2, d, value_size(d, 40), 0.35, rot(1e4, 4, yarn(4.0, 200))),
    "capped": lambda d: capped(4, 2, d, value_size(d, 24), 36.0 / d, rot(1e4, 4, waves(4.0, 200)), None, 30.0)}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", sorted(KINDS))
@pytest.mark.parametrize("dim,window,page", [(30, 40, 8), (32, 40, 8), (40, 90, 16), (64, 130, 32), (128, 65, 8), (32, 0, 8),
                                             (64, 0, 64), (128, 200, 32), (64, 33, 8)])
def test_planted_keys_at_every_edge(dtype, kind, dim, window, page):
    """Pairs of tokens with a strong input that the later one's query and the earlier one's key read alike, so that the
    later one's weight goes to the earlier one when it reads it: just inside the window and just outside, at a page's
    first and last place, and 250 tokens back.  A window one key off or a lost page moves those rows by the whole
    output."""
    hidden, n = 128, 300
    l = KINDS[kind](dim)
    if window:
        l["mixer"]["mask"] = dict(size=window)
    gen = torch.Generator().manual_seed(50 + window + dim)
    part, t = attention_part(l, hidden, 1e-5, dtype, gen, tie_keys=True)
    h = rnd(gen, n, hidden, std=0.3)
    w = window or 10 ** 6
    pairs = [(200, 200 - w + 1), (210, 210 - w), (180 + page, 180 + page - w + 1),        # the window's two sides
             (299, 49), (290, 5 * page), (280, 5 * page - 1), (270, 0)]                    # far back; a page's edges
    pairs = [(i, j) for i, j in pairs if 0 <= j < i]
    for p, (i, j) in enumerate(pairs):
        h[i, 5 * p:5 * p + 5] = 4.0
        h[j, hidden // 2 + 5 * p:hidden // 2 + 5 * p + 5] = 4.0
    ref = plain(l, t, h, 1e-5)
    if window:           # the planted rows do tell a window that is one key longer or shorter
        for other in (window + 1, window - 1):
            alt = plain(dict(l, mixer=dict(l["mixer"], mask=dict(size=other))), t, h, 1e-5)
            assert float((alt - ref).abs().max()) > 0.3 * float(ref.std())
    else:                # ... and the key at the very first place
        first = h.clone()
        first[0] = 0.0
        assert float((plain(l, t, first, 1e-5)[270] - ref[270]).abs().max()) > 0.3 * float(ref.std())
    for cuts in ([n], [150] + [1] * 150, [2] * 150, [209] + [1] * 91):
        rig = Rig(part, DT[dtype], page=page, pages=max(16, 2 * n // page))
        got = rig.run([h.to(DT[dtype])], [cuts])[0]
        near(got, ref, dtype, f"{kind}, planted keys, window {window}, portions {cuts[:2]}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [30, 32, 72, 64, 128])
def test_scores_at_their_bound(dtype, dim):
    """Scores many times the bound: the weights are those of +-softcap, far from a softmax without it, in prompts and for
    single tokens; and a bound far above the scores changes nothing."""
    gen = torch.Generator().manual_seed(dim)
    l = capped(4, 2, dim, value_size(dim, 16), 2.0, None, 60, 1.5)
    part, t = attention_part(l, 64, 1e-5, dtype, gen)
    h = rnd(gen, 90, 64)
    ref = plain(l, t, h, 1e-5)
    loose = plain(dict(l, mixer=dict(l["mixer"], softcap=None)), t, h, 1e-5)
    assert float((loose - ref).abs().max()) > float(ref.std())
    for cuts in ([90], [30] + [1] * 60):
        near(Rig(part, DT[dtype], page=8).run([h.to(DT[dtype])], [cuts])[0], ref, dtype, f"bounded scores {cuts[:2]}")
    l = capped(4, 2, dim, value_size(dim, 16), 0.1, None, 60, 1e4)
    part, t = attention_part(l, 64, 1e-5, dtype, gen)
    free = plain(dict(l, mixer=dict(l["mixer"], softcap=None)), t, h, 1e-5)
    near(Rig(part, DT[dtype], page=8).run([h.to(DT[dtype])], [[40] + [1] * 50])[0], free, dtype, "a bound out of reach")


@pytest.mark.parametrize("d,window,page,tied_values,cap,spread,gate", [
    (64, 0, 16, False, 0.0, 1.0, True), (128, 150, 16, False, 30.0, 8.0, False), (128, 70, 8, True, 0.0, 1.0, False),
    (64, 129, 32, True, 4.0, 6.0, True), (128, 0, 128, False, 5.0, 40.0, True), (64, 1, 8, False, 20.0, 2.0, False),
    (64, 300, 64, False, 1e3, 1.0, True)])
def test_three_prompt_kernels_agree(monkeypatch, d, window, page, tied_values, cap, spread, gate):
    """bfloat16 queries and cache rows through the tcgen05, the mma.sync and the plain kernel: portions that start inside
    a page, at its edge and far in, whose early pages the window has given back; scores under and far over the bound
    (both forms of its tanh)."""
    from ai_engine_b200.cache import PagedCache
    from ai_engine_b200.engine.step import StepContext, StepEntry
    from ai_engine_b200.kernels import ops
    from ai_engine_b200.parts import ATTENTION_WORK, CacheNeed, KVRequest
    gen = torch.Generator().manual_seed(d + window + page)
    H, G, w = 6, 2, d if tied_values else 2 * d
    cache = PagedCache([CacheNeed(0, "p", KVRequest(G, w, window, planes=1))], page, 2048 // page, 3, 1024, torch.bfloat16, DEV)
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    entries = []
    for have, n in ((0, 190), (page, 129), (517, 140)):
        slot = cache.admit()
        assert cache.ensure(slot, have + n)
        cache.advance(slot, have)
        entries.append(StepEntry(slot, have, [0] * n, []))
    ctx = StepContext(entries, cache, torch.device(DEV), err, planners=(ATTENTION_WORK,))
    lc = cache.part_cache(0, "p", ctx)
    T = ctx.T
    lc.k_pages.copy_(torch.randn(lc.k_pages.shape, generator=gen).to(DEV))
    for r, e in enumerate(entries):              # a place that no token has written yet holds no number
        for p in range(e.start + len(e.tokens), -(-(e.start + len(e.tokens)) // page) * page):
            lc.k_pages[int(lc.block_table[r, p // page]), :, p % page] = float("nan")
    q = (torch.randn(T, H, d, generator=gen) * spread).to(DEV).to(torch.bfloat16)
    logits = torch.randn(T, H * d + 12, generator=gen).to(DEV)[:, 8:8 + H * d] if gate else None
    go = lambda: ops.sink_attention(q, lc.k_pages, None, None, None, None, ctx, ctx.plan(ATTENTION_WORK), lc.block_table, d,
                                    d ** -0.5, window, 0, softcap=cap, tied=tied_values, gate_logits=logits).float().cpu()
    calls = []
    real = ops.paged_attention_prefill_rows
    monkeypatch.setattr(ops, "paged_attention_prefill_rows", lambda *a, **k: calls.append(real(*a, **k)) or calls[-1])
    tc = go()
    assert calls == [True]
    monkeypatch.setattr(ops, "paged_attention_prefill_rows", lambda *a, **k: False)
    mma = go()
    monkeypatch.setattr(ops, "sink_attention_fast", lambda *a, **k: False)
    ref = go()
    assert int(err.item()) == 0 and bool(torch.isfinite(ref).all())
    for name, got in (("tcgen05", tc), ("mma.sync", mma)):
        assert float((got - ref).abs().max()) <= 6e-3 * float(ref.abs().max()), name       # one rounding to bfloat16
        assert float((got - ref).abs().mean()) <= 2e-4 * float(ref.abs().max()), name


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,e,dims,unit,mag", [(4, 2, 20, 12, 12, True, 1.0), (3, 1, 10, 6, 10, True, 1.0), (6, 3, 128, 64, 128, True, 1.0),
                                                   (2, 2, 144, 8, 50, True, 1.0), (5, 1, 16, 36, 6, False, 1.2), (4, 4, 64, 64, 2, False, 0.8),
                                                   (2, 1, 7, 9, 4, False, 1.3), (8, 2, 32, 32, 0, True, 1.0), (1, 1, 128, 128, 66, False, 1.4)])
def test_prepare_kernel_rows_and_queries(dtype, H, G, d, e, dims, unit, mag):
    """Biases, rotation of neighbouring pairs with a magnitude on the rotated elements only, unit heads behind it: queries
    and the cache rows [k | v] of a portion that starts in the middle of a page."""
    from ai_engine_b200.kernels import ops
    from ai_engine_b200.cache import PagedCache
    from ai_engine_b200.engine.step import StepContext, StepEntry
    from ai_engine_b200.parts import CacheNeed, KVRequest
    gen = torch.Generator().manual_seed(d * e)
    cache = PagedCache([CacheNeed(0, "p", KVRequest(G, d + e, planes=1))], 8, 16, 2, 128, DT[dtype], DEV)
    slot, T, start = cache.admit(), 21, 13
    assert cache.ensure(slot, start + T)
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    ctx = StepContext([StepEntry(slot, start, [0] * T, [])], cache, torch.device(DEV), err)
    lc = cache.part_cache(0, "p", ctx)
    n = H * d + G * (d + e)
    proj, bias, eps = rnd(gen, T, n + 3), rnd(gen, n, std=0.3), 2e-2
    freqs = [float(torch.tensor(100.0 ** (-2.0 * i / max(dims, 1)), dtype=torch.float32)) for i in range(dims // 2)]
    inv = torch.tensor(freqs, dtype=torch.float32, device=DEV) if dims else None
    q, kept = ops.normed_attn_prepare(proj.to(DEV), bias.to(DEV), None, None, eps, inv, dims, False, lc.k_pages, ctx, lc.block_table,
                                      H, G, d, e, magnitude=mag, unit=unit)
    pos = range(start, start + T)
    full = proj[:, :n].double() + bias.double()
    turn = lambda x: pk.rotate_neighbours(x, pos, freqs, mag)
    qr, kr = turn(full[:, :H * d].view(T, H, d)), turn(full[:, H * d:(H + G) * d].view(T, G, d))
    if unit:
        qr, kr = pk.rms(qr, eps), pk.rms(kr, eps)
    v = full[:, (H + G) * d:].view(T, G, e)
    tol = 1e-5 if dtype == "float32" else 1e-2
    rows = lc.k_pages[lc.block_table[0, :5].long()].permute(1, 0, 2, 3).reshape(G, 40, d + e)[:, start:start + T].cpu().double()
    for got, ref in ((q.cpu().double(), qr), (rows[..., :d].transpose(0, 1), kr), (rows[..., d:].transpose(0, 1), v)):
        assert float((got - ref).abs().max()) <= tol * max(1.0, float(ref.abs().max()))
    assert kept is None and int(err.item()) == 0


def test_the_prepare_kernel_refuses_what_it_does_not_make():
    from ai_engine_b200.kernels import ops
    from ai_engine_b200.kernels.loader import KernelError
    gen = torch.Generator().manual_seed(1)
    part, t = attention_part(capped(2, 1, 16, 16, 0.3, rot(100.0, 8, waves(2.0, 30)), None, 5.0), 32, 1e-5, "float32", gen)
    rig = Rig(part, torch.float32, page=8, pages=8)
    ctx, lc = rig.step([(rig.admit(), 3)])
    proj, inv, ones = torch.zeros(3, 64, device=DEV), part.rope.inv_freq, torch.ones(32, device=DEV)
    go = lambda *a, **k: ops.normed_attn_prepare(proj, None, *a, lc.k_pages, ctx, lc.block_table, 2, 1, 16, 16, **k)
    with pytest.raises(KernelError):             # unit heads with split halves
        go(None, None, 1e-5, inv, 8, True, unit=True)
    with pytest.raises(KernelError):             # a magnitude with a norm over the whole projection
        go(ones, ones[:16].contiguous(), 1e-5, inv, 8, False, magnitude=1.2)
    with pytest.raises(KernelError):             # tied values where the row has a value of its own
        go(None, None, 1e-5, None, 0, False, tied=True)
