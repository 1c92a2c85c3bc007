"""Each mechanism of the Vatazen design alone, on a real cache and step context, against the plain implementation: the
shift towards the token before (portions, slots used again), the addition of a gated and normed branch (parts of a
product, expert rows, the next layer's shift made ahead), the side input, the router, experts without a gate, the
difference of two maps, latent attention with a window, a sink and stretched positions, and differential attention in
chunks (requests in unequal portions; keys planted just inside and just outside every window and chunk, at a page's
edges and far back, as one prompt, decoded token by token and in portions of two; the sink's share), and the per-head
products of small steps."""
import math

import numpy as np
import pytest
import torch

import plain_vatazen as pv
from test_fokisun_parts_gpu import DT, f64, near, rnd
from vatazen_helpers import DEV, Rig, env, load, yarn

pytestmark = pytest.mark.gpu
BOTH = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])


# ---------------------------------------------------------------------------------------------------
class ShiftRig(Rig):
    """Steps a TokenShift, whose input is float32 and whose output is the pair (shifted, as it is)."""

    def __init__(self, part, dtype):
        super().__init__(part, dtype, page=8, pages=8, max_seqs=3)
        outer = part.forward

        class Both:
            def forward(_, h, ctx, lc):
                shifted, plain = outer(h.float(), ctx, lc, plain=True)
                assert plain.dtype == dtype and torch.equal(plain.float(), h.float().to(dtype).float())
                return shifted
        self.part = Both()


def shift_part(w, dtype):
    from ai_engine_b200.parts import PartSpec, TokenShift
    return load(TokenShift(PartSpec("token_shift", dict(size=w.numel()), dict(weight="s")), env(DT[dtype], w.numel())), {"s": w}, DT[dtype])


@BOTH
@pytest.mark.parametrize("D", [5, 36, 96, 1032])
def test_shift_in_portions_and_on_slots_used_again(dtype, D):
    gen = torch.Generator().manual_seed(D)
    w = rnd(gen, D, std=0.5, mean=0.4)
    seqs = [rnd(gen, n, D) for n in (70, 9, 33)]
    rig = ShiftRig(shift_part(w, dtype), DT[dtype])
    refs = [pv.token_shift(s.double(), w.double()) for s in seqs]
    for cuts in ([[70], [9], [33]], [[1] * 30 + [40], [2, 2, 5], [3] * 11], [[2] * 35, [1] * 9, [32, 1]]):
        for got, ref in zip(rig.run(seqs, cuts), refs):
            near(got, ref, dtype, f"shift {D}, {[c[:2] for c in cuts]}")


# ---------------------------------------------------------------------------------------------------
def branch_ref(x, y, w, eps, z=None, zb=None, b=None):
    y = y if b is None else y + b
    if z is not None:
        y = y * torch.sigmoid(z if zb is None else z + zb)
    return x + pv.rms(y, w, eps)


@pytest.mark.parametrize("D", [7, 36, 96, 1024, 2048, 5000])
def test_a_gated_and_normed_branch_joins_the_stream(D):
    from ai_engine_b200.kernels import ops
    gen = torch.Generator().manual_seed(D)
    T, eps = 19, 1e-3
    x, w = rnd(gen, T, D), rnd(gen, D, mean=1.0, std=0.3)
    y, z = rnd(gen, 4, T, D), rnd(gen, 3, T, D + 8)
    b, zb = rnd(gen, D, std=0.5), rnd(gen, D, std=0.5)
    d = lambda t: t.to(DEV)
    ref = branch_ref(x.double(), y.double().sum(0), w.double(), eps, z.double().sum(0)[:, :D], zb.double(), b.double())
    xs = d(x).clone()
    out = ops.gated_norm_add(xs, d(y), d(w), eps, out_dtype=torch.bfloat16, gate=d(z), gate_bias=d(zb), bias=d(b))
    near(xs.cpu(), ref, "float32", f"stream {D}")
    assert out.dtype == torch.bfloat16 and torch.equal(out.float(), xs.to(torch.bfloat16).float())
    xs = d(x).clone()                                    # neither gate nor bias; the new stream is handed back itself
    assert ops.gated_norm_add(xs, d(y[0]), d(w), eps, out_dtype=torch.float32).data_ptr() == xs.data_ptr()
    near(xs.cpu(), branch_ref(x.double(), y[0].double(), w.double(), eps), "float32", f"stream {D} ungated")
    # a token's expert rows, summed by weight; one pair has no row
    rows, top = rnd(gen, 3 * T, D), 3
    order = torch.randperm(3 * T, generator=gen).int()
    order[5] = -1
    wt = rnd(gen, T, top)
    picked = torch.where((order.view(T, top, 1) >= 0), rows.double()[order.clamp(min=0).long()].view(T, top, D), 0.0)
    ref = branch_ref(x.double(), (picked * wt.double()[:, :, None]).sum(1), w.double(), eps, z[0, :, :D].double(), zb.double())
    xs = d(x).clone()
    ops.gated_norm_add(xs, ops.ExpertRows(d(rows), d(order), d(wt)), d(w), eps, gate=d(z[0]), gate_bias=d(zb))
    near(xs.cpu(), ref, "float32", f"stream {D}, expert rows")


@BOTH
def test_the_next_layers_shift_made_ahead(dtype):
    """Two requests that bring one token each: the addition's kernel leaves what the shift's own kernel leaves,
    in its output and in the state; in a step with a portion it refuses."""
    from ai_engine_b200.kernels import ops
    from ai_engine_b200.kernels.loader import KernelError
    gen = torch.Generator().manual_seed(3)
    for D in (36, 99, 2048):
        w, nw = rnd(gen, D, std=0.5), rnd(gen, D, mean=1.0)
        part = shift_part(w, dtype)
        rig = Rig(part, DT[dtype], page=8, pages=8)
        slots = [rig.admit(), rig.admit()]
        ctx, lc = rig.step([(slots[1], 1), (slots[0], 1)])
        lc.state.copy_(rnd(gen, *lc.state.shape))
        before = lc.state.clone()
        x, y = rnd(gen, 2, D).to(DEV), rnd(gen, 2, 2, D).to(DEV)
        xs = x.clone()
        plain, shifted = ops.gated_norm_add(xs, y, nw.to(DEV), 1e-5, out_dtype=DT[dtype], next_shift=part.ahead(lc), ctx=ctx)
        after = lc.state.clone()
        lc.state.copy_(before)
        want, want_plain = part.forward(xs, ctx, lc, plain=True)
        assert torch.equal(after, lc.state) and torch.equal(plain.float(), want_plain.float())
        assert float((shifted.float() - want.float()).abs().max()) <= (1e-6 if dtype == "float32" else 2e-2) * float(want.abs().max())
        ctx2, lc2 = rig.step([(slots[0], 3)])
        with pytest.raises(KernelError):
            ops.gated_norm_add(rnd(gen, 3, D).to(DEV), rnd(gen, 3, D).to(DEV), nw.to(DEV), 1e-5, out_dtype=DT[dtype],
                               next_shift=part.ahead(lc2), ctx=ctx2)


# ---------------------------------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("D,n,levels,T", [(40, 12, 3, 70), (128, 32, 5, 9), (36, 1, 2, 130), (64, 72, 1, 1)])
def test_side_input(dtype, D, n, levels, T):
    from ai_engine_b200.parts import PartSpec, TokenSide
    gen = torch.Generator().manual_seed(D + n)
    vocab = 50
    t = {"e": rnd(gen, vocab, levels * n), "g": rnd(gen, n, D, std=0.3), "p": rnd(gen, D, n, std=0.3)}
    ids = torch.randint(0, vocab, (T,), generator=gen)
    x = rnd(gen, T, D)
    ctx = type("C", (), {"err": torch.zeros(1, dtype=torch.int32, device=DEV), "token_ids": ids.int().to(DEV)})()
    for i in range(levels):
        part = load(TokenSide(PartSpec("token_side", dict(hidden_size=D, size=n, vocab_size=vocab, layers=levels, index=i),
                                       dict(table="e", gate="g", proj="p")), env(DT[dtype], D)), t, DT[dtype])
        out = part.forward(x.to(DEV).to(DT[dtype]), ctx).double().cpu()
        out = out.sum(0) if out.dim() == 3 else out
        e = t["e"].double()[ids][:, i * n:(i + 1) * n]
        near(out, (pv.gelu_tanh(x.double() @ t["g"].double().T) * e) @ t["p"].double().T, dtype, f"side input of layer {i}")
    assert int(ctx.err.item()) == 0
    ctx.token_ids[0] = vocab                             # a token outside the table is an error, not a read
    part.forward(x.to(DEV).to(DT[dtype]), ctx)
    assert int(ctx.err.item()) == 1


@pytest.mark.parametrize("E,top", [(8, 3), (1, 1), (5, 5), (33, 4), (64, 8), (100, 7), (250, 2), (700, 9), (90, 70)])
def test_router_choices_and_weights(E, top):
    from ai_engine_b200.kernels import ops
    gen = torch.Generator().manual_seed(E)
    T, D = 150, 24
    h, w, b = rnd(gen, T, D), rnd(gen, E, D, std=0.5), rnd(gen, E, std=1.5)
    ids, weights = pv.route(h.double(), {"router": w.double(), "router.b": b.double()}, "", dict(experts=E, top=top))
    z = (h @ w.T)
    parts = torch.stack([z * 0.25, z * 0.75]) if E % 2 else z
    wide = torch.cat([parts, torch.full(parts.shape[:-1] + (5,), 1e9)], dim=-1)          # columns behind the logits are not read
    got_ids, got_w = ops.route_chosen(wide.to(DEV), b.to(DEV), E, top)
    lead = torch.sort(h.double() @ w.double().T + b.double(), dim=1, descending=True).values
    ok = lead[:, top - 1] - lead[:, top] > 1e-4 if top < E else torch.ones(T, dtype=torch.bool)
    assert bool(ok[:8].any())
    order, ref = got_ids.cpu().long().sort(dim=1), ids.sort(dim=1)
    assert torch.equal(order.values[ok], ref.values[ok])
    assert float((got_w.cpu().double().gather(1, order.indices) - weights.gather(1, ref.indices))[ok].abs().max()) < 1e-5
    assert float((got_w.sum(dim=1).cpu() - 1.0).abs().max()) < 1e-5
    # equal logits: the lower numbers are taken, each once; far apart: the weights still sum to one
    tie_ids, tie_w = ops.route_chosen(torch.zeros(2, E, device=DEV), None, E, top)
    assert tie_ids.cpu().tolist() == [list(range(top))] * 2 and np.allclose(tie_w.cpu(), 1.0 / top)
    far = torch.arange(E, device=DEV, dtype=torch.float32)[None] * 200.0 - 3000.0
    far_ids, far_w = ops.route_chosen(far.contiguous(), None, E, top)
    assert far_ids.cpu()[0].tolist() == list(range(E - 1, E - 1 - top, -1)) and float(far_w[0, 0]) == 1.0


@BOTH
@pytest.mark.parametrize("D,F,E,top,T", [(40, 24, 6, 2, 70), (128, 128, 4, 2, 150), (36, 20, 1, 1, 5), (256, 128, 8, 3, 1), (128, 256, 5, 5, 40)])
def test_experts_without_a_gate(dtype, D, F, E, top, T):
    from ai_engine_b200.kernels import ops
    from ai_engine_b200.parts import PartSpec, RoutedMoE
    gen = torch.Generator().manual_seed(D + F + E)
    t = {"router": rnd(gen, E, D, std=0.3), "router.b": rnd(gen, E, std=0.5)}
    for e in range(E):
        t.update({f"e{e}.up": rnd(gen, F, D, std=0.2), f"e{e}.down": rnd(gen, D, F, std=0.2)})
    part = load(RoutedMoE(PartSpec("routed_moe", dict(hidden_size=D, num_experts=E, top=top, intermediate_size=F,
                                                      activation="relu_squared", score="softmax_chosen"),
                                   dict(router="router", router_bias="router.b", up="e{e}.up", down="e{e}.down")),
                          env(DT[dtype], D)), t, DT[dtype])
    h = rnd(gen, T, D)
    margins = []
    ref = pv.moe_ff(h.double(), f64(t), "", dict(router=dict(experts=E, top=top)), margins)
    ctx = type("C", (), {"err": torch.zeros(1, dtype=torch.int32, device=DEV)})()
    hd = h.to(DEV).to(DT[dtype])
    clear = margins[0] > 1e-3                            # a close call may turn either way under rounding
    near(part.forward(hd, ctx).double().cpu()[clear], ref[clear], dtype, "experts")
    # rows left for the consumer, logits made by it
    z = (h @ t["router"].T).to(DEV)
    rows = part.forward(hd, ctx, logits=z, leave_rows=True)
    assert isinstance(rows, ops.ExpertRows)
    x, w = rnd(gen, T, D), torch.ones(D)
    xs = x.to(DEV).clone()
    ops.gated_norm_add(xs, rows, w.to(DEV), 1e-5)
    near((xs.cpu() - x)[clear], pv.rms(ref, 1.0, 1e-5)[clear], dtype, "experts' rows summed by the norm")


def test_softmax_chosen_takes_no_groups_and_gated_experts_no_other_activation():
    from ai_engine_b200.parts import PartSpec, RoutedMoE
    base = dict(hidden_size=16, num_experts=4, top=2, intermediate_size=8)
    names = dict(router="r", router_bias="b", up="u{e}", down="d{e}")
    e = env(torch.float32, 16)
    with pytest.raises(ValueError, match="softmax_chosen"):
        RoutedMoE(PartSpec("m", dict(base, score="softmax_chosen", groups=2, keep=1), names), e)
    with pytest.raises(ValueError, match="silu"):
        RoutedMoE(PartSpec("m", dict(base, activation="relu_squared"), dict(names, gate="g{e}")), e)
    with pytest.raises(ValueError, match="tanh"):
        RoutedMoE(PartSpec("m", dict(base, activation="tanh"), names), e)


@BOTH
@pytest.mark.parametrize("H,e", [(3, 4), (5, 20), (4, 64), (2, 128), (3, 200), (1, 7)])
def test_difference_of_two_maps(dtype, H, e):
    from ai_engine_b200.kernels import ops
    gen = torch.Generator().manual_seed(H * 100 + e)
    a = rnd(gen, 37, H, 2, e)
    got = ops.map_difference(a.view(37, 2 * H, e).to(DEV), 0.6, 1e-4, 0.75, DT[dtype])
    o = a[:, :, 0].double() - 0.6 * a[:, :, 1].double()
    near(got.cpu(), (pv.rms(o, 1.0, 1e-4) * 0.75).reshape(37, H * e), dtype, "difference")


# ---------------------------------------------------------------------------------------------------
def latent_part(m, hidden, eps, dtype, gen, tie_keys=False, exact=True):
    from ai_engine_b200.parts import LatentAttention, PartSpec, RotaryEncoding
    H, d, r, e, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    t = {"q": rnd(gen, H * (d + r), hidden, std=0.3), "dkv": rnd(gen, rank + r, hidden, std=0.3),
         "dkv.norm": rnd(gen, rank, std=0.1, mean=1.0), "uk": rnd(gen, H * d, rank, std=0.3), "uv": rnd(gen, H * e, rank, std=0.3),
         "sink": rnd(gen, H, std=1.0), "o": rnd(gen, hidden, H * e, std=0.2)}
    if tie_keys:          # a query reads the first half of the input as the keys read the second
        fold = torch.einsum("hdr,rx->hdx", t["uk"].view(H, d, rank), t["dkv"][:rank])
        q = t["q"].view(H, d + r, hidden) * 0.1
        q[:, :d] = torch.roll(fold, -(hidden // 2), dims=2)
        t["q"] = q.reshape(H * (d + r), hidden).to(torch.bfloat16).float()
    e_ = env(DT[dtype], hidden)
    pe = None
    if m.get("rot"):
        sc = m["rot"].get("scaling")
        rope = RotaryEncoding(PartSpec("rotary", dict(rot_dim=m["rot"]["dims"], theta=m["rot"]["base"], layout="interleaved",
                                                      scaling=dict(type="yarn", **sc) if sc else None)), e_)
        rope.load(None)
        e_.position_encodings["r"] = rope
        pe = "r"
    spec = PartSpec("latent_attention", dict(
        hidden_size=hidden, num_heads=H, head_dim=d, rot_dim=r, value_dim=e, kv_rank=rank, scale=m["scale"],
        window=(m.get("mask") or {}).get("size", 0), eps=eps, sink=True, exact_weights=exact, position_encoding=pe),
        dict(q="q", dkv="dkv", dkv_norm="dkv.norm", uk="uk", uv="uv", sink="sink", o="o"))
    return load(LatentAttention(spec, e_), t, DT[dtype]), t


def lm(heads, dim, rot_dim, vdim, rank, scale, size=None, base=10000.0, scaling=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=rank, scale=scale)
    if rot_dim:
        m["rot"] = dict(base=base, dims=rot_dim, **(dict(scaling=scaling) if scaling else {}))
    if size:
        m["mask"] = dict(size=size)
    return m


LATENT_SHAPES = [
    (lm(4, 48, 16, 40, 64, 0.1, 50, 20000.0, yarn(4.0, 100, 8.0, 0.5)), 96),
    (lm(5, 12, 8, 20, 24, 0.22, 37, 3000.0, yarn(16.0, 64)), 40),
    (lm(1, 8, 2, 12, 6, 0.3, 1), 36),
    (lm(2, 64, 32, 64, 128, 0.04, None, 100.0, yarn(3.0, 30, 4.0, 1.0)), 128),
    (lm(18, 16, 16, 16, 192, 0.12, 130), 64),            # more heads than one tile of the tensor-core kernel holds
    (lm(2, 24, 0, 8, 64, 0.15, 2), 64),
]


@BOTH
@pytest.mark.parametrize("shape", range(len(LATENT_SHAPES)))
def test_latent_attention_three_requests_in_unequal_portions(dtype, shape):
    m, hidden = LATENT_SHAPES[shape]
    gen = torch.Generator().manual_seed(30 + shape)
    part, t = latent_part(m, hidden, 1e-5, dtype, gen)
    seqs = [rnd(gen, n, hidden) for n in (300, 41, 150)]
    refs = [pv.latent_attention(s.double(), f64(t), "", m, 1e-5) for s in seqs]
    rig = Rig(part, DT[dtype], page=8, pages=128)
    cuts = [[129, 2, 127, 1, 1, 40], [1, 2, 3, 35], [64, 1, 1, 1, 1, 1, 1, 80]]
    for got, ref, n in zip(rig.run([s.to(DT[dtype]) for s in seqs], cuts), refs, (300, 41, 150)):
        near(got, ref, dtype, f"latent attention shape {shape}, request of {n}")
    for got, ref in zip(rig.run([s.to(DT[dtype]) for s in seqs[:2]], [[300], [1] * 41]), refs):
        near(got, ref, dtype, f"latent attention shape {shape}, pages used again")
    rig.cache.book.check_invariants()


def plant(h, pairs):
    """Strong inputs that the later token's query and the earlier token's key read alike."""
    half = h.shape[1] // 2
    for p, (i, j) in enumerate(pairs):
        h[i, 5 * p:5 * p + 5] = 8.0
        h[j, half + 5 * p:half + 5 * p + 5] = 8.0


@BOTH
@pytest.mark.parametrize("rank", [40, 64])               # the second takes the tensor-core kernel in bfloat16
@pytest.mark.parametrize("window,page", [(40, 8), (90, 16), (130, 32), (0, 8)])
def test_latent_attention_planted_keys_at_every_edge(dtype, window, page, rank):
    hidden, n = 128, 300
    m = lm(4, 32, 8, 24, rank, 0.05, window or None, 1000.0, yarn(4.0, 64))
    gen = torch.Generator().manual_seed(50 + window)
    part, t = latent_part(m, hidden, 1e-5, dtype, gen, tie_keys=True)
    h = rnd(gen, n, hidden, std=0.3)
    w = window or 10 ** 6
    pairs = [(200, 200 - w + 1), (210, 210 - w), (180 + page, 180 + page - w + 1),        # the window's two sides
             (299, 49), (290, 5 * page), (280, 5 * page - 1), (270, 0)]                    # far back; a page's edges
    pairs = [(i, j) for i, j in pairs if 0 <= j < i]
    plant(h, pairs)
    tw = f64(t)
    ref = pv.latent_attention(h.double(), tw, "", m, 1e-5)
    if window:           # the planted rows do tell a window that is one key longer or shorter
        for other in (window + 1, window - 1):
            alt = pv.latent_attention(h.double(), tw, "", dict(m, mask=dict(size=other)), 1e-5)
            assert float((alt - ref).abs().max()) > 0.3 * float(ref.std())
    first = max(1, min(j for _, j in pairs))
    for cuts in ([n], [150] + [1] * 150, [2] * 150, [first] + [1] * (n - first)):
        rig = Rig(part, DT[dtype], page=page, pages=max(16, 2 * n // page))
        near(rig.run([h.to(DT[dtype])], [cuts])[0], ref, dtype, f"planted keys, window {window}, portions {cuts[:2]}")


@BOTH
@pytest.mark.parametrize("rank", [24, 64])
def test_the_latent_sink_takes_its_share(dtype, rank):
    """Sinks of -9 .. 9 beside scores of order one: heads that keep all of their weight, heads that lose all of it, at the
    first token and behind a hundred, in prompts and token by token."""
    m, hidden = lm(6, 16, 4, 8, rank, 0.1, 60), 64
    gen = torch.Generator().manual_seed(5)
    part, t = latent_part(m, hidden, 1e-5, dtype, gen)
    t["sink"] = torch.tensor([-9.0, -1.0, 0.0, 1.5, 4.0, 9.0])
    part.sink = t["sink"].to(DEV)
    h = rnd(gen, 130, hidden)
    ref = pv.latent_attention(h.double(), f64(t), "", m, 1e-5)
    without = pv.latent_attention(h.double(), dict(f64(t), sink=torch.full((6,), -1e9, dtype=torch.float64)), "", m, 1e-5)
    assert float((ref - without).abs().max(dim=1).values.min()) > 0.05 * float(ref.std())
    for cuts in ([130], [1] * 130, [2] * 65):
        near(Rig(part, DT[dtype], page=8, pages=32).run([h.to(DT[dtype])], [cuts])[0], ref, dtype, f"sinks, portions {cuts[:2]}")


# ---------------------------------------------------------------------------------------------------
def diff_part(m, hidden, eps, dtype, gen, tie_keys=False):
    from ai_engine_b200.parts import DifferentialAttention, PartSpec
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    t = {"q": rnd(gen, H * 2 * d, hidden, std=0.25), "k": rnd(gen, G * 2 * d, hidden, std=0.25), "v": rnd(gen, G * e, hidden, std=0.25),
         "q.b": rnd(gen, H * 2 * d, std=0.2), "k.b": rnd(gen, G * 2 * d, std=0.2), "v.b": rnd(gen, G * e, std=0.2),
         "q.norm": rnd(gen, d, std=0.2, mean=2.0), "k.norm": rnd(gen, d, std=0.2, mean=1.0),
         **{n: rnd(gen, d, std=0.2) for n in ("lq1", "lk1", "lq2", "lk2")},
         "o": rnd(gen, hidden, H * e, std=0.2), "o.b": rnd(gen, hidden, std=0.2)}
    if tie_keys:                    # k reads the second half of the input as q reads the first
        t["k"] = torch.roll(t["q"][:G * 2 * d], hidden // 2, dims=1).contiguous()
        for n in ("q.b", "k.b"):
            t[n].zero_()
        t["q.norm"].fill_(3.0)
        t["k.norm"].fill_(1.0)
    spec = PartSpec("differential_attention", dict(
        hidden_size=hidden, num_heads=H, num_kv_heads=G, head_dim=d, value_dim=e, scale=m["scale"],
        chunk=(m.get("mask") or {}).get("size", 0), eps=eps, diff=m["diff"]),
        dict(q="q", k="k", v="v", o="o", q_bias="q.b", k_bias="k.b", v_bias="v.b", o_bias="o.b", q_norm="q.norm",
             k_norm="k.norm", lq1="lq1", lk1="lk1", lq2="lq2", lk2="lk2"))
    return load(DifferentialAttention(spec, env(DT[dtype], hidden)), t, DT[dtype]), t


def dm(heads, kv_heads, dim, vdim, scale, diff, size=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, diff=diff)
    if size:
        m["mask"] = dict(size=size)
    return m


DIFF_SHAPES = [
    (dm(8, 2, 64, 40, 0.11, 0.3, 100), 96), (dm(6, 2, 16, 24, 0.3, 0.5, 37), 96), (dm(4, 1, 64, 32, 0.15, 0.2, 130), 128),
    (dm(2, 2, 128, 128, 0.07, 0.4), 64), (dm(1, 1, 12, 44, 0.4, 0.1, 2), 36), (dm(4, 2, 32, 128, 0.2, 0.25, 64), 64),
    (dm(10, 1, 32, 64, 0.2, 0.35, 20), 64),              # more query heads of one key/value head than a CTA's tile holds
    (dm(2, 1, 128, 64, 0.06, 0.0, 90), 64), (dm(3, 3, 200, 6, 0.05, 0.3, 1), 40),
]


@BOTH
@pytest.mark.parametrize("shape", range(len(DIFF_SHAPES)))
def test_differential_attention_three_requests_in_unequal_portions(dtype, shape):
    m, hidden = DIFF_SHAPES[shape]
    gen = torch.Generator().manual_seed(10 + shape)
    part, t = diff_part(m, hidden, 1e-3, dtype, gen)
    assert part.lam == pytest.approx(float(pv.differential_lambda(f64(t), "", m)), rel=1e-6)
    seqs = [rnd(gen, n, hidden) for n in (300, 41, 150)]
    refs = [pv.differential_attention(s.double(), f64(t), "", m, 1e-3) for s in seqs]
    rig = Rig(part, DT[dtype], page=8, pages=128)
    cuts = [[129, 2, 127, 1, 1, 40], [1, 2, 3, 35], [64, 1, 1, 1, 1, 1, 1, 80]]
    for got, ref, n in zip(rig.run([s.to(DT[dtype]) for s in seqs], cuts), refs, (300, 41, 150)):
        near(got, ref, dtype, f"differential attention shape {shape}, request of {n}")
    for got, ref in zip(rig.run([s.to(DT[dtype]) for s in seqs[:2]], [[300], [1] * 41]), refs):
        near(got, ref, dtype, f"differential attention shape {shape}, pages used again")
    rig.cache.book.check_invariants()


@BOTH
@pytest.mark.parametrize("sizes", [(16, 24), (32, 64), (64, 128), (128, 32)])    # all but the first: tensor-core kernels
@pytest.mark.parametrize("chunk,page", [(40, 8), (90, 16), (130, 32), (0, 8)])
def test_differential_attention_planted_keys_at_every_edge(dtype, chunk, page, sizes):
    """A chunk's first key, read from its second token and from its last; the last key of the chunk before, read from
    the chunk's first token and its middle; a page's edges; far back where there are no chunks.  (A large eps: where
    the two maps happen to cancel, the norm behind them would amplify bfloat16's rounding beyond any use.)"""
    hidden, n = 128, 300
    m = dm(2, 2, sizes[0], sizes[1], 8.0 / sizes[0], 0.3, chunk or None)
    gen = torch.Generator().manual_seed(60 + chunk)
    part, t = diff_part(m, hidden, 0.2, dtype, gen, tie_keys=True)
    h = rnd(gen, n, hidden, std=0.3)
    c = chunk or 10 ** 6
    pairs = [(c + 1, c), (2 * c - 1, c), (2 * c, 2 * c - 1), (2 * c + 7, 2 * c - 1), (2 * c + 9, 2 * c)] if chunk else \
        [(299, 49), (290, 5 * page), (280, 5 * page - 1), (270, 0), (150, 149)]
    pairs += [(c + page + 3, c // page * page + page), (c + page + 5, c // page * page + page - 1)] if chunk else []
    pairs = [(i, j) for i, j in pairs if 0 <= j < i < n]
    plant(h, pairs)
    tw = f64(t)
    ref = pv.differential_attention(h.double(), tw, "", m, 0.2)
    if chunk:            # the planted rows do tell a chunk that is one token longer or shorter
        for other in (chunk + 1, chunk - 1):
            alt = pv.differential_attention(h.double(), tw, "", dict(m, mask=dict(size=other)), 0.2)
            assert float((alt - ref).abs().max()) > 0.3 * float(ref.std())
    first = max(1, min(j for _, j in pairs))
    for cuts in ([n], [150] + [1] * 150, [2] * 150, [first] + [1] * (n - first)):
        rig = Rig(part, DT[dtype], page=page, pages=max(16, 2 * n // page))
        near(rig.run([h.to(DT[dtype])], [cuts])[0], ref, dtype, f"planted keys, chunk {chunk}, portions {cuts[:2]}")


# ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("T", [1, 5, 8, 9, 16, 31, 64])
@pytest.mark.parametrize("H,N,K", [(3, 48, 64), (16, 20, 96), (1, 7, 32), (2, 512, 128), (5, 128, 512)])
def test_per_head_products_of_small_steps(T, H, N, K):
    from ai_engine_b200.kernels import ops
    gen = torch.Generator().manual_seed(T + N)
    x, w = rnd(gen, T, H, K + 8), rnd(gen, H, N, K, std=0.2)
    xs = x.to(DEV).bfloat16()[:, :, :K]                  # rows further apart than they are long
    ref = torch.einsum("thk,hnk->thn", x[:, :, :K].double(), w.double())
    out = torch.full((T, H, N + 3), float("nan"), dtype=torch.float32, device=DEV)
    ops.head_linear(xs, w.to(DEV).bfloat16(), out)
    assert float((out[:, :, :N].cpu().double() - ref).abs().max()) <= 1e-5 * math.sqrt(K) * float(ref.abs().max())
    assert bool(torch.isnan(out[:, :, N:]).all())
    outb = torch.empty((T, H, N), dtype=torch.bfloat16, device=DEV)
    ops.head_linear(xs, w.to(DEV).bfloat16(), outb)
    assert float((outb.cpu().double() - ref).abs().max()) <= 6e-3 * float(ref.abs().max())
