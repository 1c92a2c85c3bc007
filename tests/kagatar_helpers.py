"""Shared by the Kagatar tests: small configurations (between them every size, count and constant differs, some are 1 or
equal where the others differ), model folders with random weights, and the plain implementation as oracle."""
from __future__ import annotations

import os

import torch

import plain_kagatar as pk
from tizodra_helpers import DEV, Rig, close, env, ids_for, load, oracle_dtype, read_tensors  # noqa: F401  (shared rig)


def yarn(factor, original, fast=32.0, slow=1.0):
    return dict(factor=factor, original=original, fast=fast, slow=slow)


def waves(factor, original, low=1.0, high=4.0):
    return dict(factor=factor, original=original, low=low, high=high)


def rot(base, dims, scaling=None):
    return dict(base=base, dims=dims, **(dict(scaling=scaling) if scaling else {}))


def _mixer(kind, heads, kv_heads, dim, vdim, scale, size, **more):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, **{k: v for k, v in more.items() if v is not None})
    if size:
        m["mask"] = dict(size=size)
    return dict(type=kind, mixer=m)


def tied(heads, kv_heads, dim, scale, size=None):
    return _mixer("attention", heads, kv_heads, dim, dim, scale, size)


def gated(heads, kv_heads, dim, vdim, scale, r=None, size=None):
    return _mixer("attention_2", heads, kv_heads, dim, vdim, scale, size, rot=r)


def capped(heads, kv_heads, dim, vdim, scale, r=None, size=None, cap=None):
    return _mixer("attention_3", heads, kv_heads, dim, vdim, scale, size, rot=r, softcap=cap)


def layer(l, ff=None, limit=None):
    return dict(l, mlp=None if ff is None else dict(kind="dense", ff=ff, **(dict(limit=limit) if limit is not None else {})))


def config(vocab, width, eps, layers, scale=None, cap=None, loop=None):
    c = dict(architecture="Kagatar", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)
    if scale is not None:
        c["embedding"] = dict(scale=scale)
    if cap is not None:
        c["logit_softcap"] = cap
    if loop is not None:
        c["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return c


# odd sizes; windows shorter than a prompt and no multiple of a page; grouped heads; partial rotations; a layer without
# feed-forward inside a loop that starts behind the first layer and runs three times; a tight clamp and a wide one
CFG_A = config(211, 96, 1e-4, [
    layer(capped(6, 2, 20, 12, 0.35, rot(3000.0, 12, waves(4.0, 60)), 37, 6.0), 80, 0.4),
    layer(gated(5, 1, 12, 28, 0.4, rot(700.0, 6, yarn(8.0, 40, 8.0, 0.5))), 56, 2.5),
    layer(tied(4, 2, 36, 0.12, 21)),
    layer(capped(3, 3, 44, 8, 0.2, rot(20000.0, 44, waves(2.0, 300, 2.0, 5.0)), 50, 20.0), 72, 1.0),
], scale=2.0, cap=9.0, loop=(1, 3, 3))

# the sizes the tensor-core kernels take in bfloat16 (keys and values of 32, 64 and 128, and sizes between them that are
# filled up), windows that a tile of 128 tokens crosses, feed-forwards in steps of 64 and not; the loop from the first
# layer on
CFG_B = config(257, 128, 1e-5, [
    layer(tied(4, 2, 64, 0.1, 70), 256, 0.8),
    layer(gated(4, 1, 64, 64, 0.12, rot(50000.0, 32, yarn(16.0, 256, 16.0, 2.0))), 128, 1.2),
    layer(capped(2, 2, 128, 32, 0.06, rot(10000.0, 128, waves(8.0, 128)), 130, 12.0), 200, 3.0),
    layer(tied(2, 1, 128, 0.05, 133), 64, 0.5),
    layer(gated(6, 3, 40, 56, 0.2, rot(900.0, 40, yarn(3.0, 100))), 192, 0.6),
    layer(capped(4, 2, 32, 88, 0.25, rot(1e6, 16, waves(32.0, 2048)), 64, 40.0), 128, 0.9),
    layer(tied(9, 1, 24, 0.2, 90), 320, 1.7),
], scale=1.0, cap=30.0, loop=(0, 3, 2))

# no loop and no bounds; sizes of 1: one head, windows of one and of two keys, a rotation of one pair; a width that is no
# multiple of 8; an unscaled embedding; no rotation and no stretching where they may be absent
CFG_C = config(130, 36, 1e-6, [
    layer(tied(1, 1, 12, 0.3, 2), 52),
    layer(gated(1, 1, 8, 44, 0.4, rot(50.0, 2)), 24, 0.7),
    layer(capped(3, 3, 10, 6, 0.5, rot(100.0, 10), 1, 3.0), 20, 0.3),
    layer(capped(2, 1, 14, 14, 0.3, None, 9), 33, 1.1),
    layer(gated(3, 1, 16, 4, 0.3)),
])

# a loop of one layer that runs once and is the last layer; windows everywhere and nowhere
CFG_D = config(97, 48, 1e-3, [
    layer(gated(2, 2, 8, 8, 0.5, rot(10000.0, 8, yarn(2.0, 30, 4.0, 1.0)), 16), 32, 1.0),
    layer(tied(2, 2, 16, 0.3), 40, 2.0),
    layer(capped(4, 2, 24, 12, 0.3, rot(777.0, 24, waves(16.0, 50, 0.5, 8.0)), 5, 8.0), 64, 0.5),
], scale=0.5, cap=4.0, loop=(2, 3, 1))

CONFIGS = {"A": CFG_A, "B": CFG_B, "C": CFG_C, "D": CFG_D}


def make_dir(tmp_path, name, seed=0, gain=3.0):
    """A model folder for configuration `name`: random weights N(0, 0.07) written by the engine's random-weights mode, norm
    weights 1 + N(0, 0.1), query projections multiplied by `gain` so that scores spread and single keys stand out (heads
    that are divided by their root mean square lean on their scale instead), gate and up projections by 3 so that the
    clamps bind, and the embedding scaled up to a stream of order one."""
    import ai_engine_b200 as aie
    from safetensors import safe_open
    from safetensors.torch import save_file

    d = os.path.join(str(tmp_path), f"kagatar_{name}_{seed}_{gain}")
    if os.path.exists(os.path.join(d, "model.safetensors")):
        return d
    aie.write_random_model(aie.KagatarConfig.from_dict(CONFIGS[name]), d, seed=seed, std=0.07, norm_std=0.1)
    path = os.path.join(d, "model.safetensors")
    tensors = {}
    with safe_open(path, "pt") as f:
        for k in f.keys():
            t = f.get_tensor(k)
            by = gain if k.endswith("mix.q") else 3.0 if k.endswith(("mlp.gate", "mlp.up")) else 10.0 if k == "embed" else 1.0
            tensors[k] = (t.float() * by).to(t.dtype).clone().contiguous()          # a copy: the file is written again below
    save_file(tensors, path)
    return d


_REFS = {}


def plain_logits(d, name, ids, dtype=torch.float64):
    """[len(ids), vocab] from the plain implementation (cached per folder and sequence)."""
    key = (d, tuple(ids), dtype)
    if key not in _REFS:
        _REFS[key] = pk.forward(read_tensors(d), CONFIGS[name], ids, dtype=dtype).to(torch.float64).numpy()
    return _REFS[key]
