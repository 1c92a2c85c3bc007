"""Shared by the Vatazen tests: small configurations (between them every size, count and constant differs, some are 1
or equal where the others differ), model folders with random weights, the plain implementation as oracle, and
tolerances relative to the spread of the logits."""
from __future__ import annotations

import os

import numpy as np
import torch

import plain_vatazen as pv
from zupitar_helpers import AFTER, DEV, Ref, Rig, close, env, ids_for, load, oracle_dtype, read_tensors  # noqa: F401


def yarn(factor, original, fast=32.0, slow=1.0):
    return dict(factor=factor, original=original, fast=fast, slow=slow)


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, size=None, base=10000.0, scaling=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale, rot=dict(base=base, dims=rot_dim))
    if scaling:
        m["rot"]["scaling"] = scaling
    if size:
        m["mask"] = dict(size=size)
    return dict(type="latent_attention", mixer=m)


def diff(heads, kv_heads, dim, vdim, scale, lam, size=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, diff=lam)
    if size:
        m["mask"] = dict(size=size)
    return dict(type="attention", mixer=m)


def moe(ff, experts, top):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))


def layer(l, mlp=None):
    return dict(l, mlp=mlp)


def config(vocab, width, eps, layers, scale=None, side=None):
    c = dict(architecture="Vatazen", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)
    if scale is not None:
        c["embedding"] = dict(scale=scale)
    if side is not None:
        c["token_side"] = dict(dim=side)
    return c


# odd sizes; windows and chunks shorter than a prompt and none a multiple of a page; grouped heads; a layer without
# feed-forward; two stretchings of the positions and none
CFG_A = config(211, 96, 1e-4, [
    layer(diff(6, 2, 12, 20, 0.3, 0.4, 50), moe(40, 6, 2)),
    layer(latent(5, 12, 8, 20, 24, 0.25, 37, 3000.0, yarn(4.0, 64, 8.0, 0.5)), moe(24, 5, 3)),
    layer(latent(3, 20, 4, 12, 40, 0.2, 21, 500.0)),
    layer(diff(4, 4, 24, 8, 0.2, 0.15, 23), moe(48, 4, 1)),
    layer(latent(2, 8, 16, 28, 20, 0.22, 70, 100000.0, yarn(16.0, 128)), moe(32, 7, 7)),
], scale=0.7, side=12)

# the sizes the tensor-core kernels take in bfloat16 (maps of 32, 64 and 128 over values of 32, 64 and 128; latents of
# 64, 128 and 192; experts of 128 on a width of 128), a window and a chunk that a tile of 128 tokens crosses
CFG_B = config(257, 128, 1e-5, [
    layer(latent(4, 32, 16, 48, 64, 0.15, 70, 50000.0, yarn(8.0, 256, 16.0, 2.0)), moe(128, 6, 2)),
    layer(diff(4, 2, 64, 64, 0.13, 0.25, 90), moe(128, 4, 3)),
    layer(diff(2, 1, 128, 32, 0.09, 0.35, 130), moe(64, 3, 1)),
    layer(latent(2, 64, 32, 64, 128, 0.1, 33), moe(128, 2, 1)),
    layer(diff(2, 2, 32, 128, 0.2, 0.1, 64)),
    layer(latent(17, 16, 48, 16, 192, 0.12, 140, 10000.0, yarn(2.0, 100)), moe(64, 5, 5)),
], scale=2.0, side=32)

# sizes of 1: one head, one expert, one choice, a window of one and of two keys, a chunk of one and of two; a width that
# is no multiple of 8; an unscaled embedding; a side input of one number
CFG_C = config(130, 36, 3e-2, [
    layer(diff(1, 1, 12, 44, 0.4, 0.2, 2), moe(52, 1, 1)),
    layer(latent(1, 8, 2, 12, 6, 0.3, 2), moe(44, 3, 3)),
    layer(diff(3, 1, 10, 6, 0.35, 0.0, 1), moe(60, 2, 1)),
    layer(latent(3, 4, 6, 20, 10, 0.3, 1, 50.0, yarn(3.0, 20, 4.0, 1.0))),
], side=1)

# no masks but causality, no side input, no rotated part in one layer
CFG_D = config(97, 48, 1e-5, [
    layer(latent(3, 16, 0, 8, 16, 0.2), moe(16, 8, 2)),
    layer(diff(4, 2, 16, 12, 0.25, 0.3), moe(32, 4, 4)),
    layer(latent(2, 8, 8, 24, 32, 0.3, None, 777.0, yarn(40.0, 30, 20.0, 1.5)), moe(24, 3, 2)),
], scale=1.5)
CFG_D["layers"][0]["mixer"].pop("rot")

CONFIGS = {"A": CFG_A, "B": CFG_B, "C": CFG_C, "D": CFG_D}


# Sublayers read the stream unnormed, so scores grow with it: with the larger gain a model's attention is all but a
# choice of one key and the models amplify a rounding of their input a thousandfold, which float32 affords.  A choice of
# expert that turns under rounding spoils every later token that attends to it: the bfloat16 models' routers lean on
# biases that stand well apart (the float32 models and the router alone are tested on choices by the token).
GAIN = {"float32": 3.0, "bfloat16": 1.0}


def make_dir(tmp_path, name, dtype="float32", seed=0):
    """A model folder for configuration `name`: random weights N(0, 0.07) written by the engine's random-weights
    mode, norm weights (1 +) N(0, 0.1), and what sets the size of the queries (the weight of the maps' query norm, the
    latent layers' query projection) multiplied by GAIN[dtype] so that scores spread and single keys stand
    out.  The embedding is scaled up to a stream of order one."""
    gain = GAIN[dtype]
    import ai_engine_b200 as aie
    from safetensors import safe_open
    from safetensors.torch import save_file

    d = os.path.join(str(tmp_path), f"vatazen_{name}_{seed}_{gain}")
    if os.path.exists(os.path.join(d, "model.safetensors")):
        return d
    aie.write_random_model(aie.VatazenConfig.from_dict(CONFIGS[name]), d, seed=seed, std=0.07, norm_std=0.1)
    path = os.path.join(d, "model.safetensors")
    tensors = {}
    with safe_open(path, "pt") as f:
        for k in f.keys():
            t = f.get_tensor(k)
            if k.endswith("mix.q.norm") or (k.endswith("mix.q") and k[:-1] + "dkv" in f.keys()):
                t = (t.float() * gain).to(t.dtype)
            if dtype == "bfloat16" and k.endswith("mlp.router"):
                t = (t.float() * 0.03).to(t.dtype)
            if dtype == "bfloat16" and k.endswith("mlp.router.b"):
                order = torch.randperm(t.numel(), generator=torch.Generator().manual_seed(t.numel() + seed))
                t = (t.float() * 0.1 + 1.5 * order).to(t.dtype)
            if k in ("embed", "side.embed"):
                t = (t.float() * 10.0).to(t.dtype)
            tensors[k] = t.clone().contiguous()          # a copy: the file is written again below
    save_file(tensors, path)
    return d


_REFS = {}
CLEAR = 0.1      # a router's choice stands when its last chosen logit leads the first one left out by this much


def plain_logits(d, name, ids, dtype=torch.float64):
    """[len(ids), vocab] from the plain implementation, with the rows whose routing is clear (cached per folder and
    sequence)."""
    key = (d, tuple(ids), dtype)
    if key not in _REFS:
        margins = []
        logits = pv.forward(CONFIGS[name], read_tensors(d), ids, dtype=dtype, margins_out=margins)[0].to(torch.float64).numpy()
        m = torch.stack(margins).min(dim=0).values.double().numpy() if margins else np.full(len(ids), np.inf)
        ok = m >= CLEAR
        clear = np.array([bool(ok[max(0, i - AFTER):i + 1].all()) for i in range(len(ids))])
        _REFS[key] = Ref(logits, clear)
    return _REFS[key]
