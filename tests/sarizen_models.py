"""Small Sarizen configurations and model folders for the tests.

Weights are drawn so that nothing hides: decays from 0.3 to 1 (a state remembers a few tokens in one head and hundreds in
another), sinks from well under to well over a usual score, gates away from one half, router matrices large enough for decisive
scores away from 0 and 1 (so that a weight on the output, which passes the gated unit unsquared, differs from one on the input).
The folders are written in bfloat16 (what a float32 engine widens exactly), so the plain implementation and the library compute
from the same numbers.
"""
import json
import os

import numpy as np
import torch


def lightning(heads, dim, vdim, decay):
    assert len(decay) == heads
    m = {"heads": heads, "dim": dim, "decay": list(decay)}
    if vdim:
        m["vdim"] = vdim
    return m


def latent(heads, dim, rot_dim, vdim, rank, base, scaling, scale, window):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "kv_rank": rank, "scale": scale, "rot": {"base": base, "dims": rot_dim}}
    if vdim:
        m["vdim"] = vdim
    if scaling:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if window:
        m["mask"] = {"size": window}
    return m


def layer(mixer, mlp):
    return {"type": "lightning" if "decay" in mixer else "latent_attention", "mixer": mixer, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, shared):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


# Sizes differ in everything from layer to layer and between the models: one to sixteen heads (from eight on decoding stages a
# latent's row once for all of them and splits pages); value heads narrower and wider than key heads; key sizes of the linear
# attention under, at and over a warp's 32 lanes; latents from 12 to 96; 2 to 16 rotated dimensions, stretched (the ramp inside,
# before and behind the pairs) or not; windows of one token, inside a page, of exactly a page, over several pages, and none; one to
# all of 1 to 40 experts; shared expert or none; dense and no feed-forward; widths that are no multiple of 8.
CFG_A = {"architecture": "Sarizen", "vocab": 171, "width": 64, "norm": {"eps": 1e-5}, "logit_scale": 0.7, "layers": [
    layer(latent(4, 16, 8, 24, 40, 700.0, (3.0, 48, 6.0, 0.5), 0.35, 21), moe(24, 6, 2, 32)),
    layer(lightning(3, 24, 40, (0.3, 0.9, 0.998)), dense(72)),
    layer(latent(8, 8, 4, 8, 24, 90.0, (6.0, 200, 9.0, 1.5), 0.5, 64), moe(16, 5, 1, 40)),
    layer(lightning(2, 40, 16, (1.0, 0.95)), moe(40, 7, 3, None)),
]}
CFG_B = {"architecture": "Sarizen", "vocab": 97, "width": 50, "norm": {"eps": 3e-4}, "layers": [
    layer(lightning(5, 10, 6, (0.99, 0.9, 0.7, 0.4, 0.995)), moe(20, 3, 3, 18)),
    layer(latent(3, 10, 6, 14, 12, 50.0, None, 0.4, 1), dense(30)),
    layer(latent(5, 12, 2, None, 30, 4000.0, (2.0, 30, 3.0, 0.2), 0.3, None), None),
    layer(lightning(1, 72, 8, (0.97,)), moe(14, 1, 1, None)),
]}
CFG_C = {"architecture": "Sarizen", "vocab": 120, "width": 48, "norm": {"eps": 1e-6}, "logit_scale": 3.0, "layers": [
    layer(lightning(2, 32, None, (0.85, 0.99)), None),
    layer(latent(16, 6, 10, 20, 18, 3000.0, (5.0, 4, 2.0, 1.0), 0.45, 130), moe(32, 40, 4, 24)),
    layer(latent(1, 24, 16, 8, 36, 100.0, (1.0, 500, 20.0, 2.0), 0.25, 65), moe(8, 9, 2, None)),
]}
# sizes that the tensor-core kernels take: widths and latents that are multiples of 8, prompt attention with key heads of 96, 64 and
# 128 over value heads of 64, 32 and 128, the chunked linear attention reading 16 bytes at a time
CFG_D = {"architecture": "Sarizen", "vocab": 144, "width": 72, "norm": {"eps": 1e-5}, "logit_scale": 1.6, "layers": [
    layer(latent(3, 48, 48, 64, 64, 2500.0, (4.0, 96, 8.0, 1.0), 0.15, 100), moe(48, 4, 1, 56)),
    layer(lightning(2, 64, 32, (0.93, 0.997)), dense(104)),
    layer(latent(5, 48, 16, 32, 96, 800.0, (2.5, 64, 4.0, 0.5), 0.2, None), moe(24, 6, 2, 16)),
    layer(latent(2, 96, 32, 128, 48, 60.0, None, 0.11, 64), None),
]}
CONFIGS = {"a": CFG_A, "b": CFG_B, "c": CFG_C, "d": CFG_D}


def tensors_for(cfg, seed):
    g = np.random.default_rng(seed)
    D, V = cfg["width"], cfg["vocab"]
    W = {}

    def mat(name, rows, cols, gain=1.0):
        W[name] = g.normal(0.0, gain / np.sqrt(cols), size=(rows, cols))

    def vec(name, n, lo, hi):
        W[name] = g.uniform(lo, hi, size=(n,))

    W["embed"] = g.normal(0.0, 0.7, size=(V, D))
    for i, L in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", L["mixer"], L.get("mlp")
        vec(p + "norm1", D, 0.6, 1.4)
        H, d = m["heads"], m["dim"]
        e = m.get("vdim") or d
        if L["type"] == "lightning":
            for s, n in (("q", H * d), ("k", H * d), ("v", H * e)):
                mat(p + "mix." + s, n, D, 1.5)
            mat(p + "mix.g", H * e, D, 2.0)
            vec(p + "mix.norm", H * e, 0.5, 1.5)
        else:
            r, rd = m["kv_rank"], m["rot_dim"]
            mat(p + "mix.q", H * (d + rd), D, 2.0)
            mat(p + "mix.dkv", r + rd, D, 2.0)
            vec(p + "mix.dkv.norm", r, 0.6, 1.4)
            mat(p + "mix.uk", H * d, r, 1.5)
            mat(p + "mix.uv", H * e, r, 1.5)
            vec(p + "mix.sink", H, -1.0, 3.0)
            mat(p + "mix.g", H, D, 2.0)
        mat(p + "mix.o", D, H * e)
        if not mlp:
            continue
        vec(p + "norm2", D, 0.6, 1.4)
        if mlp["kind"] == "dense":
            mat(p + "mlp.up", mlp["ff"], D, 1.2)
            mat(p + "mlp.down", D, mlp["ff"])
            continue
        ff = mlp["expert"]["ff"]
        for x in range(mlp["router"]["experts"]):
            mat(f"{p}mlp.e{x}.gate", ff, D, 2.5)
            mat(f"{p}mlp.e{x}.up", ff, D, 2.5)
            mat(f"{p}mlp.e{x}.down", D, ff)
        mat(p + "mlp.router", mlp["router"]["experts"], D, 2.0)
        if mlp.get("shared"):
            sf = mlp["shared"]["ff"]
            mat(p + "mlp.shared.gate", sf, D, 1.5)
            mat(p + "mlp.shared.up", sf, D, 1.5)
            mat(p + "mlp.shared.down", D, sf)
    vec("final.norm", D, 0.6, 1.4)
    mat("head", V, D, 1.5)
    return W


def write_dir(path, cfg, seed, overrides=None):
    """config.json and model.safetensors (bfloat16) for `cfg`; `overrides`: name -> array put in place of the drawn one."""
    from edgelm_b200.weights import write_file
    os.makedirs(path, exist_ok=True)
    W = tensors_for(cfg, seed)
    for k, v in (overrides or {}).items():
        assert k in W and np.shape(v) == W[k].shape, k
        W[k] = np.asarray(v)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_file(os.path.join(path, "model.safetensors"), {k: torch.tensor(v, dtype=torch.float32).to(torch.bfloat16) for k, v in W.items()})
    return path


def tokens(cfg, n, salt):
    return [int(t) for t in np.random.default_rng(7000 + salt).integers(0, cfg["vocab"], size=n)]
