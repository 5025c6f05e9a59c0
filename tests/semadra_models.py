"""Small Semadra configurations and model folders for the tests.

Weights are drawn so that nothing hides: norm weights stored around zero well away from it, query and key norm weights that make
decisive scores, gates away from one half, router matrices large enough for decisive scores, a token table of the size of the
stream.  The folders are written in bfloat16 (what a float32 engine widens exactly), so the plain implementation and the library
compute from the same numbers.
"""
import json
import os

import numpy as np
import torch


def attention(heads, kv_heads, dim, vdim, scale, size=None, keep=None):
    m = {"heads": heads, "dim": dim, "scale": scale}
    if kv_heads:
        m["kv_heads"] = kv_heads
    if vdim:
        m["vdim"] = vdim
    if size:
        m["mask"] = {"size": size, **({"keep_first": keep} if keep is not None else {})}
    return m


def latent(heads, dim, vdim, q_rank, kv_rank, scale, size=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}
    if vdim:
        m["vdim"] = vdim
    if size:
        m["mask"] = {"size": size}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def layer(mixer, mlp):
    return {"type": "latent_attention" if "kv_rank" in mixer else "attention", "mixer": mixer, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, groups=None, scale=None, shared=None):
    router = {"experts": experts, "top": top}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    if scale is not None:
        router["scale"] = scale
    return {"kind": "moe", "expert": {"ff": ff}, "router": router, **({"shared": {"ff": shared}} if shared else {})}


def model(vocab, width, eps, layers, side=None, scale=None, mult=None):
    out = {"architecture": "Semadra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if side:
        out["token_side"] = {"dim": side}
    if scale is not None:
        out["embedding"] = {"scale": scale}
    if mult is not None:
        out["residual_mult"] = mult
    return out


# Sizes differ in everything from layer to layer and between the models: one to nineteen query heads, one to all of them with a key
# head of their own; value heads narrower and wider than key heads; windows of one token, inside a page, of exactly a page, over
# several pages, and none; no kept tokens, a few, and more than a page of them (more than the window too); latents read by the next
# layer and by a later one, through other windows, heads and query latents than their own layer's; one to all of 1 to 48 experts in
# groups of one, of several and ungrouped; shared expert or none, dense and no feed-forward; with and without the token input.
CFG_A = model(173, 64, 1e-5, [
    layer(attention(4, 2, 16, 24, 0.3, 21, 5), moe(24, 8, 2, (4, 2), 1.5, 40)),
    layer(latent(4, 16, 24, 20, 40, 0.35, 30), dense(72)),
    layer(latent(9, 8, 12, 28, 40, 0.5, 64, kv_from=1), moe(16, 6, 3, (2, 1), 0.7)),
    layer(attention(6, 6, 24, 8, 0.25, 40, 70), None),
], side=12, scale=2.5, mult=0.4)
CFG_B = model(99, 50, 3e-4, [
    layer(latent(3, 10, None, 14, 12, 0.4, 1), moe(20, 3, 3, None, None, 18)),
    layer(attention(5, 1, 10, None, 0.4), dense(30)),
    layer(latent(5, 14, 6, 9, 12, 0.3, None, kv_from=0), moe(14, 1, 1)),
    layer(attention(3, 3, 7, 11, 0.5, 66), None),
])
CFG_C = model(120, 48, 1e-6, [
    layer(attention(16, 2, 8, 20, 0.3, 130, 64), moe(32, 48, 4, (8, 3), 2.5, 24)),
    layer(attention(1, 1, 24, 8, 0.3, 64, 1), moe(8, 9, 2, (9, 4))),
    layer(latent(19, 6, 10, 30, 48, 0.3, None), moe(12, 12, 2, (3, 2), 1.0, 8)),
    layer(latent(2, 12, 16, 24, 48, 0.3, 65, kv_from=2), dense(56)),
    layer(latent(1, 20, 9, 11, 33, 0.3, 77), None),
], side=7, scale=1.5, mult=0.35)
# sizes that the tensor-core kernels take: widths, latents and the token input in multiples of 8 and 16, heads of 64 and 96
CFG_D = model(144, 72, 1e-5, [
    layer(attention(6, 2, 64, 32, 0.12, 100, 10), moe(48, 4, 1, (2, 1), 1.3, 56)),
    layer(latent(3, 64, 64, 48, 64, 0.15, 90), dense(104)),
    layer(latent(20, 32, 32, 40, 64, 0.2, 140, kv_from=1), moe(24, 8, 2, (4, 2), 2.0, 16)),
    layer(attention(4, 4, 96, 96, 0.1, 64, 128), None),
], side=16, scale=3.0, mult=0.6)
CONFIGS = {"a": CFG_A, "b": CFG_B, "c": CFG_C, "d": CFG_D}


def tensors_for(cfg, seed):
    g = np.random.default_rng(seed)
    D, V, side = cfg["width"], cfg["vocab"], cfg.get("token_side")
    W = {}

    def mat(name, rows, cols, gain=1.0):
        W[name] = g.normal(0.0, gain / np.sqrt(cols), size=(rows, cols))

    def vec(name, n, lo, hi):
        W[name] = g.uniform(lo, hi, size=(n,))

    W["embed"] = g.normal(0.0, 0.7, size=(V, D))
    if side:
        W["side.embed"] = g.normal(0.0, 1.0, size=(V, side["dim"] * len(cfg["layers"])))
    for i, L in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", L["mixer"], L.get("mlp")
        vec(p + "norm1", D, -0.6, 0.5)
        H, d = m["heads"], m["dim"]
        e = m.get("vdim") or d
        if L["type"] == "attention":
            G = m.get("kv_heads") or H
            for s, n in (("q", H * d), ("k", G * d), ("v", G * e)):
                mat(p + "mix." + s, n, D, 1.5)
            vec(p + "mix.q.norm", H * d, 0.5, 2.5)
            vec(p + "mix.k.norm", G * d, 0.5, 2.5)
            mat(p + "mix.g", H * e, D, 2.0)
        else:
            r, qr = m["kv_rank"], m["q_rank"]
            mat(p + "mix.dq", qr, D, 2.0)
            vec(p + "mix.dq.norm", qr, 0.6, 1.4)
            mat(p + "mix.uq", H * d, qr, 1.5)
            if m.get("kv_from") is None:
                mat(p + "mix.dkv", r, D, 2.0)
                vec(p + "mix.dkv.norm", r, 0.6, 1.4)
            mat(p + "mix.uk", H * d, r, 1.5)
            mat(p + "mix.uv", H * e, r, 1.5)
        mat(p + "mix.o", D, H * e)
        if side:
            mat(p + "side.gate", side["dim"], D, 1.5)
            mat(p + "side.proj", D, side["dim"], 1.5)
            vec(p + "side.norm", D, 0.5, 1.5)
        if not mlp:
            continue
        vec(p + "norm2", D, -0.6, 0.5)
        if mlp["kind"] == "dense":
            for k, (rows, cols) in (("gate", (mlp["ff"], D)), ("up", (mlp["ff"], D)), ("down", (D, mlp["ff"]))):
                mat(p + "mlp." + k, rows, cols, 1.5)
            continue
        units = [(f"mlp.e{x}.", mlp["expert"]["ff"]) for x in range(mlp["router"]["experts"])]
        units += [("mlp.shared.", mlp["shared"]["ff"])] if mlp.get("shared") else []
        for name, ff in units:
            for k, (rows, cols) in (("gate", (ff, D)), ("up", (ff, D)), ("down", (D, ff))):
                mat(p + name + k, rows, cols, 1.5)
        mat(p + "mlp.router", mlp["router"]["experts"], D, 2.0)
    vec("final.norm", D, -0.5, 0.5)
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
    return [int(t) for t in np.random.default_rng(9000 + salt).integers(0, cfg["vocab"], size=n)]
