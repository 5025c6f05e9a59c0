"""The Sarizen decoder in plain NumPy (float64), one function per mechanism, whole sequences recomputed from their
first token: no cache, no state, no batches.  What the library computes is compared with this.

A model is (config, weights): `config` is the config.json dictionary, `weights` maps tensor names to arrays.
"""
import math

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rms_norm(x, eps, weight=None):
    """x / sqrt(mean(x^2) + eps) over the last axis, times `weight`."""
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if weight is None else y * weight


# ----------------------------------------------------------------------------- rotation
def yarn_frequencies(dims, base, scaling=None):
    """(frequency of every pair, what sine and cosine are multiplied by).  Without `scaling`: base^(-2i/dims) and 1."""
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    if not scaling:
        return f, 1.0
    factor, original = scaling["factor"], scaling["original"]

    def pair_that_turns(times):      # the (fractional) pair whose angle makes `times` turns over the original length
        return dims * math.log(original / (2.0 * math.pi * times)) / (2.0 * math.log(base))
    lo = max(math.floor(pair_that_turns(scaling["fast"])), 0)
    hi = min(math.ceil(pair_that_turns(scaling["slow"])), dims - 1)
    out = []
    for i in range(dims // 2):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f[i] / factor * r + f[i] * (1.0 - r))
    return np.array(out), 0.1 * math.log(factor) + 1.0


def rotate_neighbours(x, positions, freq, mult):
    """x [n, heads, 2 len(freq)]: dimensions 2i and 2i + 1 are turned by position * freq[i], sine and cosine times `mult`."""
    out = np.empty_like(x)
    for i, f in enumerate(freq):
        ang = np.asarray(positions, dtype=np.float64)[:, None] * f
        c, s = np.cos(ang) * mult, np.sin(ang) * mult
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


# ----------------------------------------------------------------------------- mixers
def window_softmax_attention(q, k, v, scale, window, sink):
    """q, k [n, H, d], v [n, H, e] from position 0; position i sees its last `window` keys (None: all); the denominator of
    head h also holds exp(sink[h]) (None: no such term).  -> [n, H, e]"""
    n, H = q.shape[:2]
    out = np.zeros((n, H, v.shape[2]))
    for h in range(H):
        for i in range(n):
            lo = 0 if window is None else max(0, i - window + 1)
            s = (k[lo:i + 1, h] @ q[i, h]) * scale
            top = s.max() if sink is None else max(s.max(), sink[h])
            p = np.exp(s - top)
            out[i, h] = (p / (p.sum() + (0.0 if sink is None else np.exp(sink[h] - top)))) @ v[lo:i + 1, h]
    return out


def latent_attention_mixer(h, w, m, pre, eps):
    """Keys and values per head from a shared normed latent, one rotated key part for all heads, a window, a sink, a gate a head."""
    n, H, d, rd, r = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    e = m.get("vdim") or d
    q = (h @ w[pre + "q"].T).reshape(n, H, d + rd)
    down = h @ w[pre + "dkv"].T
    c = rms_norm(down[:, :r], eps, w[pre + "dkv.norm"])
    freq, mult = yarn_frequencies(rd, m["rot"]["base"], m["rot"].get("scaling"))
    pos = np.arange(n)
    q_rot = rotate_neighbours(q[:, :, d:], pos, freq, mult)
    k_rot = rotate_neighbours(down[:, None, r:], pos, freq, mult)
    k = np.concatenate([(c @ w[pre + "uk"].T).reshape(n, H, d), np.repeat(k_rot, H, axis=1)], axis=2)
    v = (c @ w[pre + "uv"].T).reshape(n, H, e)
    mask = m.get("mask")
    o = window_softmax_attention(np.concatenate([q[:, :, :d], q_rot], axis=2), k, v, m["scale"], mask["size"] if mask else None, w[pre + "sink"])
    o = o * sigmoid(h @ w[pre + "g"].T)[:, :, None]
    return o.reshape(n, H * e) @ w[pre + "o"].T


def decayed_linear_attention(q, k, v, decay):
    """Per head S_t = decay_h S_(t-1) + k_t v_t^T and o_t = S_t^T q_t, S_0 = 0.  q, k [n, H, d], v [n, H, e] -> [n, H, e]"""
    n, H, d = q.shape
    out = np.zeros((n, H, v.shape[2]))
    for head in range(H):
        S = np.zeros((d, v.shape[2]))
        for t in range(n):
            S = decay[head] * S + np.outer(k[t, head], v[t, head])
            out[t, head] = S.T @ q[t, head]
    return out


def lightning_mixer(h, w, m, pre, eps):
    """silu projections, the decayed outer-product recurrence, one norm over all heads, a sigmoid gate per channel."""
    n, H, d = h.shape[0], m["heads"], m["dim"]
    e = m.get("vdim") or d
    q, k, v = (silu(h @ w[pre + s].T) for s in "qkv")
    o = decayed_linear_attention(q.reshape(n, H, d), k.reshape(n, H, d), v.reshape(n, H, e), np.asarray(m["decay"], dtype=np.float64))
    o = rms_norm(o.reshape(n, H * e), eps, w[pre + "norm"]) * sigmoid(h @ w[pre + "g"].T)
    return o @ w[pre + "o"].T


MIXERS = {"lightning": lightning_mixer, "latent_attention": latent_attention_mixer}


# ----------------------------------------------------------------------------- feed-forwards
def squared_relu_ffn(h, w, pre):
    return np.square(np.maximum(h @ w[pre + "up"].T, 0.0)) @ w[pre + "down"].T


def gated_expert(h, w, pre):
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def route(z, top):
    """z [n, E] -> (chosen [n, top], their scores [n, top]): the largest sigmoids, as they are."""
    s = sigmoid(z)
    chosen = np.argsort(-s, axis=1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, axis=1)


def moe_ffn(h, w, mlp, pre):
    """Every chosen expert reads its score times the token's input; a shared expert reads the input as it is."""
    chosen, weight = route(h @ w[pre + "router"].T, mlp["router"]["top"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(chosen[t], weight[t]):
            out[t] += gated_expert(a * h[t:t + 1], w, f"{pre}e{e}.")[0]
    if mlp.get("shared"):
        out += gated_expert(h, w, pre + "shared.")
    return out


# ----------------------------------------------------------------------------- the model
def forward(cfg, w, tokens, return_layers=False):
    """Logits [n, vocab] of one sequence from its first token (and the residual stream after every layer)."""
    eps = cfg["norm"]["eps"]
    x, runs = w["embed"][np.asarray(tokens)].copy(), []
    for i, L in enumerate(cfg["layers"]):
        pre, mlp = f"l{i}.", L.get("mlp")
        y = MIXERS[L["type"]](rms_norm(x, eps, w[pre + "norm1"]), w, L["mixer"], pre + "mix.", eps)
        if mlp:
            h2 = rms_norm(x, eps, w[pre + "norm2"])
            y = y + (squared_relu_ffn(h2, w, pre + "mlp.") if mlp["kind"] == "dense" else moe_ffn(h2, w, mlp, pre + "mlp."))
        x = x + y
        runs.append(x.copy())
    logits = rms_norm(x, eps, w["final.norm"]) @ w["head"].T * cfg.get("logit_scale", 1.0)
    return (logits, np.stack(runs)) if return_layers else logits


def closest_call(cfg, w, tokens):
    """The smallest distance, over the tokens and the routers, between the last chosen score and the first left-out one."""
    eps, least = cfg["norm"]["eps"], 1.0
    _, runs = forward(cfg, w, tokens, return_layers=True)
    before = np.concatenate([w["embed"][np.asarray(tokens)][None], runs[:-1]])
    for i, L in enumerate(cfg["layers"]):
        mlp = L.get("mlp")
        if not mlp or mlp["kind"] != "moe" or mlp["router"]["top"] == mlp["router"]["experts"]:
            continue
        s = sigmoid(rms_norm(before[i], eps, w[f"l{i}.norm2"]) @ w[f"l{i}.mlp.router"].T)
        s, top = np.sort(s, axis=1)[:, ::-1], mlp["router"]["top"]
        least = min(least, float((s[:, top - 1] - s[:, top]).min()))
    return least


def load(model_dir):
    """(config.json dictionary, name -> float64 array) of a model folder."""
    import json
    import os

    from plain_redenex import read_safetensors
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(model_dir, "model.safetensors"))
