"""The Semadra decoder in plain NumPy (float64), one function per mechanism, whole sequences recomputed from their first
token: no cache, no batches, keys and values of every token and head written out.  What the library computes is compared
with this.

A model is (config, weights): `config` is the config.json dictionary, `weights` maps tensor names to arrays.
"""
import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def rms_norm(x, eps, weight=None):
    """x / sqrt(mean(x^2) + eps) over the last axis, times `weight`."""
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if weight is None else y * weight


# ----------------------------------------------------------------------------- attention
def visible(n, mask):
    """[n, n] booleans: whether query i sees key j.  A window of `size` keys ends at the query; the first `keep_first` keys of
    the sequence stay visible behind it."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    see = j <= i
    if mask:
        see &= (i - j < mask["size"]) | (j < mask.get("keep_first", 0))
    return see


def softmax_attention(q, k, v, scale, mask):
    """q [n, H, d], k [n, G, d], v [n, G, e] -> [n, H, e]; query head h uses key/value head h // (H / G)."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    see, out = visible(n, mask), np.zeros((n, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        s = np.where(see, (q[:, h] @ k[:, g].T) * scale, -np.inf)
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (p / p.sum(axis=1, keepdims=True)) @ v[:, g]
    return out


def attention_mixer(h, w, m, pre, eps):
    """Grouped heads without positions; queries and keys normed over the whole projection; an element-wise output gate."""
    n, H, d = h.shape[0], m["heads"], m["dim"]
    G, e = m.get("kv_heads") or H, m.get("vdim") or d
    q = rms_norm(h @ w[pre + "q"].T, eps, w[pre + "q.norm"]).reshape(n, H, d)
    k = rms_norm(h @ w[pre + "k"].T, eps, w[pre + "k.norm"]).reshape(n, G, d)
    v = (h @ w[pre + "v"].T).reshape(n, G, e)
    o = softmax_attention(q, k, v, m["scale"], m.get("mask")).reshape(n, H * e)
    return (o * sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


def latent(h, w, pre, eps):
    """The normed latent that a layer keeps."""
    return rms_norm(h @ w[pre + "dkv"].T, eps, w[pre + "dkv.norm"])


def latent_attention_mixer(h, c, w, m, pre, eps):
    """Queries through a normed latent of their own, keys and values per head from the latent c (this layer's or another's)."""
    n, H, d = h.shape[0], m["heads"], m["dim"]
    e = m.get("vdim") or d
    q = (rms_norm(h @ w[pre + "dq"].T, eps, w[pre + "dq.norm"]) @ w[pre + "uq"].T).reshape(n, H, d)
    k, v = (c @ w[pre + "uk"].T).reshape(n, H, d), (c @ w[pre + "uv"].T).reshape(n, H, e)
    return softmax_attention(q, k, v, m["scale"], m.get("mask")).reshape(n, H * e) @ w[pre + "o"].T


# ----------------------------------------------------------------------------- feed-forwards
def gated_unit(h, w, pre):
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def route(z, top, groups=None, scale=1.0):
    """z [n, E] -> (chosen [n, top], weights [n, top]).  Scores are sigmoids; with `groups` {count, keep} only the experts of the
    `keep` groups whose two largest scores sum highest can be chosen; the weights are the chosen scores times `scale`."""
    s = sigmoid(z)
    allowed = s.copy()
    if groups:
        parts = s.reshape(s.shape[0], groups["count"], -1)
        worth = np.sort(parts, axis=2)[:, :, ::-1][:, :, :2].sum(axis=2)
        kept = np.argsort(-worth, axis=1, kind="stable")[:, :groups["keep"]]
        for t in range(s.shape[0]):
            out = np.ones(groups["count"], dtype=bool)
            out[kept[t]] = False
            allowed[t].reshape(groups["count"], -1)[out] = -np.inf
    chosen = np.argsort(-allowed, axis=1, kind="stable")[:, :top]
    return chosen, scale * np.take_along_axis(s, chosen, axis=1)


def moe_ffn(h, w, mlp, pre):
    """The weighted sum of the chosen experts' outputs, and a shared expert for every token."""
    r = mlp["router"]
    chosen, weight = route(h @ w[pre + "router"].T, r["top"], r.get("groups"), r.get("scale", 1.0))
    out = np.zeros_like(h)
    for e in range(r["experts"]):
        t, k = np.nonzero(chosen == e)
        if len(t):
            out[t] += weight[t, k][:, None] * gated_unit(h[t], w, f"{pre}e{e}.")
    if mlp.get("shared"):
        out += gated_unit(h, w, pre + "shared.")
    return out


# ----------------------------------------------------------------------------- the per-layer token input
def token_side(x, tokens, w, pre, layer, dim, eps):
    """What a layer adds for the token itself: its slice of the token's row of a second table, gated by the stream."""
    e = w["side.embed"][np.asarray(tokens), layer * dim:(layer + 1) * dim]
    y = (gelu_tanh(x @ w[pre + "side.gate"].T) * e) @ w[pre + "side.proj"].T
    return rms_norm(y, eps, w[pre + "side.norm"])


# ----------------------------------------------------------------------------- the model
def forward(cfg, w, tokens, return_layers=False):
    """Logits [n, vocab] of one sequence from its first token (and the residual stream after every layer)."""
    eps, mult, side = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0), cfg.get("token_side")
    x = w["embed"][np.asarray(tokens)] * cfg.get("embedding", {}).get("scale", 1.0)
    runs, kept = [], {}
    for i, L in enumerate(cfg["layers"]):
        pre, m, mlp = f"l{i}.", L["mixer"], L.get("mlp")
        if L["type"] == "attention":
            y = attention_mixer(x, w, m, pre + "mix.", eps)
        else:
            src = m.get("kv_from")
            kept[i] = latent(x, w, pre + "mix.", eps) if src is None else kept[src]
            y = latent_attention_mixer(x, kept[i], w, m, pre + "mix.", eps)
        x = x + mult * rms_norm(y, eps, 1.0 + w[pre + "norm1"])
        if mlp:
            y = gated_unit(x, w, pre + "mlp.") if mlp["kind"] == "dense" else moe_ffn(x, w, mlp, pre + "mlp.")
            x = x + mult * rms_norm(y, eps, 1.0 + w[pre + "norm2"])
        if side:
            x = x + mult * token_side(x, tokens, w, pre, i, side["dim"], eps)
        runs.append(x.copy())
    logits = rms_norm(x, eps, 1.0 + w["final.norm"]) @ w["embed"].T
    return (logits, np.stack(runs)) if return_layers else logits


def load(model_dir):
    """(config.json dictionary, name -> float64 array) of a model folder."""
    import json
    import os

    from plain_redenex import read_safetensors
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(model_dir, "model.safetensors"))


def closest_call(cfg, w, tokens):
    """The smallest distance, over the tokens and the routers, between a chosen score (or a kept group's worth) and the first left-out one."""
    side = cfg.get("token_side")
    least, seen = 1.0, []

    def watch(h, w_, mlp, pre, inner=moe_ffn):
        seen.append((sigmoid(h @ w_[pre + "router"].T), mlp["router"]))
        return inner(h, w_, mlp, pre)
    keep = globals()["moe_ffn"]
    globals()["moe_ffn"] = watch
    try:
        forward(cfg, w, tokens)
    finally:
        globals()["moe_ffn"] = keep
    for s, r in seen:
        groups = r.get("groups")
        if groups:
            parts = s.reshape(s.shape[0], groups["count"], -1)
            worth = np.sort(np.sort(parts, axis=2)[:, :, ::-1][:, :, :2].sum(axis=2), axis=1)[:, ::-1]
            if groups["keep"] < groups["count"]:
                least = min(least, float((worth[:, groups["keep"] - 1] - worth[:, groups["keep"]]).min()))
            order = np.argsort(-np.sort(parts, axis=2)[:, :, ::-1][:, :, :2].sum(axis=2), axis=1, kind="stable")[:, :groups["keep"]]
            s = np.stack([parts[t, order[t]].reshape(-1) for t in range(len(s))])
        if r["top"] < s.shape[1]:
            s = np.sort(s, axis=1)[:, ::-1]
            least = min(least, float((s[:, r["top"] - 1] - s[:, r["top"]]).min()))
    return least
