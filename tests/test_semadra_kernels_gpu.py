"""The kernels of the Semadra decoder's mechanisms, each alone against the plain implementation's function for the same mechanism
(tests/plain_semadra.py): the norm over the whole query and key projections with the cache append; attention through a window with
kept first keys and a gate per channel in every form (single tokens, pages split over blocks, tiles of a prompt, the tensor cores);
single tokens over shared latent rows on the tensor cores; the norms of both latents and the fetch of kept rows; small products per
head; the router that chooses inside the groups whose two best scores sum highest; the experts' sum with its norm; the norm added to
the residual stream; the gate of the token's own numbers."""
import numpy as np
import pytest
import torch

import plain_semadra as plain
from edgelm_b200.csrc import ops
from edgelm_b200.parts.rope import rotary_frequencies
from test_vosulorn_kernels_gpu import PagedKV, f32, i32, make_tiles, packed

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]


def rounder(dtype):
    return lambda a: torch.tensor(np.asarray(a), dtype=dtype).double().numpy()


def nan(*shape, dtype=torch.float32):
    return torch.full(shape, float("nan"), dtype=dtype, device=DEV)


def no_error():
    return torch.zeros(1, dtype=torch.int32, device=DEV)


# ----------------------------------------------------------------------------- the norm over the whole projection
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv,rot,interleaved,bias", [(4, 2, 16, 24, 0, False, False), (3, 1, 7, 11, 0, False, True), (8, 8, 64, 32, 0, False, False),
                                                            (6, 3, 20, 12, 8, True, True), (2, 2, 10, 6, 10, False, False), (19, 1, 64, 64, 0, False, True)])
def test_norm_over_the_whole_projection(H, G, dk, dv, rot, interleaved, bias, dtype):
    """Few and many tokens; rows that belong to a wider product; pieces of four values and single ones; with the rotation that other
    designs would put behind it."""
    for lengths in ([1, 1, 1], [70, 3, 64]):
        g = np.random.default_rng(dk + sum(lengths))
        eps, T = 1e-2, sum(lengths)
        width = (H + G) * dk + G * dv
        u, b = rounder(torch.float32)(g.normal(size=(T, width))), rounder(torch.float32)(g.normal(size=width)) if bias else np.zeros(width)
        u[1] *= 30.0
        qn, kn = rounder(torch.float32)(g.uniform(0.5, 2.0, H * dk)), rounder(torch.float32)(g.uniform(0.5, 2.0, G * dk))
        kv = PagedKV([n + 40 for n in lengths], G, dk, dv, dtype, seed=1)
        pos = np.concatenate([np.arange(37, 37 + n) for n in lengths])
        _, tok_seq = packed(lengths)
        q_want = plain.rms_norm(u[:, :H * dk] + b[:H * dk], eps, qn).reshape(T, H, dk)
        k_want = plain.rms_norm(u[:, H * dk:(H + G) * dk] + b[H * dk:(H + G) * dk], eps, kn).reshape(T, G, dk)
        freq = None
        if rot:
            freq = rotary_frequencies(rot, 100.0).to(DEV)
            from plain_sarizen import rotate_neighbours
            order = np.arange(rot) if interleaved else np.stack([np.arange(rot // 2), np.arange(rot // 2) + rot // 2], 1).reshape(-1)
            for x in (q_want, k_want):
                x[..., order] = rotate_neighbours(x[..., order], pos, 100.0 ** (-2.0 * np.arange(rot // 2) / rot), 1.0)
        wide = nan(T, width + 3)
        wide[:, :width] = f32(u)
        for rows in (f32(u), wide[:, :width]):
            q, err = nan(T, H * dk), no_error()
            ops.norm_append(rows, f32(b) if bias else None, q, i32(pos), tok_seq, i32(kv.table), kv.k, kv.v, H, G, dk, dv, rot, interleaved, freq, err, f32(qn), f32(kn), eps)
            assert int(err.item()) == 0 and np.abs(q.cpu().numpy() - q_want.reshape(T, -1)).max() < 2e-5
            tol = 2e-5 if dtype == torch.float32 else 2e-2
            for t, (s, p) in enumerate(zip(tok_seq.cpu().numpy(), pos)):
                page = kv.table[s, p // 64]
                assert np.abs(kv.k[page, :, p % 64].float().cpu().numpy() - k_want[t]).max() < tol
                v = (u[t] + b)[(H + G) * dk:].reshape(G, dv)
                assert np.abs(kv.v[page, :, p % 64].float().cpu().numpy() - v).max() < tol * max(1.0, np.abs(v).max())


# ----------------------------------------------------------------------------- windows with kept first keys
def gated(o, gate):
    return (o * plain.sigmoid(gate).reshape(o.shape)).reshape(o.shape[0], -1)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv,size,keep", [
    (4, 2, 16, 24, 21, 5), (3, 3, 10, 14, 70, 3), (8, 1, 64, 32, 40, 100), (4, 4, 64, 64, 64, 64), (6, 2, 96, 64, 100, 1), (2, 1, 128, 128, 1, 65),
    (9, 3, 64, 48, 130, 64), (2, 2, 32, 32, 65, 130), (1, 1, 72, 104, 33, 2), (12, 1, 40, 8, 2, 63), (4, 2, 64, 16, 50, 0)])
def test_attention_with_kept_first_keys_and_a_gate(H, G, dk, dv, size, keep, dtype):
    """Every form against the plain attention, over scrambled pages: single tokens (keys split over blocks or not, in both kernels),
    prompts whole and in pieces, on the CUDA cores and on the tensor cores, from pages and from a step's own rows.  Two keys of every
    sequence stand out for every query, the last kept one and the first one behind: where they are seen, or not, decides."""
    g = np.random.default_rng(dk + size)
    lengths, scale = [200, 67, 1, keep + size + 70], 0.9 / np.sqrt(dk)
    rnd, kv = rounder(dtype), PagedKV([200, 67, 1, keep + size + 70], G, dk, dv, dtype, seed=3)
    mask = {"size": size, "keep_first": keep}
    Q, K, V, gates, want, bare = [], [], [], [], [], []
    for s, n in enumerate(lengths):
        q, k, v = g.normal(size=(n, H, dk)), rnd(g.normal(size=(n, G, dk))), rnd(g.normal(size=(n, G, dv)))
        for at in (keep - 1, keep):
            if 0 <= at < n:
                k[at] = rnd(k[at] * 12.0 / np.sqrt(dk))
                q += 0.35 * np.repeat(k[at], H // G, axis=0)[None]
        q, gate = rounder(torch.float32)(q), rounder(torch.float32)(2.0 * g.normal(size=(n, H * dv)))
        kv.put(s, k, v)
        o = plain.softmax_attention(q, k, v, scale, mask)
        for lst, x in ((Q, q), (K, k), (V, v), (gates, gate), (want, gated(o, gate)), (bare, o.reshape(n, -1))):
            lst.append(x)
    # (the edges matter: with one kept key less or one more the plain attention is another)
    n = lengths[3]
    for other in ({"size": size, "keep_first": keep + 1}, *([{"size": size, "keep_first": keep - 1}] if keep else [])):
        moved = np.abs(plain.softmax_attention(Q[3], K[3], V[3], scale, other).reshape(n, -1) - bare[3]).max(axis=1)
        assert moved[-1] > 0.05 * np.abs(bare[3]).max()
    table, tol = i32(kv.table), 3e-5 if dtype == torch.float32 else 2e-2
    args = (scale, ops.MASK_WINDOW, size, None)

    def check(got, ref, what):
        assert np.abs(got.float().cpu().numpy() - ref).max() < tol * max(1.0, np.abs(ref).max()), what
    wide = lambda rows: torch.cat([f32(rows), nan(len(rows), 3)], 1)[:, :H * dv]       # (the gate's columns in a wider product)
    for pieces in ([(0, n) for n in lengths], [(n // 3, n - n // 3) for n in lengths]):
        live = [(s, a, n) for s, (a, n) in enumerate(pieces) if n]
        q = f32(np.concatenate([Q[s][a:a + n].reshape(n, H * dk) for s, a, n in live]))
        gate = wide(np.concatenate([gates[s][a:a + n] for s, a, n in live]))
        ref, ref0 = (np.concatenate([w[s][a:a + n] for s, a, n in live]) for w in (want, bare))
        tb, n_new, first = table[[s for s, _, _ in live]].contiguous(), [n for _, _, n in live], [a for _, a, _ in live]
        tile = max(1, 32 // (H // G))
        tseq, ttok0, tntok, tpos0, count = make_tiles(n_new, first, tile)
        for gt, rf in ((gate, ref), (None, ref0)):
            out = nan(q.shape[0], H * dv, dtype=dtype)
            ops.masked_attn_tiled(q, out, kv.k, kv.v, tb, tseq, ttok0, tntok, tpos0, count, tile, H, G, dk, dv, *args, gate=gt, keep=keep)
            check(out, rf, ("tiled", pieces[0]))
        forms = ["pages"] + (["own rows"] if not any(first) else [])
        kx, vx = (torch.tensor(np.concatenate([x[s].reshape(lengths[s], -1) for s, _, _ in live]), dtype=dtype, device=DEV) for x in (K, V))
        for form in forms:
            src = (kv.k, kv.v, tb) if form == "pages" else (kx, vx, None)
            out = nan(q.shape[0], H * dv, dtype=dtype)
            ops.masked_attn_tiled(q, out, *src, tseq, ttok0, tntok, tpos0, count, tile, H, G, dk, dv, *args, gate=gate, keep=keep)
            check(out, ref, ("tiled", form))
            if not ops.attn_prefill_split_takes(dtype, dk, dv):
                continue
            stile = make_tiles(n_new, first, ops.SPLIT_PREFILL_TILE)
            for most in (64, 4000):      # (one warp group a tile, and two that share its pages)
                out = nan(q.shape[0], H * dv, dtype=dtype)
                ops.attn_prefill_split(q, out, *src, *stile, H, G, dk, dv, scale, gate=gate, max_keys=most, mask=ops.MASK_WINDOW, mask_size=size, keep=keep)
                check(out, ref, ("tensor cores", form, most))
    for back in (0, 1, 2, 63, 65):
        live = [(s, n - 1 - back) for s, n in enumerate(lengths) if n - 1 - back >= 0]
        q, gate = f32(np.stack([Q[s][p].reshape(H * dk) for s, p in live])), wide(np.stack([gates[s][p] for s, p in live]))
        ref, B = np.stack([want[s][p] for s, p in live]), len(live)
        tb, pos, idx = table[[s for s, _ in live]].contiguous(), i32([p for _, p in live]), torch.arange(B, dtype=torch.int32, device=DEV)
        for splits in (1, 2, 5):
            part = nan(B * H * splits * (2 + dv))
            out = nan(B, H * dv, dtype=dtype)
            ops.masked_attn(q, out, kv.k, kv.v, pos, idx, tb, H, G, dk, dv, *args, size + keep, gate=gate, n_splits=splits, part=part, keep=keep)
            check(out, ref, ("single", back, splits))
            out = nan(B, H * dv, dtype=dtype)
            ops.masked_attn_tiled(q, out, kv.k, kv.v, tb, idx, idx, torch.ones_like(idx), pos, B, 1, H, G, dk, dv, *args, n_splits=splits, part=part, gate=gate, keep=keep)
            check(out, ref, ("single as tiles", back, splits))


@pytest.mark.parametrize("kind,size", [("causal", 0), ("window", 90), ("chunk", 70)])
@pytest.mark.parametrize("H,G,dk,dv", [(4, 2, 64, 64), (3, 3, 128, 72), (6, 1, 104, 128), (2, 2, 24, 8)])
def test_single_tokens_whole_rows_at_a_time(H, G, dk, dv, kind, size):
    """The bfloat16 kernel that reads whole key and value rows, under the other masks, with sinks and gates per head."""
    g = np.random.default_rng(dk)
    lengths, scale, rnd = [300, 65, 2, 1], 0.2, rounder(torch.bfloat16)
    kv = PagedKV(lengths, G, dk, dv, torch.bfloat16, seed=6)
    sink, gate = rounder(torch.float32)(g.uniform(-1, 3, H)), rounder(torch.float32)(g.normal(size=(4, H)))
    q, ref = rounder(torch.float32)(g.normal(size=(4, H, dk))), []
    for s, n in enumerate(lengths):
        k, v = rnd(g.normal(size=(n, G, dk))), rnd(g.normal(size=(n, G, dv)))
        kv.put(s, k, v)
        lo = {"causal": 0, "window": max(0, n - size), "chunk": (n - 1) // size * size if size else 0}[kind]
        row = []
        for h in range(H):
            sc = k[lo:, h // (H // G)] @ q[s, h] * scale
            top = max(sc.max(), sink[h])
            p = np.exp(sc - top)
            row.append((p / (p.sum() + np.exp(sink[h] - top))) @ v[lo:, h // (H // G)] * plain.sigmoid(gate[s, h]))
        ref.append(np.concatenate(row))
    mk = {"causal": ops.MASK_CAUSAL, "window": ops.MASK_WINDOW, "chunk": ops.MASK_CHUNK}[kind]
    for splits in (1, 3):
        out, part = nan(4, H * dv, dtype=torch.bfloat16), nan(4 * H * splits * (2 + dv))
        ops.masked_attn(f32(q.reshape(4, -1)), out, kv.k, kv.v, i32([n - 1 for n in lengths]), i32(range(4)), i32(kv.table), H, G, dk, dv, scale, mk, size, f32(sink),
                        size or 1 << 30, gate=f32(gate), n_splits=splits, part=part)
        assert np.abs(out.float().cpu().numpy() - np.array(ref)).max() < 8e-3 * max(1.0, np.abs(ref).max())


# ----------------------------------------------------------------------------- latents
@pytest.mark.parametrize("H,dc,dv,kind,size,keep", [(4, 48, 48, "window", 30, 0), (32, 512, 512, "window", 100, 0), (19, 64, 64, "causal", 0, 0), (16, 96, 80, "chunk", 70, 0),
                                                    (40, 128, 112, "window", 64, 70), (1, 16, 16, "window", 1, 0), (33, 576, 512, "causal", 0, 0), (9, 272, 256, "window", 65, 3)])
def test_single_tokens_over_latent_rows(H, dc, dv, kind, size, keep):
    """Rows that are key and value at once on the tensor cores: float32 scores and weights (the difference to the exact attention of the
    same bfloat16 rows is float32 rounding), under every mask, splits of every number, one row standing out."""
    g = np.random.default_rng(dc + H)
    assert ops.latent_decode_takes(torch.bfloat16, H, dc, dv) in (16, 32) and ops.latent_decode_takes(torch.float32, H, dc, dv) == 0
    lengths, scale, rnd = [260, 64, 65, 1, 30], 2.0 / np.sqrt(dc), rounder(torch.bfloat16)
    kv = PagedKV(lengths, 1, dc, dc, torch.bfloat16, seed=8, values_in_keys=True)
    q, sink, gate = rounder(torch.float32)(g.normal(size=(5, H, dc))), rounder(torch.float32)(g.uniform(-1, 3, H)), rounder(torch.float32)(g.normal(size=(5, H)))
    ref = []
    for s, n in enumerate(lengths):
        k = rnd(g.normal(size=(n, 1, dc)))
        k[n // 2] = rnd(3.0 * k[n // 2])
        kv.put(s, k)
        i = np.arange(n)
        see = {"causal": i >= 0, "window": (i > n - 1 - size) | (i < keep), "chunk": i // size == (n - 1) // size if size else i >= 0}[kind]
        sc = np.where(see[:, None], k[:, 0] @ q[s].T * scale, -np.inf)
        top = np.maximum(sc.max(0), sink)
        p = np.exp(sc - top)
        ref.append(((p / (p.sum(0) + np.exp(sink - top))).T @ k[:, 0, :dv] * plain.sigmoid(gate[s])[:, None]).reshape(-1))
    mk = {"causal": ops.MASK_CAUSAL, "window": ops.MASK_WINDOW, "chunk": ops.MASK_CHUNK}[kind]
    for splits in (1, 2, 4, 7):
        out, part = nan(5, H * dv), nan(5 * H * splits * (2 + dv))
        ops.latent_decode(f32(q.reshape(5, -1)), out, kv.k, i32([n - 1 for n in lengths]), i32(range(5)), i32(kv.table), H, dc, dv, scale, mk, size, f32(sink), splits, part,
                          gate=f32(gate), keep=keep)
        assert np.abs(out.cpu().numpy() - np.array(ref)).max() < 2e-5 * max(1.0, np.abs(ref).max()), splits


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [1, 7, 16, 17, 90])
@pytest.mark.parametrize("H,K,N", [(4, 64, 512), (9, 512, 64), (3, 40, 24), (2, 8, 17), (5, 136, 33), (1, 10, 6)])
def test_small_products_per_head(T, H, K, N, dtype):
    g = np.random.default_rng(K + N + T)
    a, w = rounder(torch.float32)(g.normal(size=(T, H * (K + 8)))), rounder(dtype)(g.normal(size=(H, N, K)))
    ref = np.stack([a[:, h * (K + 8):h * (K + 8) + K] @ w[h].T for h in range(H)], 1)
    for out_dtype in {torch.float32, dtype}:
        out = nan(T, H * (N + 3), dtype=out_dtype)
        ops.head_matmul(f32(a), K + 8, torch.tensor(w, dtype=dtype, device=DEV), out, N + 3)
        got = out.float().cpu().numpy().reshape(T, H, N + 3)
        assert np.abs(got[..., :N] - ref).max() < (2e-6 if out_dtype == torch.float32 else 5e-3) * np.abs(ref).max() and np.isnan(got[..., N:]).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,qr,r", [(3, 24, 40), (100, 128, 48), (1, 9, 33), (70, 300, 16)])
def test_norms_of_both_latents_and_kept_rows(T, qr, r, dtype):
    """Both norms and the append from one product's columns; a reader's norm alone; the rows fetched back as another layer reads them."""
    g = np.random.default_rng(T + qr)
    u, qw, kw = rounder(torch.float32)(g.normal(size=(T, qr + r))), rounder(torch.float32)(g.uniform(0.5, 1.5, qr)), rounder(torch.float32)(g.uniform(0.5, 1.5, r))
    eps, tol = 1e-2, 2e-6 if dtype == torch.float32 else 1.6e-2
    kv = PagedKV([T + 30], 1, r, r, dtype, seed=4, values_in_keys=True)
    pos, seq, table, err = i32(np.arange(30, 30 + T)), i32([0] * T), i32(kv.table), no_error()
    cq, rows, back = nan(T, qr, dtype=dtype), nan(T, r, dtype=dtype), nan(T, r, dtype=dtype)
    ops.latent_prepare(f32(u), qr, True, None, 0, 0, False, f32(kw), eps, pos, seq, table, kv.k, 0, 8, 0, r, None, err, row_out=rows, q_latent=(0, f32(qw), cq))
    want_q, want_c = plain.rms_norm(u[:, :qr], eps, qw), plain.rms_norm(u[:, qr:], eps, kw)
    assert np.abs(cq.float().cpu().numpy() - want_q).max() < tol * np.abs(want_q).max() and np.abs(rows.float().cpu().numpy() - want_c).max() < tol * np.abs(want_c).max()
    ops.latent_rows(kv.k, back, pos, seq, table, err)
    assert torch.equal(back, rows)
    alone = nan(T, qr, dtype=dtype)
    ops.latent_prepare(f32(u), qr, False, None, 0, 0, False, None, eps, pos, seq, None, None, 0, 8, 0, r, None, err, q_latent=(0, f32(qw), alone))
    assert torch.equal(alone, cq) and int(err.item()) == 0


# ----------------------------------------------------------------------------- experts
@pytest.mark.parametrize("T", [5, 120])
@pytest.mark.parametrize("E,top,count,keep", [(8, 2, 4, 2), (16, 3, 4, 3), (6, 3, 2, 1), (9, 2, 9, 4), (12, 2, 3, 2), (96, 6, 48, 5), (300, 8, 100, 3), (10, 10, 1, 1), (40, 4, 5, 5)])
def test_router_chooses_inside_the_best_groups(E, top, count, keep, T):
    """A group's worth is the sum of its two largest sigmoids (of its only one in groups of one); the weights are the scores times the
    constant.  Groups whose best single score is largest often are not the ones whose two best sum highest."""
    g = np.random.default_rng(E + top)
    D = 1040 if E < 20 else 56
    h, wr = rounder(torch.float32)(g.normal(size=(T, D))), rounder(torch.float32)(2.0 * g.normal(size=(E, D)) / np.sqrt(D))
    groups = {"count": count, "keep": keep}
    z = h @ wr.T
    chosen, wts = plain.route(z, top, groups, 1.7)
    idx, got = torch.empty(T, top, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV)
    ops.moe_route_scored(f32(h), f32(wr), None, idx, got, top, E, count, keep, 1.7, score="sigmoid", renormalize=False, group_score="top2_sum")
    s = plain.sigmoid(z).reshape(T, count, -1)
    worth = np.sort(np.sort(s, 2)[:, :, ::-1][:, :, :2].sum(2), 1)
    clear = (np.diff(worth, axis=1).min(1) > 1e-5) if count > 1 else np.ones(T, bool)
    clear &= np.diff(np.sort(plain.sigmoid(z), 1), axis=1).min(1) > 1e-6 if E < 20 else True
    assert clear.any()
    assert np.array_equal(idx.cpu().numpy()[clear], chosen[clear]) or (E >= 20 and (idx.cpu().numpy() == chosen)[clear].mean() > 0.99)
    same = clear[:, None] & (idx.cpu().numpy() == chosen)
    assert np.abs(got.cpu().numpy() - wts)[same].max() < 2e-6
    if 1 < keep < count and E // count > 1 and T > 100:
        by_best = np.argsort(-s.max(2), axis=1)[:, :keep]
        by_two = np.argsort(-np.sort(s, 2)[:, :, ::-1][:, :, :2].sum(2), axis=1)[:, :keep]
        assert (np.sort(by_best, 1) != np.sort(by_two, 1)).any()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,D,top,with_shared", [(3, 64, 2, True), (100, 50, 3, True), (70, 2048, 1, False), (9, 4100, 4, True), (2, 3, 1, False), (5, 16500, 2, True)])
def test_experts_sum_with_its_norm(T, D, top, with_shared, dtype):
    g = np.random.default_rng(D)
    rows = T * top + 5
    y, wts, shared, x, w = (rounder(torch.float32)(a) for a in (g.normal(size=(rows, D)), g.uniform(0.2, 2.0, (T, top)), g.normal(size=(T, D)), g.normal(size=(T, D)), g.uniform(0.5, 1.5, D)))
    pair_row = g.permutation(rows)[:T * top]
    sums = (wts[:, :, None] * y[pair_row].reshape(T, top, D)).sum(1) + (shared if with_shared else 0.0)
    want = x + plain.rms_norm(sums, 1e-3, w)
    xd, cast = f32(x), nan(T, D, dtype=dtype)
    ops.moe_combine_norm(xd, f32(y), f32(wts), i32(pair_row), f32(w), 1e-3, shared=f32(shared) if with_shared else None, cast=cast)
    assert np.abs(xd.cpu().numpy() - want).max() < 1e-5 and torch.equal(cast, xd.to(dtype))
    xd = f32(x)
    ops.moe_combine_norm(xd, f32(y), None, i32(pair_row), f32(w), 1e-3, top=top)
    assert np.abs(xd.cpu().numpy() - (x + plain.rms_norm(y[pair_row].reshape(T, top, D).sum(1), 1e-3, w))).max() < 1e-5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,D", [(1, 64), (3, 50), (100, 576), (70, 2048), (8, 4096), (65, 9000), (2, 16388), (4, 6)])
def test_a_norm_added_to_the_stream(T, D, dtype):
    g = np.random.default_rng(D)
    x, y1, y2, w = (rounder(torch.float32)(g.normal(size=s)) for s in ((T, D), (T, D), (T, D), (D,)))
    for a, b in ((1.0, None), (0.7, 1.3)):
        xd, cast = f32(x), nan(T, D, dtype=dtype)
        ops.rmsnorm_add(xd, f32(y1), f32(w), 1e-2, a=a, y2=f32(y2) if b else None, b=b or 0.0, cast=cast)
        want = x + plain.rms_norm(a * y1 + (b or 0.0) * y2, 1e-2, w)
        assert np.abs(xd.cpu().numpy() - want).max() < 2e-5 and torch.equal(cast, xd.to(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,n", [(1, 7), (9, 64), (300, 24)])
def test_the_gate_of_a_tokens_own_numbers(T, n, dtype):
    g = np.random.default_rng(n)
    u, table, ids = rounder(torch.float32)(3.0 * g.normal(size=(T, n))), rounder(dtype)(g.normal(size=(50, n))), g.integers(0, 50, T)
    out, err = nan(T, n, dtype=dtype), no_error()
    ops.token_gate(f32(u), i32(ids), torch.tensor(table, dtype=dtype, device=DEV), out, err)
    want = plain.gelu_tanh(u) * table[ids]
    assert np.abs(out.float().cpu().numpy() - want).max() < (2e-6 if dtype == torch.float32 else 5e-3) * np.abs(want).max() and int(err.item()) == 0
    ids[0] = 50
    ops.token_gate(f32(u), i32(ids), torch.tensor(table, dtype=dtype, device=DEV), out, err)
    assert int(err.item()) == 1 and (out[0] == 0).all()
