"""The kernels of the Sarizen decoder's mechanisms, each alone against the plain implementation's function for the same mechanism
(tests/plain_sarizen.py): the stretched rotation of neighbouring pairs far into a sequence; latent attention with a window, a sink
and a gate in every form (single tokens, tiles of a prompt, pages split over blocks, the step's own keys on the CUDA cores and on
the tensor cores); prompt attention on the tensor cores under every mask over the cache's pages; the router of sigmoids; weights
on the experts' inputs; the squared ReLU in every product that has it; the linear attention over steps."""
import types

import numpy as np
import pytest
import torch

import plain_sarizen as plain
from edgelm_b200.csrc import ops
from edgelm_b200.parts import linear
from edgelm_b200.parts.rope import rotary_frequencies, rotary_magnitude
from test_vosulorn_kernels_gpu import PagedKV, f32, i32, make_tiles, packed

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def rounder(dtype):
    return lambda a: torch.tensor(np.asarray(a), dtype=dtype).double().numpy()


# ----------------------------------------------------------------------------- rotation and latent attention
@pytest.mark.parametrize("scaling", [None, {"factor": 6.0, "original": 300, "fast": 8.0, "slow": 1.0}])
@pytest.mark.parametrize("interleaved", [True, False])
def test_rotation_far_into_a_sequence(scaling, interleaved):
    """Queries, the shared key part and the latent's norm at positions up to 90,000: float32 angles alone would be off by more than
    the tolerance there."""
    H, d, rd, r, base, eps = 3, 10, 12, 20, 1000.0, 1e-5
    g = np.random.default_rng(4)
    pos = np.array([0, 1, 63, 64, 1000, 4097, 30001, 90000])
    T = len(pos)
    u = rounder(torch.float32)(g.normal(size=(T, H * (d + rd) + r + rd)))
    nw = rounder(torch.float32)(g.uniform(0.5, 1.5, r))
    f, mult = plain.yarn_frequencies(rd, base, scaling)
    pages = (int(pos.max()) // 64) + 1
    table = torch.full((1, pages), -1, dtype=torch.int32, device=DEV)
    for i, p in enumerate(sorted({int(x) // 64 for x in pos})):
        table[0, p] = i
    kc = torch.full((T, 1, 64, r + rd), float("nan"), device=DEV)
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    q = torch.full((T, H * (d + rd)), float("nan"), device=DEV)
    wide = torch.full((T, u.shape[1] + 5), float("nan"), device=DEV)          # (rows of a wider product)
    wide[:, :u.shape[1]] = f32(u)
    ops.latent_prepare(wide[:, :u.shape[1]], H * (d + rd), True, q, d + rd, d, True, f32(nw), eps, i32(pos), i32([0] * T), table, kc, H, d, rd, r,
                       rotary_frequencies(rd, base, scaling).to(DEV), err, interleaved=interleaved, rot_mult=rotary_magnitude(scaling))
    turn = plain.rotate_neighbours
    if not interleaved:       # half-split pairs are neighbouring pairs of the shuffled vector
        order = np.stack([np.arange(rd // 2), np.arange(rd // 2) + rd // 2], 1).reshape(-1)
        turn = lambda x, p, f_, m: plain.rotate_neighbours(x[..., order], p, f_, m)[..., np.argsort(order)]
    qq = u[:, :H * (d + rd)].reshape(T, H, d + rd)
    want_q = np.concatenate([qq[..., :d], turn(qq[..., d:], pos, f, mult)], -1).reshape(T, -1)
    c = plain.rms_norm(u[:, H * (d + rd):H * (d + rd) + r], eps, nw)
    want_row = np.concatenate([c, turn(u[:, None, H * (d + rd) + r:], pos, f, mult)[:, 0]], -1)
    got_row = np.stack([kc[int(table[0, p // 64]), 0, p % 64].cpu().numpy() for p in pos])
    assert np.abs(q.cpu().numpy() - want_q).max() < 3e-6 and np.abs(got_row - want_row).max() < 3e-6
    assert int(err.item()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,d,rd,e,r,window", [(4, 16, 8, 24, 32, 50), (9, 10, 4, 6, 20, 70), (1, 12, 4, 30, 20, None), (2, 24, 8, 32, 64, 64), (3, 48, 48, 64, 72, 100),
                                               (2, 48, 16, 32, 40, 1), (5, 96, 32, 128, 48, None), (17, 8, 24, 32, 24, 65)])
def test_latent_attention_with_window_sink_and_gate(H, d, rd, e, r, window, dtype):
    """Every form against the plain way (keys and values expanded per head for every token): a prompt through tiles over the
    cache's rows and with the step's own keys, then one token a sequence, the pages split over blocks or not.  One key of every
    sequence is large, so that it decides where it is seen."""
    g = np.random.default_rng(r + d)
    rnd, lengths, eps, base, scale = rounder(dtype), [140, 9, 131], 1e-5, 300.0, 0.25
    scaling = {"factor": 3.0, "original": 60, "fast": 5.0, "slow": 0.5}
    uk, uv, nw = rnd(g.normal(size=(H * d, r)) / np.sqrt(r)), rnd(g.normal(size=(H * e, r)) / np.sqrt(r)), rounder(torch.float32)(g.uniform(0.6, 1.4, r))
    sink = rounder(torch.float32)(g.uniform(-2.0, 4.0, H))
    width = H * (d + rd) + r + rd
    U = [rounder(torch.float32)(g.normal(size=(n, width + H))) for n in lengths]
    for u, n in zip(U, lengths):
        u[n // 3, width - rd:width] *= 4.0
    kv = PagedKV(lengths, 1, r + rd, r, dtype, seed=5, values_in_keys=True)
    table, err = i32(kv.table), torch.zeros(1, dtype=torch.int32, device=DEV)
    freq = rotary_frequencies(rd, base, scaling).to(DEV)
    f, mult = plain.yarn_frequencies(rd, base, scaling)
    rot = dict(interleaved=True, rot_mult=rotary_magnitude(scaling))
    w_ukt = torch.tensor(uk.reshape(H, d, r).transpose(0, 2, 1).copy(), dtype=dtype, device=DEV)
    w_uv = torch.tensor(uv.reshape(H, e, r), dtype=dtype, device=DEV).contiguous()
    mask = (ops.MASK_WINDOW, window) if window else (ops.MASK_CAUSAL, 0)
    want = []
    for u, n in zip(U, lengths):
        q = u[:, :H * (d + rd)].reshape(n, H, d + rd)
        c = rnd(plain.rms_norm(u[:, H * (d + rd):H * (d + rd) + r], eps, nw))                    # (the cache's rounding)
        kr = rnd(plain.rotate_neighbours(u[:, None, H * (d + rd) + r:width], np.arange(n), f, mult)[:, 0])
        qq = np.concatenate([q[..., :d], plain.rotate_neighbours(q[..., d:], np.arange(n), f, mult)], -1)
        kk = np.concatenate([(c @ uk.T).reshape(n, H, d), np.broadcast_to(kr[:, None], (n, H, rd))], -1)
        o = plain.window_softmax_attention(qq, kk, (c @ uv.T).reshape(n, H, e), scale, window, sink)
        want.append((o * plain.sigmoid(u[:, width:])[:, :, None]).reshape(n, H * e))
    tol = 3e-5 if dtype == torch.float32 else 4e-2
    for phase in ("prompt", "single"):
        live = [(s, 0, n - 1) for s, n in enumerate(lengths)] if phase == "prompt" else [(s, n - 1, 1) for s, n in enumerate(lengths)]
        rows_u = f32(np.concatenate([U[s][a:a + n] for s, a, n in live]))
        u, gate, T = rows_u[:, :width], rows_u[:, width:], rows_u.shape[0]
        pos = i32(np.concatenate([np.arange(a, a + n) for _, a, n in live]))
        _, tok_seq = packed([n for _, _, n in live])
        tb = table[[s for s, _, _ in live]].contiguous()
        ref = np.concatenate([want[s][a0:a0 + n] for s, a0, n in live])
        qf = torch.full((T, H * (r + rd)), float("nan"), device=DEV)
        ops.latent_prepare(u, H * (d + rd), True, qf, r + rd, r, False, f32(nw), eps, pos, tok_seq, tb, kv.k, H, d, rd, r, freq, err, **rot)
        ops.head_matmul(u, d + rd, w_ukt, qf, r + rd)

        def expanded(ol):
            a = torch.full((T, H * e), float("nan"), dtype=dtype, device=DEV)
            ops.head_matmul(ol, r, w_uv, a, e)
            return a.float().cpu().numpy()
        forms = {}
        if phase == "prompt":
            tile = max(1, 32 // H)
            tseq, ttok0, tntok, tpos0, count = make_tiles([n for _, _, n in live], [a for _, a, _ in live], tile)
            ol = torch.full((T, H * r), float("nan"), device=DEV)
            ops.masked_attn_tiled(qf, ol, kv.k, None, tb, tseq, ttok0, tntok, tpos0, count, tile, H, 1, r + rd, r, scale, *mask, f32(sink), gate=gate)
            forms["tiles"] = expanded(ol)
            q2 = torch.full((T, H * (d + rd)), float("nan"), device=DEV)
            rows = torch.full((T, r + rd), float("nan"), dtype=dtype, device=DEV)
            ops.latent_prepare(u, H * (d + rd), True, q2, d + rd, d, True, f32(nw), eps, pos, tok_seq, tb, kv.k, H, d, rd, r, freq, err, row_out=rows, **rot)
            c = rows[:, :r].float()
            kn = (c @ torch.tensor(uk, dtype=torch.float32, device=DEV).T).to(dtype).contiguous()
            vx = (c @ torch.tensor(uv, dtype=torch.float32, device=DEV).T).to(dtype).contiguous()
            kx = torch.full((T, H * (d + rd)), float("nan"), dtype=dtype, device=DEV)
            ops.latent_expand_keys(kn, rows, kx, H, d, rd, r)
            a2 = torch.full((T, H * e), float("nan"), dtype=dtype, device=DEV)
            tseq, ttok0, tntok, tpos0, count = make_tiles([n for _, _, n in live], [0] * len(live), 32)
            ops.masked_attn_tiled(q2, a2, kx, vx, None, tseq, ttok0, tntok, tpos0, count, 32, H, H, d + rd, e, scale, *mask, f32(sink), gate=gate)
            forms["own keys"] = a2.float().cpu().numpy()
            if ops.attn_prefill_split_takes(dtype, d + rd, e):
                tseq, ttok0, tntok, tpos0, count = make_tiles([n for _, _, n in live], [0] * len(live), ops.SPLIT_PREFILL_TILE)
                for most in (140, 4000):       # (one warp group a tile, and two that share its pages)
                    a3 = torch.full((T, H * e), float("nan"), dtype=dtype, device=DEV)
                    ops.attn_prefill_split(q2, a3, kx, vx, None, tseq, ttok0, tntok, tpos0, count, H, H, d + rd, e, scale, gate=gate, max_keys=most,
                                           mask=mask[0], mask_size=mask[1], sink=f32(sink))
                    forms[f"own keys, tensor cores, {most}"] = a3.float().cpu().numpy()
                    assert np.abs(forms[f"own keys, tensor cores, {most}"] - forms["own keys"]).max() < 8e-3 * max(1.0, np.abs(ref).max())     # (the output's rounding)
        else:
            ol = torch.full((T, H * r), float("nan"), device=DEV)
            ops.masked_attn(qf, ol, kv.k, None, pos, tok_seq, tb, H, 1, r + rd, r, scale, *mask, f32(sink), window or 1 << 30, gate=gate)
            forms["a block a head"] = expanded(ol)
            for splits in (1, 2, 3):
                ol = torch.full((T, H * r), float("nan"), device=DEV)
                part = torch.full((T * H * splits * (2 + r),), float("nan"), device=DEV)
                idx = torch.arange(T, dtype=torch.int32, device=DEV)
                ops.masked_attn_tiled(qf, ol, kv.k, None, tb, idx, idx, torch.ones_like(idx), pos, T, 1, H, 1, r + rd, r, scale, *mask, f32(sink), n_splits=splits,
                                      part=part if splits > 1 else None, gate=gate)
                forms[f"shared rows, {splits} splits"] = expanded(ol)
        for how, got in forms.items():
            assert np.abs(got - ref).max() < tol * max(1.0, np.abs(ref).max()), (phase, how)
    assert int(err.item()) == 0


@pytest.mark.parametrize("H,G,dk,dv", [(4, 2, 64, 32), (3, 1, 96, 64), (2, 2, 128, 96), (2, 1, 64, 64), (2, 2, 32, 32), (1, 1, 96, 32), (2, 1, 128, 128), (1, 1, 128, 64),
                                       (1, 1, 128, 32), (1, 1, 96, 96)])
@pytest.mark.parametrize("kind,size", [("causal", 0), ("window", 1), ("window", 64), ("window", 77), ("window", 200), ("chunk", 50), ("chunk", 64), ("chunk", 130)])
def test_prompt_attention_on_tensor_cores_under_every_mask(H, G, dk, dv, kind, size):
    """Paged keys and values, sequences that start at position 0 and pieces that go on in the middle of a page, one standout key a
    sequence; the exact attention of the same bfloat16 keys and values, with a sink."""
    g = np.random.default_rng(dk + size)
    rnd, lengths, first, scale = rounder(torch.bfloat16), [300, 70, 129], [0, 37, 64], 0.3
    q = rounder(torch.float32)(g.normal(size=(sum(n - a for n, a in zip(lengths, first)), H, dk)))
    sink = rounder(torch.float32)(g.uniform(-1.0, 4.0, H))
    kv = PagedKV(lengths, G, dk, dv, torch.bfloat16, seed=2)
    kv.v.fill_(1e4)
    want, at = [], 0
    for s, (n, a) in enumerate(zip(lengths, first)):
        k, v = rnd(g.normal(size=(n, G, dk))), rnd(g.normal(size=(n, G, dv)))
        k[n // 3] = rnd(k[n // 3] * 3.0)
        kv.put(s, k, v)
        for i in range(a, n):
            lo = {"causal": 0, "window": max(0, i - size + 1), "chunk": i // size * size if size else 0}[kind]
            row = []
            for h in range(H):
                sc = (k[lo:i + 1, h // (H // G)] @ q[at, h]) * scale
                top = max(sc.max(), sink[h])
                p = np.exp(sc - top)
                row.append((p / (p.sum() + np.exp(sink[h] - top))) @ v[lo:i + 1, h // (H // G)])
            want.append(np.concatenate(row))
            at += 1
    want = np.array(want)
    n_new = [n - a for n, a in zip(lengths, first)]
    tseq, ttok0, tntok, tpos0, count = make_tiles(n_new, first, ops.SPLIT_PREFILL_TILE)
    mask = {"causal": ops.MASK_CAUSAL, "window": ops.MASK_WINDOW, "chunk": ops.MASK_CHUNK}[kind]
    for most in (64, 4000):
        out = torch.full((sum(n_new), H * dv), float("nan"), dtype=torch.bfloat16, device=DEV)
        ops.attn_prefill_split(f32(q.reshape(len(q), H * dk)), out, kv.k, kv.v, i32(kv.table), tseq, ttok0, tntok, tpos0, count, H, G, dk, dv, scale, max_keys=most,
                               mask=mask, mask_size=size, sink=f32(sink))
        assert np.abs(out.float().cpu().numpy() - want).max() < 6e-3 * max(1.0, np.abs(want).max())


# ----------------------------------------------------------------------------- experts
@pytest.mark.parametrize("E,top", [(1, 1), (4, 2), (9, 9), (33, 4), (64, 1), (100, 8), (300, 3)])
@pytest.mark.parametrize("correction", [False, True])
def test_router_of_sigmoids(E, top, correction):
    """Each expert's sigmoid by itself, the largest chosen, the weights as they are; with a correction the choice looks at the
    corrected score and the weight stays the score.  Equal scores: the first."""
    g = np.random.default_rng(E + top)
    T, D = 150, 48
    h, wr = rounder(torch.float32)(g.normal(size=(T, D))), rounder(torch.float32)(g.normal(size=(E, D)) * 2 / np.sqrt(D))
    corr = rounder(torch.float32)(g.uniform(-0.5, 0.5, E)) if correction else np.zeros(E)
    s = plain.sigmoid(h @ wr.T)
    chosen, wts = plain.route(h @ wr.T, top)
    if correction:
        chosen = np.argsort(-(s + corr), axis=1, kind="stable")[:, :top]
        wts = np.take_along_axis(s, chosen, axis=1)
    idx = torch.empty(T, top, dtype=torch.int32, device=DEV)
    got = torch.empty(T, top, device=DEV)
    ops.moe_route_scored(f32(h), f32(wr), f32(corr) if correction else None, idx, got, top, E, score="sigmoid", renormalize=False)
    ranked = np.sort(s + corr, axis=1)[:, ::-1][:, :top + 1]
    clear = np.abs(np.diff(ranked, axis=1)).min(axis=1) > 1e-6 if ranked.shape[1] > 1 else np.ones(T, bool)
    assert clear.mean() > 0.9
    assert np.array_equal(idx.cpu().numpy()[clear], chosen[clear]) and np.abs(got.cpu().numpy()[clear] - wts[clear]).max() < 1e-6
    ops.moe_route_scored(f32(h), f32(np.tile(wr[:1], (E, 1))), None, idx, got, top, E, scale=2.0, score="sigmoid", renormalize=True)
    assert np.array_equal(idx.cpu().numpy(), np.tile(np.arange(top), (T, 1))) and np.abs(got.cpu().numpy() - 2.0 / top).max() < 1e-5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,D,E,top,ff", [(37, 64, 4, 2, 40), (1, 50, 2, 1, 30), (200, 48, 6, 3, 24), (9, 64, 5, 5, 16), (300, 72, 3, 1, 136), (70, 32, 1, 1, 8)])
def test_weights_on_the_experts_inputs(T, D, E, top, ff, dtype):
    """From the router to the sum: sum of expert(weight h), which differs from weight expert(h)."""
    g = np.random.default_rng(T + E)
    rnd = rounder(dtype)
    W = {"router": rounder(torch.float32)(g.normal(size=(E, D)) / np.sqrt(D))}
    for e in range(E):
        W[f"e{e}.gate"], W[f"e{e}.up"], W[f"e{e}.down"] = rnd(2.5 * g.normal(size=(ff, D)) / np.sqrt(D)), rnd(2.5 * g.normal(size=(ff, D)) / np.sqrt(D)), rnd(g.normal(size=(D, ff)) / np.sqrt(ff))
    h = rnd(g.normal(size=(T, D)))
    want = plain.moe_ffn(h, W, {"router": {"top": top}}, "")
    chosen, weight = plain.route(h @ W["router"].T, top)
    on_output = np.stack([sum(a * plain.gated_expert(h[t:t + 1], W, f"e{e}.")[0] for e, a in zip(chosen[t], weight[t])) for t in range(T)])
    assert np.abs(on_output - want).max() > 0.1 * np.abs(want).max()
    hd = torch.tensor(h, dtype=dtype, device=DEV)
    idx, wts = torch.empty(T, top, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV)
    ops.moe_route_scored(hd, f32(W["router"]), None, idx, wts, top, E, score="sigmoid", renormalize=False)
    ranked = np.sort(plain.sigmoid(h @ W["router"].T), axis=1)[:, ::-1][:, :top + 1]
    clear = np.abs(np.diff(ranked, axis=1)).min(axis=1) > 1e-6 if ranked.shape[1] > 1 else np.ones(T, bool)
    stack = lambda n: torch.tensor(np.stack([W[f"e{e}.{n}"] for e in range(E)]), dtype=dtype, device=DEV)
    tol, err = 2e-5 if dtype == torch.float32 else 2e-2, torch.zeros(1, dtype=torch.int32, device=DEV)
    for tensor_cores in ((False, True) if dtype == torch.bfloat16 else (False,)):
        if tensor_cores and (D % 8 or ff % 8):
            continue
        rows = ops.moe_tile_rows(tensor_cores)
        max_tiles = ops.moe_max_tiles(T * top, E, rows)
        row_pair, pair_row = torch.empty(max_tiles * rows, dtype=torch.int32, device=DEV), torch.empty(T * top, dtype=torch.int32, device=DEV)
        tile_expert = torch.empty(max_tiles, dtype=torch.int32, device=DEV)
        ops.moe_plan(idx, E, rows, row_pair, pair_row, tile_expert)
        mid = torch.full((max_tiles * rows, ff), float("nan"), dtype=dtype, device=DEV)
        y = torch.full((max_tiles * rows, D), float("nan"), device=DEV)
        if tensor_cores:
            a = torch.full((max_tiles * rows, D), float("nan"), dtype=dtype, device=DEV)
            ops.moe_gather_rows(hd, a, row_pair, top)
            ops.gemm_tc_grouped(a, stack("gate"), mid, tile_expert, err, epilogue=ops.EPI_SWIGLU, w2=stack("up"), row_pair=row_pair, in_weight=wts)
            ops.gemm_tc_grouped(mid, stack("down"), y, tile_expert, err)
        else:
            ops.moe_gate_up(hd, stack("gate"), stack("up"), mid, row_pair, tile_expert, top, in_weight=wts)
            ops.moe_down(mid, stack("down"), y, row_pair, tile_expert, top)
        x = torch.ones(T, D, device=DEV)
        ops.moe_combine(x, y, None, pair_row, top=top)
        assert np.abs(x.cpu().numpy()[clear] - 1.0 - want[clear]).max() < tol * max(1.0, np.abs(want).max()), tensor_cores
    assert int(err.item()) == 0


# ----------------------------------------------------------------------------- products
@pytest.mark.parametrize("M,N,K", [(1, 100, 72), (8, 640, 256), (16, 33, 40), (5, 9000, 1024), (17, 96, 64), (64, 256, 2048), (100, 72, 40), (300, 576, 576), (2048, 4096, 1024),
                                   (3, 41, 30), (90, 50, 26)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_squared_relu_in_every_product(M, N, K, dtype):
    """The dispatch's kernels (few rows on tensor cores and CUDA cores, narrow, wide, split and persistent tcgen05 tiles, any size) and
    each forced one, against float64."""
    g = torch.Generator(device=DEV).manual_seed(M + N)
    a = (torch.randn(M, K, generator=g, device=DEV)).to(dtype)
    w = (torch.randn(N, K, generator=g, device=DEV) / K ** 0.5).to(dtype)
    want = torch.clamp(a.double() @ w.double().T, min=0.0).square().cpu().numpy()
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    ctx = types.SimpleNamespace(err=err, n_sms=148)
    runs = {"dispatch": lambda o: linear.matmul(ctx, a, w, o, epilogue=linear.EPI_RELU2)}
    if M <= 300:
        runs["any size"] = lambda o: ops.gemm_simt(a, w, o, epilogue=ops.EPI_RELU2)
    if M <= 16 and ops.gemv_takes(a, w):
        runs["few rows"] = lambda o: ops.gemv(a, w, o, epilogue=ops.EPI_RELU2)
    if ops.gemm_tc_takes(a, w, None):
        runs["tcgen05"] = lambda o: ops.gemm_tc(a, w, o, err, epilogue=ops.EPI_RELU2)
    tol = 3e-5 if dtype == torch.float32 else 1e-2
    for how, run in runs.items():
        o = torch.full((M, N), float("nan"), dtype=dtype, device=DEV)
        run(o)
        got = o.double().cpu().numpy()
        assert (np.abs(got - want) <= tol * np.maximum(1.0, want)).all(), how
    assert int(err.item()) == 0


# ----------------------------------------------------------------------------- linear attention
@pytest.mark.parametrize("H,d,e,decay", [(2, 32, 16, (0.4, 1.0)), (3, 20, 44, (0.99, 0.7, 0.999)), (1, 72, 8, (0.95,)), (2, 64, 96, (0.5, 0.998)), (1, 130, 12, (0.9,))])
def test_linear_attention_over_steps(H, d, e, decay):
    """The recurrence in whole prompts (walked and chunk by chunk), in pieces and token by token, on scattered slots."""
    g = np.random.default_rng(d + e)
    lengths = [200, 67]
    off_k, off_v, width = H * d, 2 * H * d, 2 * H * d + H * e
    U = [rounder(torch.float32)(g.normal(size=(n, width))) for n in lengths]
    want = [plain.decayed_linear_attention(plain.silu(u[:, :off_k]).reshape(-1, H, d), plain.silu(u[:, off_k:off_v]).reshape(-1, H, d),
                                           plain.silu(u[:, off_v:]).reshape(-1, H, e), np.array(decay)).reshape(-1, H * e) for u in U]
    slots, dec, powers = i32([3, 1]), f32(decay), ops.decay_powers(decay).to(DEV)
    for how in ("walk", "chunks"):
        if how == "chunks" and not ops.decay_chunked_takes(d, e):
            continue
        for cuts in ([(200,), (67,)], [(64, 2, 100, 1, 33), (1, 63, 1, 1, 1)]):
            state = torch.zeros(5, H, e, d, device=DEV)
            at, got = [0, 0], [[], []]
            for k in range(len(cuts[0])):
                ns = [c[k] for c in cuts]
                u = f32(np.concatenate([U[s][at[s]:at[s] + n] for s, n in enumerate(ns)]))
                tok0, _ = packed(ns)
                o = torch.full((sum(ns), H * e), float("nan"), device=DEV)
                if how == "walk":
                    ops.decay_scan(u, 0, off_k, off_v, dec, state, o, tok0, slots, 2, H, d, e, act="silu")
                else:
                    tseq, ttok0, tntok, tpos0, count = make_tiles(ns, at, ops.DECAY_CHUNK)
                    scratch = torch.empty(ops.decay_chunked_scratch_floats(count, H, d, e), device=DEV)
                    ops.decay_chunked(u, 0, off_k, off_v, powers, state, o, tok0, slots, 2, ttok0, tntok, count, H, d, e, act="silu", scratch=scratch)
                host = o.cpu().numpy()
                for s in range(2):
                    got[s].append(host[sum(ns[:s]):sum(ns[:s + 1])])
                    at[s] += ns[s]
            for s in range(2):
                assert np.abs(np.concatenate(got[s]) - want[s]).max() < 2e-5 * max(1.0, np.abs(want[s]).max()), (how, cuts)
