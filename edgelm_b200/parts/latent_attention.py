"""Attention whose keys and values are expanded from a shared low-rank latent.

Per token the mixer keeps a latent c (size `kv_rank`, RMS-normed with a weight) and one rotated key part (size
`rot_dim`) shared by all heads: [c | k_rot] = W_dkv h.  A query head is [q_n (size `head_dim`) | q_r (size `rot_dim`)];
q_r and k_rot are rotated by position * f_i, with half-split pairs (i, i + rot_dim / 2) (`rot_pairs` "half") or neighbouring ones
(2i, 2i + 1) ("interleaved"); frequencies and the rotated vectors' length may be scaled (`parts.rope.rotary_frequencies`,
`rotary_magnitude`).  Per head the unrotated key is W_uk c and the value W_uv c, and score = (q_n . W_uk c + q_r . k_rot) * scale.

Since q_n . (W_uk c) = (W_uk^T q_n) . c, the queries are moved into the latent's space once per token and attention
runs over the cache rows [c | k_rot] as they are: one key head of size kv_rank + rot_dim for all query heads, whose first
kv_rank dimensions are also its value; the weighted latents are then expanded with W_uv.  Nothing per head is ever
computed for a cached token.  A prompt step whose sequences all start at position 0 (and which keeps its own latent) sees
only its own tokens: it expands their keys and values per head once, with two matrix products over the rows it has just
written, and attends over those, heads of head_dim + rot_dim against values of v_head_dim, which is several times fewer
multiply-adds than rows of the latent's size (on the tensor cores, where their kernel takes the head sizes).  A layer with `reads_cache` keeps nothing: it has no W_dkv and reads the rows that an
earlier layer of the same kv_rank, rot_dim and rotation left in its cache, with its own W_uk, W_uv, queries and mask; a prompt step
of first tokens fetches its own tokens' rows from there and then goes the same way.

Options: `q_rank`: the queries go through a latent of their own, q = W_uq c_q with c_q the RMS-normed W_dq h (`names` dq, dq_norm, uq
instead of q); a `mask` (as in `masked_attention.py`); `names["sink"]`, a tensor with one number per head: the softmax's denominator
then also holds exp(sink_h), without a key, a value or the scale; `head_gate` True: `names["gate"]` [heads, hidden] rides in the
input product, and head h's output is multiplied by the sigmoid of its number (the attention kernels multiply before they round; in
the latent's space this comes to the same, the expansion by W_uv being linear).

Angles, the latent's norm, scores, the softmax and the weighted latents are float32 in both precisions; the cache rows
are kept in the compute dtype.
"""
import torch

from ..config.base import ConfigError
from ..csrc import ops
from . import linear
from .base import KVNeed, Part, as_matrix, as_vector, nbytes
from .masked_attention import MASKS, MAX_SPLITS, SHARED_KEYS_MIN_GROUP, decode_splits, kept_first, most_keys, read_mask, single_token_tiles, splits_room
from .registry import register_mixer
from .rope import rotary_frequencies, rotary_magnitude


@register_mixer("latent_attention")
class LatentAttention(Part):
    graph_safe = True

    def __init__(self, spec, env):
        self.hidden = spec["hidden_size"]
        self.nh, self.d, self.rd, self.dv, self.rank = spec["num_heads"], spec["head_dim"], spec["rot_dim"], spec["v_head_dim"], spec["kv_rank"]
        self.scale, self.eps = float(spec["scale"]), float(spec["eps"])
        self.rot_base, self.rot_scaling = float(spec.get("rot_base") or 10000.0), spec.get("rot_scaling")
        self.interleaved = spec.get("rot_pairs", "half") == "interleaved"
        self.rot_mult = rotary_magnitude(self.rot_scaling)
        self.head_gate = bool(spec.get("head_gate", False))
        self.reads_foreign_cache = bool(spec.get("reads_cache", False))
        self.names = dict(spec["names"])
        self.dtype = env.dtype
        if self.nh < 1 or self.d < 0 or self.rd < 0 or self.rd % 2 or self.d + self.rd < 1 or self.dv < 1 or self.rank < 1:
            raise ConfigError(f"latent_attention: {self.nh} heads of {self.d} + {self.rd}, values of {self.dv}, a latent of {self.rank}")
        if self.rank + self.rd > 1024 or self.rank > 512:
            raise ConfigError(f"latent_attention: a latent of {self.rank} + {self.rd} is not taken (latent to 512, row to 1024)")
        self.q_rank = int(spec.get("q_rank") or 0)          # 0: the queries are a projection of the mixer's input
        self.mask, self.mask_size = read_mask(spec.get("mask"), "latent_attention")
        self.keep = kept_first(spec.get("mask"), "latent_attention")
        self.dq, self.dc = self.d + self.rd, self.rank + self.rd
        self.d_q = self.q_rank or self.nh * self.dq          # columns of the input product that the queries take
        self.d_qkv = self.d_q + (0 if self.reads_foreign_cache else self.dc)
        self.d_in = self.d_qkv + (self.nh if self.head_gate else 0)         # columns of the input product: q | latent row | gate
        self.d_row = (self.d_in + 7) // 8 * 8 if self.head_gate else self.d_in      # their pitch: rows start on 16-byte boundaries
        self.tile_tokens = max(1, 32 // self.nh)
        self.freq = self.norm_w = self.sink = self.qn_w = self.w_uq = None

    EXPANDED_TILE = 32      # tokens a tile when every head has its own keys (a block's 32 rows are 32 tokens of one head)

    def _on_tensor_cores(self):
        """Whether prompt steps that see their own tokens only take the tensor-core kernel with float32 scores and weights."""
        return ops.attn_prefill_split_takes(self.dtype, self.dq, self.dv)

    def tile_sizes(self):
        return (self.tile_tokens, ops.SPLIT_PREFILL_TILE if self._on_tensor_cores() else self.EXPANDED_TILE)

    def sizes(self):
        return {"heads": self.nh, "head_dim": self.d, "rot_dim": self.rd, "v_head_dim": self.dv, "kv_rank": self.rank,
                **({"q_rank": self.q_rank} if self.q_rank else {}),
                "mask": {v: k for k, v in MASKS.items()}[self.mask], "reads_cache": self.reads_foreign_cache,
                **({"kept_first": self.keep} if self.keep else {}),
                **({"mask_size": self.mask_size} if self.mask != ops.MASK_CAUSAL else {}), **({"sink": True} if "sink" in self.names else {}),
                **({"head_gate": True} if self.head_gate else {})}

    def flops(self, n_tokens, attended):
        proj = 2.0 * n_tokens * (self.hidden * (self.d_in + self.nh * self.dv) + self.nh * self.rank * (self.d + self.dv) +
                                 self.q_rank * self.nh * self.dq)
        if self.mask != ops.MASK_CAUSAL:
            attended = min(attended, n_tokens * (self.mask_size + self.keep))
        return proj + 2.0 * attended * self.nh * (self.dc + self.rank)

    def weight_shapes(self, prefix):
        n = self.names
        out = {prefix + n["uk"]: (self.nh * self.d, self.rank),
               prefix + n["uv"]: (self.nh * self.dv, self.rank), prefix + n["o"]: (self.hidden, self.nh * self.dv)}
        if self.q_rank:
            out.update({prefix + n["dq"]: (self.q_rank, self.hidden), prefix + n["dq_norm"]: (self.q_rank,), prefix + n["uq"]: (self.nh * self.dq, self.q_rank)})
        else:
            out[prefix + n["q"]] = (self.nh * self.dq, self.hidden)
        if not self.reads_foreign_cache:
            out[prefix + n["dkv"]] = (self.dc, self.hidden)
            out[prefix + n["dkv_norm"]] = (self.rank,)
        if self.head_gate:
            out[prefix + n["gate"]] = (self.nh, self.hidden)
        if "sink" in n:
            out[prefix + n["sink"]] = (self.nh,)
        return out

    def load(self, tensors, prefix, device):
        n = self.names
        mats = [as_matrix(tensors[prefix + n["dq" if self.q_rank else "q"]], self.dtype, device)]
        if self.q_rank:
            self.qn_w, self.w_uq = as_vector(tensors[prefix + n["dq_norm"]], device), as_matrix(tensors[prefix + n["uq"]], self.dtype, device)
        if not self.reads_foreign_cache:
            mats.append(as_matrix(tensors[prefix + n["dkv"]], self.dtype, device))
            self.norm_w = as_vector(tensors[prefix + n["dkv_norm"]], device)
        if self.head_gate:
            mats.append(as_matrix(tensors[prefix + n["gate"]], self.dtype, device))
        if "sink" in n:
            self.sink = as_vector(tensors[prefix + n["sink"]], device)
        self.w_in = torch.cat(mats, dim=0).contiguous()
        # per head: W_uk^T as [rank, d] (queries into the latent's space) and W_uv as [dv, rank] (weighted latents out of it)
        self.w_uk = as_matrix(tensors[prefix + n["uk"]], self.dtype, device)        # [heads * d, rank]: a step's own keys
        self.w_ukt = self.w_uk.view(self.nh, self.d, self.rank).transpose(1, 2).contiguous()
        self.w_uv2 = as_matrix(tensors[prefix + n["uv"]], self.dtype, device)       # [heads * dv, rank]: a step's own values
        self.w_uv = self.w_uv2.view(self.nh, self.dv, self.rank)
        self.w_o = as_matrix(tensors[prefix + n["o"]], self.dtype, device)
        if self.rd:
            self.freq = rotary_frequencies(self.rd, self.rot_base, self.rot_scaling).to(device).contiguous()

    def first_weights(self):
        return (self.w_in,)

    def cache_need(self):
        if self.reads_foreign_cache:
            return None
        return KVNeed(1, self.dc, None, v_head_dim=self.rank, values_in_keys=True)

    def workspace_bytes(self, n_tokens, n_seqs):
        f32 = torch.float32
        absorbed = nbytes((n_tokens, self.nh * self.dc), f32) + nbytes((n_tokens, self.nh * self.rank), f32)
        expanded = (nbytes((n_tokens, self.nh * self.dq), f32) + nbytes((n_tokens, self.dc), self.dtype) + nbytes((n_tokens, self.nh * self.d), self.dtype) +
                    nbytes((n_tokens, self.nh * self.dq), self.dtype) + nbytes((n_tokens, self.nh * self.dv), self.dtype))
        return (nbytes((n_tokens, self.d_row), f32) +
                (nbytes((n_tokens, self.q_rank), self.dtype) + nbytes((n_tokens, self.nh * self.dq), f32) if self.q_rank else 0) + max(absorbed + splits_room(n_seqs, self.nh, self.rank), expanded) +
                nbytes((n_tokens, self.nh * self.dv), self.dtype) + nbytes((n_tokens, self.hidden), self.dtype))

    def _decode_splits(self, ctx, heads):
        """Blocks that share a token's pages in `latent_decode`: as many as fill the device once, at most a block a page of the mask."""
        splits = max(1, min(MAX_SPLITS, ctx.n_sms // max(1, ctx.n_seqs * -(-self.nh // heads))))
        if self.mask != ops.MASK_CAUSAL:
            splits = min(splits, (self.mask_size + 63) // 64 + 1 + (self.keep + 63) // 64)
        return splits

    def _prepare(self, ctx, u, cache, q_out, q_pitch, q_off, copy_q, rows=None):
        """Queries from their latent if they have one; rotation; the latent's norm and the cache append (and the step's `rows`).
        q_out receives the queries' rotated part at q_off of every q_pitch values, with `copy_q` the unrotated part ahead of it.
        Returns the product that the unrotated parts stand in (its head h at h * dq)."""
        own, table = not self.reads_foreign_cache, ctx.page_table(cache.group)
        kv = (self.norm_w, self.eps, ctx.tok_pos, ctx.tok_seq, table if own else None, cache.k if own else None)
        sizes = (self.d, self.rd, self.rank, self.freq, ctx.err)
        rot = dict(interleaved=self.interleaved, rot_mult=self.rot_mult)
        if not self.q_rank:
            ops.latent_prepare(u, self.d_q, own, q_out, q_pitch, q_off, copy_q, *kv, self.nh, *sizes, row_out=rows, **rot)
            return u
        cq = ctx.ws.alloc((u.shape[0], self.q_rank), self.dtype)
        ops.latent_prepare(u, self.d_q, own, None, 0, 0, False, *kv, 0, *sizes, row_out=rows, q_latent=(0, self.qn_w, cq), **rot)
        if copy_q and not self.rd:      # (nothing to rotate: the product is what is asked for)
            linear.matmul(ctx, cq, self.w_uq, q_out, prefetch=(self.w_uk,))
            return q_out
        q = ctx.ws.alloc((u.shape[0], self.nh * self.dq), torch.float32)
        linear.matmul(ctx, cq, self.w_uq, q, prefetch=(self.w_ukt,))
        if self.rd:
            ops.latent_prepare(q, 0, False, q_out, q_pitch, q_off, copy_q, None, self.eps, ctx.tok_pos, ctx.tok_seq, None, None, self.nh, *sizes, **rot)
        return q

    def _forward_own_keys(self, ctx, u, gate, x, cache, accumulate):
        """A prompt step that sees only its own tokens: keys and values expanded per head for the step's tokens."""
        T, ws = u.shape[0], ctx.ws
        q = ws.alloc((T, self.nh * self.dq), torch.float32)
        rows = ws.alloc((T, self.dc), self.dtype)
        with ctx.prof("latent_prepare"):
            self._prepare(ctx, u, cache, q, self.dq, self.d, True, rows=None if self.reads_foreign_cache else rows)
            if self.reads_foreign_cache:
                ops.latent_rows(cache.k, rows, ctx.tok_pos, ctx.tok_seq, ctx.page_table(cache.group), ctx.err)
        kn = ws.alloc((T, self.nh * self.d), self.dtype)
        kx = ws.alloc((T, self.nh * self.dq), self.dtype) if self.rd else kn
        vx = ws.alloc((T, self.nh * self.dv), self.dtype)
        with ctx.prof("latent_expand"):
            linear.matmul(ctx, rows[:, :self.rank], self.w_uk, kn)
            linear.matmul(ctx, rows[:, :self.rank], self.w_uv2, vx)
            if self.rd:
                ops.latent_expand_keys(kn, rows, kx, self.nh, self.d, self.rd, self.rank)
        a = ws.alloc((T, self.nh * self.dv), self.dtype)
        with ctx.prof("attn_latent"):
            if self._on_tensor_cores():
                tiles = ctx.tiles(ops.SPLIT_PREFILL_TILE)
                ops.attn_prefill_split(q, a, kx, vx, None, tiles.seq, tiles.tok0, tiles.ntok, tiles.pos0, tiles.count, self.nh, self.nh, self.dq, self.dv,
                                       self.scale, gate=gate, max_keys=max(ctx.seq_lengths), mask=self.mask, mask_size=self.mask_size, sink=self.sink,
                                       keep=self.keep)
            else:
                tiles = ctx.tiles(self.EXPANDED_TILE)
                ops.masked_attn_tiled(q, a, kx, vx, None, tiles.seq, tiles.tok0, tiles.ntok, tiles.pos0, tiles.count, self.EXPANDED_TILE,
                                      self.nh, self.nh, self.dq, self.dv, self.scale, self.mask, self.mask_size, self.sink, gate=gate, keep=self.keep)
        with ctx.prof("o_proj"):
            linear.matmul(ctx, a, self.w_o, x, epilogue=linear.EPI_RESIDUAL if accumulate else linear.EPI_STORE,
                          residual=x if accumulate else None, prefetch=ctx.weights_after)

    def forward(self, ctx, h, x, cache, accumulate=True):
        h = linear.as_tensor(h)
        T, ws, f32 = h.shape[0], ctx.ws, torch.float32
        if cache is None or cache.k is None or cache.k.shape[-1] != self.dc or cache.v is not None:
            raise ConfigError("latent_attention: the cache entry it was given does not hold rows of its latent's size")
        u = ws.alloc((T, self.d_row), f32)[:, :self.d_in]
        gate = u[:, self.d_qkv:] if self.head_gate else None
        with ctx.prof("latent_in_proj"):
            linear.matmul(ctx, h, self.w_in, u, prefetch=(self.w_uq,) if self.q_rank else (self.w_o,))
        if self.d and not ctx.all_single and ctx.all_fresh and (self._on_tensor_cores() or ops.masked_attn_tiled_takes(self.dq, self.dv)):
            return self._forward_own_keys(ctx, u, gate, x, cache, accumulate)
        qf = ws.alloc((T, self.nh * self.dc), f32)
        table = ctx.page_table(cache.group)
        with ctx.prof("latent_prepare"):
            q = self._prepare(ctx, u, cache, qf, self.dc, self.rank, False)
            if self.d:
                ops.head_matmul(q, self.dq, self.w_ukt, qf, self.dc)
            else:
                qf.view(T, self.nh, self.dc)[:, :, :self.rank].zero_()
        ol = ws.alloc((T, self.nh * self.rank), f32)
        tiled = ops.masked_attn_tiled_takes(self.dc, self.rank, own_values=False)      # (rows that a block can stage a page of)
        with ctx.prof("attn_latent"):
            heads = ops.latent_decode_takes(self.dtype, self.nh, self.dc, self.rank) if ctx.all_single else 0
            if heads:       # single tokens on the tensor cores: a row of the latent is staged once, as key and as value, for up to 32 heads
                splits = self._decode_splits(ctx, heads)
                part = ws.alloc((T * self.nh * splits * (2 + self.rank),), f32)
                ops.latent_decode(qf, ol, cache.k, ctx.tok_pos, ctx.tok_seq, table, self.nh, self.dc, self.rank, self.scale, self.mask, self.mask_size,
                                  self.sink, splits, part, gate=gate, keep=self.keep)
            elif ctx.all_single and self.nh >= SHARED_KEYS_MIN_GROUP and tiled:     # a row of the latent is staged once for all the heads
                splits = decode_splits(ctx, 1, self.nh, self.mask, self.mask_size, self.keep)
                part = ws.alloc((T * self.nh * splits * (2 + self.rank),), f32) if splits > 1 else None
                tseq, ttok0, tntok, tpos0 = single_token_tiles(ctx)
                ops.masked_attn_tiled(qf, ol, cache.k, None, table, tseq, ttok0, tntok, tpos0, T, 1, self.nh, 1, self.dc, self.rank, self.scale,
                                      self.mask, self.mask_size, self.sink, n_splits=splits, part=part, gate=gate, keep=self.keep)
            elif ctx.all_single or not tiled:
                ops.masked_attn(qf, ol, cache.k, None, ctx.tok_pos, ctx.tok_seq, table, self.nh, 1, self.dc, self.rank, self.scale,
                                self.mask, self.mask_size, self.sink, most_keys(self.mask, self.mask_size, self.keep), gate=gate, keep=self.keep)
            else:
                tiles = ctx.tiles(self.tile_tokens)
                ops.masked_attn_tiled(qf, ol, cache.k, None, table, tiles.seq, tiles.tok0, tiles.ntok, tiles.pos0, tiles.count,
                                      self.tile_tokens, self.nh, 1, self.dc, self.rank, self.scale, self.mask, self.mask_size, self.sink, gate=gate, keep=self.keep)
        a = ws.alloc((T, self.nh * self.dv), self.dtype)
        with ctx.prof("latent_values"):
            ops.head_matmul(ol, self.rank, self.w_uv, a, self.dv)
        with ctx.prof("o_proj"):
            linear.matmul(ctx, a, self.w_o, x, epilogue=linear.EPI_RESIDUAL if accumulate else linear.EPI_STORE,
                          residual=x if accumulate else None, prefetch=ctx.weights_after)
