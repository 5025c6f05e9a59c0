// Decode steps of an attention over shared latent rows (bfloat16 rows that are key and value at once, one for all query heads) on
// the tensor cores, with float32 scores and weights: the float32 operand of each product goes as three bfloat16 terms.
//
//   latent_decode    a block per (token, group of up to 32 heads, split of the token's pages).  A page of rows is staged once and
//                    used twice: S = Q K^T (the heads are the 16-row operand, the page's 64 keys the columns; a warp owns a tile of heads
//                    and 8 or 16 keys), then O += P K over the first dv columns (a warp owns columns).  Leaves every head's maximum,
//                    denominator and weighted rows for `masked_attn_fold`, where sinks and gates join.
//   head_matmul_few  out[t][h][n] = sum_k a[t][h][k] w[h][n][k] for up to 16 tokens: queries into the latent's space, weighted latents out
//                    of it.  The weights are the 16-row operand, fetched 16 bytes a thread with the K order permuted alike on both
//                    sides; warps share K; the float32 activations go as three terms.
#include <math_constants.h>

#include "mma_split.cuh"

namespace edgelm {

enum : int { LD_MASK_CAUSAL = 0, LD_MASK_WINDOW = 1, LD_MASK_CHUNK = 2 };

constexpr int LD_WARPS = 8;

__host__ __device__ constexpr size_t latent_decode_smem(int mt, int dc) {
  return (size_t)3 * 16 * mt * (dc + 8) * 2 + (size_t)PAGE * (dc + 8) * 2 + (size_t)16 * mt * (PAGE + 4) * 4 + (size_t)3 * 16 * mt * (PAGE + 8) * 2 +
         (size_t)3 * 16 * mt * 4;
}

template <int MT, int NV>      // tiles of 16 heads a block; tiles of 8 value columns a warp owns (even)
__global__ void __launch_bounds__(LD_WARPS * 32)
latent_decode_kernel(const float* __restrict__ q, const __nv_bfloat16* __restrict__ kcache, const int32_t* __restrict__ tok_pos,
                     const int32_t* __restrict__ tok_seq, const int32_t* __restrict__ page_table, int table_stride, int n_pages, int H, int dc,
                     int dv, float scale, int mask, int mask_size, int keep, int n_splits, float* __restrict__ part) {
  constexpr int ROWS = 16 * MT, SP = PAGE + 4, PP = PAGE + 8;
  extern __shared__ __align__(16) uint8_t ld_raw[];
  const int pitch = dc + 8;                                                   // (an odd number of 16-byte pieces: dc is a multiple of 16)
  __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(ld_raw);               // [3 terms][ROWS][pitch]
  __nv_bfloat16* Ks = Qs + (size_t)3 * ROWS * pitch;                          // [PAGE][pitch]
  float* Ss = reinterpret_cast<float*>(Ks + (size_t)PAGE * pitch);            // [ROWS][SP]
  __nv_bfloat16* Ps = reinterpret_cast<__nv_bfloat16*>(Ss + ROWS * SP);       // [3 terms][ROWS][PP]
  float* row_m = reinterpret_cast<float*>(Ps + 3 * ROWS * PP);                // running maximum, denominator, what the page before is scaled by
  float* row_l = row_m + ROWS;
  float* row_c = row_l + ROWS;
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, h0 = blockIdx.y * ROWS, split = blockIdx.z;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, gid = lane >> 2, tig = lane & 3;
  const int heads = min(ROWS, H - h0);
  const int pos = tok_pos[t];
  if (pos < 0) return;
  const int32_t* pages = page_table + (size_t)tok_seq[t] * table_stride;
  const int lo = mask == LD_MASK_WINDOW ? max(0, pos - mask_size + 1) : (mask == LD_MASK_CHUNK ? pos / mask_size * mask_size : 0);
  // the pages to visit: those of the kept keys that lie ahead of the first one behind the mask, then the rest
  const int first_page = lo / PAGE, kept_pages = min(first_page, (keep + PAGE - 1) / PAGE), n_visit = kept_pages + pos / PAGE - first_page + 1;
  const int per = (n_visit + n_splits - 1) / n_splits, v_begin = split * per, v_end = min(n_visit, v_begin + per);
  float* out = part + (((size_t)t * H + h0) * n_splits + split) * (2 + dv);   // head h0's; a head further: n_splits (2 + dv) on
  const size_t head_step = (size_t)n_splits * (2 + dv);
  if (v_begin >= v_end) {
    if (threadIdx.x < heads) {
      out[threadIdx.x * head_step] = -CUDART_INF_F;
      out[threadIdx.x * head_step + 1] = 0.f;
    }
    return;
  }
  auto load_page = [&](int kt) {
    const int page = pages[kt];
    const bool held = page >= 0 && page < n_pages;
    const int valid = held ? min(PAGE, pos + 1 - kt * PAGE) : 0;              // rows past the last key: zeros, nothing is read
    const __nv_bfloat16* src = kcache + (size_t)(held ? page : 0) * PAGE * dc;
    const int chunks = dc / 8;
    for (int i = threadIdx.x; i < PAGE * chunks; i += LD_WARPS * 32) {
      const int r = i / chunks, c = i - r * chunks;
      sp_cp16(sp_smem(Ks + (size_t)r * pitch + c * 8), r < valid ? src + (size_t)r * dc + c * 8 : kcache, r < valid ? 16 : 0);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  auto page_at = [&](int i) { return i < kept_pages ? i : first_page + i - kept_pages; };
  load_page(page_at(v_begin));
  {   // the queries' three terms
    const float* src = q + ((size_t)t * H + h0) * dc;
    for (int i = threadIdx.x * 4; i < ROWS * dc; i += LD_WARPS * 32 * 4) {
      const int r = i / dc, d = i - r * dc;
      const float4 v = r < heads ? *reinterpret_cast<const float4*>(src + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      uint32_t a[3], b[3];
      sp_split(v.x, v.y, a[0], a[1], a[2]);
      sp_split(v.z, v.w, b[0], b[1], b[2]);
#pragma unroll
      for (int k = 0; k < 3; ++k) *reinterpret_cast<uint2*>(Qs + ((size_t)k * ROWS + r) * pitch + d) = make_uint2(a[k], b[k]);
    }
    if (threadIdx.x < ROWS) {
      row_m[threadIdx.x] = -CUDART_INF_F;
      row_l[threadIdx.x] = 0.f;
    }
  }
  float o[NV][MT][4];
#pragma unroll
  for (int j = 0; j < NV; ++j)
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) o[j][mt][0] = o[j][mt][1] = o[j][mt][2] = o[j][mt][3] = 0.f;
  const int tile0 = warp * NV, v_tiles = dv / 8;
  constexpr int NK = MT;                                   // key tiles of 8 a warp scores
  const int s_mt = MT == 2 ? warp >> 2 : 0, s_kt = MT == 2 ? (warp & 3) * 2 : warp;
  for (int vi = v_begin; vi < v_end; ++vi) {
    const int kt = page_at(vi);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    // ---- scores of this warp's tile of heads and keys, a sum per term
    float s[NK][3][4];
#pragma unroll
    for (int n = 0; n < NK; ++n)
#pragma unroll
      for (int k = 0; k < 3; ++k) s[n][k][0] = s[n][k][1] = s[n][k][2] = s[n][k][3] = 0.f;
    {
      const __nv_bfloat16* qa = Qs + (size_t)(s_mt * 16 + (lane & 15)) * pitch + (lane >> 4) * 8;
      const int mi = lane >> 3;
      const __nv_bfloat16* kb = NK == 2 ? Ks + (size_t)((s_kt + (mi >> 1)) * 8 + (lane & 7)) * pitch + (mi & 1) * 8
                                        : Ks + (size_t)(s_kt * 8 + (lane & 7)) * pitch + (mi & 1) * 8;
#pragma unroll 4
      for (int d = 0; d < dc; d += 16) {
        uint32_t b[4];
        if constexpr (NK == 2) sp_ldmatrix_x4(sp_smem(kb + d), b[0], b[1], b[2], b[3]);
        else sp_ldmatrix_x2(sp_smem(kb + d), b[0], b[1]);
#pragma unroll
        for (int k = 0; k < 3; ++k) {
          uint32_t a0, a1, a2, a3;
          sp_ldmatrix_x4(sp_smem(qa + (size_t)k * ROWS * pitch + d), a0, a1, a2, a3);
          sp_mma(s[0][k], a0, a1, a2, a3, b[0], b[1]);
          if constexpr (NK == 2) sp_mma(s[NK - 1][k], a0, a1, a2, a3, b[2], b[3]);
        }
      }
    }
#pragma unroll
    for (int n = 0; n < NK; ++n)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int r = s_mt * 16 + gid + (j >> 1) * 8, c = (s_kt + n) * 8 + tig * 2 + (j & 1), p = kt * PAGE + c;
        const float v = (s[n][2][j] + s[n][1][j]) + s[n][0][j];               // (the small terms first)
        Ss[r * SP + c] = p <= pos && (p >= lo || p < keep) ? v * scale : -CUDART_INF_F;
      }
    __syncthreads();
    // ---- running maximum and denominator, weights as three terms (a warp: 2 MT rows, a lane two keys)
#pragma unroll
    for (int rr = 0; rr < 2 * MT; ++rr) {
      const int r = warp * 2 * MT + rr;
      const float2 v = *reinterpret_cast<const float2*>(Ss + r * SP + lane * 2);
      const float m_old = row_m[r], m_new = fmaxf(m_old, warp_max(fmaxf(v.x, v.y)));
      const bool some = m_new != -CUDART_INF_F;
      const float p0 = some ? expf(v.x - m_new) : 0.f, p1 = some ? expf(v.y - m_new) : 0.f;
      const float corr = some ? expf(m_old - m_new) : 1.f;
      const float sum = warp_sum(p0 + p1);
      uint32_t a[3];
      sp_split(p0, p1, a[0], a[1], a[2]);
#pragma unroll
      for (int k = 0; k < 3; ++k) *reinterpret_cast<uint32_t*>(Ps + ((size_t)k * ROWS + r) * PP + lane * 2) = a[k];
      __syncwarp();
      if (lane == 0) {
        row_m[r] = m_new;
        row_l[r] = row_l[r] * corr + sum;
        row_c[r] = corr;
      }
    }
    __syncthreads();
    // ---- weighted rows: this warp's columns
    if (tile0 < v_tiles) {
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        const float cA = row_c[mt * 16 + gid], cB = row_c[mt * 16 + gid + 8];
#pragma unroll
        for (int j = 0; j < NV; ++j) {
          o[j][mt][0] *= cA;
          o[j][mt][1] *= cA;
          o[j][mt][2] *= cB;
          o[j][mt][3] *= cB;
        }
      }
      const int mi = lane >> 3;
#pragma unroll
      for (int ks = 0; ks < PAGE / 16; ++ks) {
        uint32_t a[MT][3][4];
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
          for (int k = 0; k < 3; ++k)
            sp_ldmatrix_x4(sp_smem(Ps + ((size_t)k * ROWS + mt * 16 + (lane & 15)) * PP + ks * 16 + (lane >> 4) * 8), a[mt][k][0], a[mt][k][1], a[mt][k][2], a[mt][k][3]);
#pragma unroll
        for (int j = 0; j < NV; j += 2) {
          if (tile0 + j >= v_tiles) break;      // (dv is a multiple of 16: tiles come in pairs)
          uint32_t b0, b1, b2, b3;
          sp_ldmatrix_x4_trans(sp_smem(Ks + (size_t)(ks * 16 + (mi & 1) * 8 + (lane & 7)) * pitch + (tile0 + j + (mi >> 1)) * 8), b0, b1, b2, b3);
#pragma unroll
          for (int k = 2; k >= 0; --k)
#pragma unroll
            for (int mt = 0; mt < MT; ++mt) {
              sp_mma(o[j][mt], a[mt][k][0], a[mt][k][1], a[mt][k][2], a[mt][k][3], b0, b1);
              sp_mma(o[j + 1][mt], a[mt][k][0], a[mt][k][1], a[mt][k][2], a[mt][k][3], b2, b3);
            }
        }
      }
    }
    __syncthreads();                           // the page's rows and the weights are used up
    if (vi + 1 < v_end) load_page(page_at(vi + 1));
  }
#pragma unroll
  for (int mt = 0; mt < MT; ++mt) {
    const int rA = mt * 16 + gid, rB = rA + 8;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      if (tile0 + j >= v_tiles) break;
      const int c = 2 + (tile0 + j) * 8 + tig * 2;
      if (rA < heads) *reinterpret_cast<float2*>(out + rA * head_step + c) = make_float2(o[j][mt][0], o[j][mt][1]);
      if (rB < heads) *reinterpret_cast<float2*>(out + rB * head_step + c) = make_float2(o[j][mt][2], o[j][mt][3]);
    }
  }
  if (threadIdx.x < heads) {
    out[threadIdx.x * head_step] = row_m[threadIdx.x];
    out[threadIdx.x * head_step + 1] = row_l[threadIdx.x];
  }
}

// ---- small products per head for few tokens
template <typename TO, int NT, int KS>     // tiles of 8 tokens; warps that share K
__global__ void __launch_bounds__(256)
head_matmul_few_kernel(const float* __restrict__ a, int lda, int a_hs, const __nv_bfloat16* __restrict__ w, TO* __restrict__ out, int ldo,
                       int out_hs, int n_tokens, int K, int N) {
  __shared__ float red[KS > 1 ? 8 : 1][NT][32][4];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, gid = lane >> 2, tig = lane & 3;
  const int h = blockIdx.x, ks = warp % KS, n0 = (blockIdx.y * (8 / KS) + warp / KS) * 16;
  const __nv_bfloat16* wr[2] = {w + ((size_t)h * N + n0 + gid) * K, w + ((size_t)h * N + n0 + gid + 8) * K};
  const bool in[2] = {n0 + gid < N, n0 + gid + 8 < N};
  const int steps = (K + 31) / 32;
  uint4 wv[2][2];
  auto fetch = [&](int kb, int slot) {
    const int k = kb * 32 + tig * 8;
#pragma unroll
    for (int r = 0; r < 2; ++r) wv[slot][r] = in[r] && k < K ? *reinterpret_cast<const uint4*>(wr[r] + k) : make_uint4(0u, 0u, 0u, 0u);
  };
  pdl_launch_dependents();
  fetch(ks, 0);            // (nothing on the stream writes the weights: they are read ahead of the wait)
  fetch(ks + KS, 1);
  pdl_wait();
  float acc[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  for (int kb = ks, it = 0; kb < steps; kb += KS, ++it) {
    uint4 w0 = wv[0][0], w1 = wv[0][1];
    wv[0][0] = wv[1][0];
    wv[0][1] = wv[1][1];
    fetch(kb + 2 * KS, 1);
    const int k = kb * 32 + tig * 8;
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int t = i * 8 + gid;
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f), y = x;
      if (t < n_tokens && k < K) {
        const float* src = a + (size_t)t * lda + (size_t)h * a_hs + k;
        x = *reinterpret_cast<const float4*>(src);
        y = *reinterpret_cast<const float4*>(src + 4);
      }
      uint32_t b[4][3];
      sp_split(x.x, x.y, b[0][0], b[0][1], b[0][2]);
      sp_split(x.z, x.w, b[1][0], b[1][1], b[1][2]);
      sp_split(y.x, y.y, b[2][0], b[2][1], b[2][2]);
      sp_split(y.z, y.w, b[3][0], b[3][1], b[3][2]);
#pragma unroll
      for (int j = 2; j >= 0; --j) {
        sp_mma(acc[i], w0.x, w1.x, w0.y, w1.y, b[0][j], b[1][j]);
        sp_mma(acc[i], w0.z, w1.z, w0.w, w1.w, b[2][j], b[3][j]);
      }
    }
  }
  if constexpr (KS > 1) {
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) red[warp][i][lane][j] = acc[i][j];
    __syncthreads();
    if (ks != 0) return;
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        float s = 0.f;
#pragma unroll
        for (int x = 0; x < KS; ++x) s += red[warp + x][i][lane][j];
        acc[i][j] = s;
      }
  }
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + gid + (j >> 1) * 8, t = i * 8 + tig * 2 + (j & 1);
      if (n < N && t < n_tokens) out[(size_t)t * ldo + (size_t)h * out_hs + n] = from_f32<TO>(acc[i][j]);
    }
}

template <int MT, int NV>
static int launch_latent_decode(const float* q, const void* kcache, const int32_t* tok_pos, const int32_t* tok_seq, const int32_t* page_table,
                                int table_stride, int n_pages, int n_tokens, int H, int dc, int dv, float scale, int mask, int mask_size, int keep,
                                int n_splits, float* part, cudaStream_t stream) {
  const size_t smem = latent_decode_smem(MT, dc);
  auto kern = latent_decode_kernel<MT, NV>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) {
    set_error("latent_decode: %zu bytes of shared memory refused: %s", smem, cudaGetErrorString(e));
    return -2;
  }
  launch_pdl(pdl_bit_for_tokens(n_tokens), kern, dim3(n_tokens, (H + 16 * MT - 1) / (16 * MT), n_splits), dim3(LD_WARPS * 32), smem, stream, q,
             (const __nv_bfloat16*)kcache, tok_pos, tok_seq, page_table, table_stride, n_pages, H, dc, dv, scale, mask, mask_size, keep, n_splits, part);
  return 0;
}

static int latent_decode_tiles(int H, int dc) {      // tiles of heads a block, or 0 if its shared memory does not hold them
  constexpr size_t most = 227 * 1024;
  if (H > 16 && latent_decode_smem(2, dc) <= most) return 2;
  return latent_decode_smem(1, dc) <= most ? 1 : 0;
}

}  // namespace edgelm

using namespace edgelm;

// Heads that a block takes together for these sizes (rows of dc values of which the first dv are the value), or 0: not taken.
extern "C" int edgelm_latent_decode_takes(int H, int dc, int dv) {
  if (H < 1 || dc < 16 || dc % 16 != 0 || dv < 16 || dv % 16 != 0 || dv > dc || dv > 512) return 0;
  return 16 * latent_decode_tiles(H, dc);
}

// q [tokens][H][dc] float32, one token a sequence; kcache bfloat16 pages [page][64][dc].  part [tokens][H][n_splits][2 + dv] float32
// receives what `masked_attn_fold` merges.
extern "C" int edgelm_latent_decode(const float* q, const void* kcache, const int32_t* tok_pos, const int32_t* tok_seq, const int32_t* page_table,
                                    int table_stride, int n_pages, int n_tokens, int H, int dc, int dv, float scale, int mask, int mask_size, int keep,
                                    int n_splits, float* part, cudaStream_t stream) {
  if (n_tokens == 0) return 0;
  EL_REFUSE(edgelm_latent_decode_takes(H, dc, dv) > 0, "latent_decode: %d heads over rows of %d with values of %d", H, dc, dv);
  EL_REFUSE(mask == LD_MASK_CAUSAL || ((mask == LD_MASK_WINDOW || mask == LD_MASK_CHUNK) && mask_size >= 1), "latent_decode: mask %d of size %d", mask, mask_size);
  EL_REFUSE(keep >= 0 && (keep == 0 || mask == LD_MASK_WINDOW), "latent_decode: %d kept keys without a window", keep);
  EL_REFUSE(n_tokens > 0 && n_splits >= 1 && n_splits <= 64 && part != nullptr && (uintptr_t)part % 8 == 0 && (uintptr_t)q % 16 == 0 && (uintptr_t)kcache % 16 == 0,
            "latent_decode: %d splits, or unaligned rows", n_splits);
  const int mt = latent_decode_tiles(H, dc), nv = (dv / 8 + LD_WARPS - 1) / LD_WARPS;
  int rc = 0;
#define EL_LD(MT, NV) rc = launch_latent_decode<MT, NV>(q, kcache, tok_pos, tok_seq, page_table, table_stride, n_pages, n_tokens, H, dc, dv, scale, mask, mask_size, keep, n_splits, part, stream)
  if (mt == 2) { if (nv <= 2) EL_LD(2, 2); else if (nv <= 4) EL_LD(2, 4); else EL_LD(2, 8); }
  else { if (nv <= 2) EL_LD(1, 2); else if (nv <= 4) EL_LD(1, 4); else EL_LD(1, 8); }
#undef EL_LD
  if (rc) return rc;
  EL_LAUNCH_CHECK("latent_decode");
  return 0;
}

// 1 if `edgelm_head_matmul_few` takes these operands
extern "C" int edgelm_head_matmul_few_takes(const float* a, int lda, int a_hs, const void* w, int n_tokens, int K) {
  return n_tokens >= 1 && n_tokens <= 16 && K % 8 == 0 && lda % 4 == 0 && a_hs % 4 == 0 && (uintptr_t)a % 16 == 0 && (uintptr_t)w % 16 == 0 ? 1 : 0;
}

extern "C" int edgelm_head_matmul_few(const float* a, int lda, int a_hs, const void* w, void* out, int out_dtype, int ldo, int out_hs, int n_tokens,
                                      int H, int K, int N, cudaStream_t stream) {
  if (n_tokens == 0) return 0;
  EL_REFUSE(edgelm_head_matmul_few_takes(a, lda, a_hs, w, n_tokens, K) && H > 0 && N > 0, "head_matmul_few: %d tokens, %d heads, K %d, N %d", n_tokens, H, K, N);
  const int steps = (K + 31) / 32, ks = steps >= 8 ? 8 : (steps >= 4 ? 4 : (steps >= 2 ? 2 : 1));
  const dim3 grid(H, ((N + 15) / 16 + 8 / ks - 1) / (8 / ks)), block(256);
  const int bit = pdl_bit_for_tokens(n_tokens);
#define EL_HF(TO, NT, KS) launch_pdl(bit, head_matmul_few_kernel<TO, NT, KS>, grid, block, (size_t)0, stream, a, lda, a_hs, (const __nv_bfloat16*)w, (TO*)out, ldo, out_hs, n_tokens, K, N)
#define EL_HFK(TO, NT) do { if (ks == 8) EL_HF(TO, NT, 8); else if (ks == 4) EL_HF(TO, NT, 4); else if (ks == 2) EL_HF(TO, NT, 2); else EL_HF(TO, NT, 1); } while (0)
  if (out_dtype == DT_F32) { if (n_tokens <= 8) EL_HFK(float, 1); else EL_HFK(float, 2); }
  else if (out_dtype == DT_BF16) { if (n_tokens <= 8) EL_HFK(__nv_bfloat16, 1); else EL_HFK(__nv_bfloat16, 2); }
  else EL_REFUSE(false, "head_matmul_few: unknown dtype code %d", out_dtype);
#undef EL_HFK
#undef EL_HF
  EL_LAUNCH_CHECK("head_matmul_few");
  return 0;
}
