// Attention of many new tokens over bfloat16 keys and values on the tensor cores, for designs whose scores AND softmax
// weights are float32: the float32 operand of each product is written as the sum of three bfloat16 terms (8 + 8 + 8 of its 24
// mantissa bits), each of which the tensor cores multiply exactly with the bfloat16 operand from the cache, sums in float32:
//
//   S = (q1 + q2 + q3) K^T        q float32 queries (after rotation), K bfloat16 rows
//   O += (p1 + p2 + p3) V         p float32 softmax weights, V bfloat16 rows
//
// so a score or an output differs from the float32 product of the same numbers by float32 rounding only, at three times
// the multiply-adds of a bfloat16 attention instead of the CUDA cores' rate.  Flash style: no score matrix reaches memory.
//
// grid (query tile, query head); a block of 4 warps (times NG groups) owns 64 consecutive new tokens of one sequence for one
// head, 16 rows a warp.  Keys and values are visited page by page (64 positions): all threads of a group copy the page's K
// and V rows of the head's kv head into shared memory with 16-byte cp.async into rows padded by 16 bytes, two stages; K
// fragments by ldmatrix, V fragments by ldmatrix.trans; scale, mask, running maximum and sum per row in float32,
// scores in units of log 2.  With NG warp groups a block, group i visits the pages i, i + NG, ... with stages and a named
// barrier of its own; the groups' partial (maximum, sum, output) are merged in shared memory in the order of the groups.
// An optional gate per (token, head) multiplies the head's output by its sigmoid before the rounding; an optional sink per head is
// one more term exp(sink_h) of the softmax's denominator, without a key, a value or the scale.
// (or, with a gate per channel, every channel by its own).
// Masks as in the CUDA-core kernels: causal, a sliding window (with the sequence's first `keep` keys kept visible), or chunks; pages before the first key that the tile's first row sees
// are not visited.  Keys and values come from the cache's pages (the page table's rows are the step's sequences) or, without a page
// table, from the step's own rows (every sequence of the step then starts at position 0).
// Takes key head sizes 32, 64, 96, 128 over value head sizes of these that are not larger.
#include <math_constants.h>

#include "mma_split.cuh"

namespace edgelm {

enum : int { SP_MASK_CAUSAL = 0, SP_MASK_WINDOW = 1, SP_MASK_CHUNK = 2 };

// the first key that a query at `pos` sees
__device__ __forceinline__ int sp_first_key(int pos, int mask, int size) {
  if (mask == SP_MASK_WINDOW) return max(0, pos - size + 1);
  if (mask == SP_MASK_CHUNK) return (pos / size) * size;
  return 0;
}

constexpr int SP_WARPS = 4;
constexpr int SP_ROWS = 16 * SP_WARPS;  // new tokens per block

template <int HDT, int VDT, int NG>  // key and value head sizes / 16 (even); warp groups that share the pages of a tile
__global__ void __launch_bounds__(SP_WARPS * 32 * NG)
attn_prefill_split_kernel(const float* __restrict__ q, int ldq, __nv_bfloat16* __restrict__ out, int ldo,
                          const __nv_bfloat16* __restrict__ kcache, const __nv_bfloat16* __restrict__ vcache,
                          const int32_t* __restrict__ page_table, int table_stride, const int32_t* __restrict__ tile_seq,
                          const int32_t* __restrict__ tile_tok0, const int32_t* __restrict__ tile_ntok,
                          const int32_t* __restrict__ tile_pos0, int nh, int nkv, float scale, const float* __restrict__ gate, int ldg,
                          int mask, int mask_size, const float* __restrict__ sink, int keep, int gate_ch) {
  constexpr int HD = HDT * 16, VD = VDT * 16;
  constexpr int PITCH = HD + 8, VPITCH = VD + 8;   // elements: 16 bytes of padding per row
  constexpr int CHUNKS = HD / 8, VCHUNKS = VD / 8; // 16-byte chunks per row
  extern __shared__ __align__(16) uint8_t sp_raw[];
  constexpr int STAGE = PAGE * (PITCH + VPITCH);
  const int group = threadIdx.x / (SP_WARPS * 32), gtid = threadIdx.x % (SP_WARPS * 32);
  __nv_bfloat16* sm = reinterpret_cast<__nv_bfloat16*>(sp_raw) + (size_t)group * 2 * STAGE;  // this group's [2 stages][K: 64 x PITCH | V: 64 x VPITCH]

  const int tile = blockIdx.x, head = blockIdx.y;
  const int g = nh / nkv, kvh = head / g;
  const int lane = threadIdx.x & 31, warp = (threadIdx.x >> 5) % SP_WARPS, gid = lane >> 2, tig = lane & 3;
  const int seq = tile_seq[tile], tok0 = tile_tok0[tile], ntok = tile_ntok[tile], pos0 = tile_pos0[tile];
  const int32_t* pages = page_table ? page_table + (size_t)seq * table_stride : nullptr;
  const int nkeys_block = pos0 + ntok;      // keys 0 .. pos0 + ntok - 1
  const int n_pages = (nkeys_block + PAGE - 1) / PAGE;
  const int rowA = warp * 16 + gid, rowB = rowA + 8;      // this lane's two rows (token index inside the tile)
  const int limA = rowA < ntok ? pos0 + rowA : -1;         // last key a row may see; -1: no such row
  const int limB = rowB < ntok ? pos0 + rowB : -1;
  const int warp_limit = min(ntok - 1, warp * 16 + 15) >= warp * 16 ? pos0 + min(ntok - 1, warp * 16 + 15) : -1;
  const int warp_min_limit = warp * 16 < ntok ? pos0 + warp * 16 : -1;   // what the warp's first row sees: pages up to here need no mask
  // what the mask leaves out in front: per row, and for the warp's first (the smallest) and last row
  const int firstA = sp_first_key(max(limA, 0), mask, mask_size), firstB = sp_first_key(max(limB, 0), mask, mask_size);
  const int warp_first = sp_first_key(max(warp_min_limit, 0), mask, mask_size), warp_last_first = sp_first_key(max(warp_limit, 0), mask, mask_size);
  // the pages to visit: those of the kept keys that lie ahead of the window's first, then the window's
  const int first_page = sp_first_key(pos0, mask, mask_size) / PAGE, kept_pages = min(first_page, (keep + PAGE - 1) / PAGE);
  const int n_visit = kept_pages + n_pages - first_page;
  auto page_at = [&](int i) { return i < kept_pages ? i : first_page + i - kept_pages; };
  const float scale2 = scale * 1.4426950408889634f;                     // scores in units of log 2

  auto load_page = [&](int pg, int stage) {
    const int page = pages ? pages[pg] : 0;
    // the page's first row of this head and the rows' pitch, in rows (own rows: position p is packed row tok0 - pos0 + p)
    const size_t row0 = pages ? ((size_t)max(page, 0) * nkv + kvh) * PAGE : (size_t)(tok0 - pos0 + pg * PAGE) * nkv + kvh;
    const int pitch = pages ? 1 : nkv;
    const __nv_bfloat16* kp = kcache + row0 * HD;
    const __nv_bfloat16* vp = vcache + row0 * VD;
    const int valid = page >= 0 ? min(PAGE, nkeys_block - pg * PAGE) : 0;     // (a page that is not there: zeros, never read)
    __nv_bfloat16* ks = sm + stage * STAGE;
    __nv_bfloat16* vs = ks + PAGE * PITCH;
    for (int i = gtid; i < PAGE * CHUNKS; i += SP_WARPS * 32) {
      const int r = i / CHUNKS, c = i - r * CHUNKS;
      const int bytes = r < valid ? 16 : 0;   // rows past the last key: zero fill, nothing is read
      sp_cp16(sp_smem(ks + r * PITCH + c * 8), bytes ? kp + (size_t)r * pitch * HD + c * 8 : kcache, bytes);
      if (VD == HD) sp_cp16(sp_smem(vs + r * VPITCH + c * 8), bytes ? vp + (size_t)r * pitch * VD + c * 8 : vcache, bytes);
    }
    if (VD != HD)
      for (int i = gtid; i < PAGE * VCHUNKS; i += SP_WARPS * 32) {
        const int r = i / VCHUNKS, c = i - r * VCHUNKS;
        const int bytes = r < valid ? 16 : 0;
        sp_cp16(sp_smem(vs + r * VPITCH + c * 8), bytes ? vp + (size_t)r * pitch * VD + c * 8 : vcache, bytes);
      }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };

  // Q fragments for the whole kernel: three terms of every float32 query value
  uint32_t qa[3][HDT][4];
  {
    const float* qA = q + (size_t)(tok0 + min(rowA, ntok - 1)) * ldq + head * HD;
    const float* qB = q + (size_t)(tok0 + min(rowB, ntok - 1)) * ldq + head * HD;
#pragma unroll
    for (int ks = 0; ks < HDT; ++ks) {
      const int d = ks * 16 + tig * 2;
      const float2 a0 = rowA < ntok ? *reinterpret_cast<const float2*>(qA + d) : make_float2(0.f, 0.f);
      const float2 b0 = rowB < ntok ? *reinterpret_cast<const float2*>(qB + d) : make_float2(0.f, 0.f);
      const float2 a1 = rowA < ntok ? *reinterpret_cast<const float2*>(qA + d + 8) : make_float2(0.f, 0.f);
      const float2 b1 = rowB < ntok ? *reinterpret_cast<const float2*>(qB + d + 8) : make_float2(0.f, 0.f);
      sp_split(a0.x, a0.y, qa[0][ks][0], qa[1][ks][0], qa[2][ks][0]);
      sp_split(b0.x, b0.y, qa[0][ks][1], qa[1][ks][1], qa[2][ks][1]);
      sp_split(a1.x, a1.y, qa[0][ks][2], qa[1][ks][2], qa[2][ks][2]);
      sp_split(b1.x, b1.y, qa[0][ks][3], qa[1][ks][3], qa[2][ks][3]);
    }
  }
  float o[VD / 8][4];
#pragma unroll
  for (int i = 0; i < VD / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float mA = -CUDART_INF_F, mB = -CUDART_INF_F, lA = 0.f, lB = 0.f;

  auto group_sync = [&]() {   // the 128 threads of this group (barrier 0 is __syncthreads)
    if (NG == 1) __syncthreads();
    else asm volatile("bar.sync %0, %1;" ::"r"(group + 1), "r"(SP_WARPS * 32) : "memory");
  };
  if (group < n_visit) load_page(page_at(group), 0);
  for (int vi = group, it = 0; vi < n_visit; vi += NG, ++it) {
    const int stage = it & 1, pg = page_at(vi);
    if (vi + NG < n_visit) {
      load_page(page_at(vi + NG), stage ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    group_sync();
    if (pg * PAGE <= warp_limit && (pg * PAGE + PAGE - 1 >= warp_first || pg * PAGE < keep)) {   // else: no row of this warp sees this page
      const __nv_bfloat16* ks = sm + stage * STAGE;
      const __nv_bfloat16* vs = ks + PAGE * PITCH;
      // ---- S = Q K^T : 8 tiles of 8 keys, three query terms against every key fragment
      float s[8][4];
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
        s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f;
#pragma unroll
        for (int ks2 = 0; ks2 < HDT; ks2 += 2) {
          // four 8x8 matrices: (keys nt*8.., d block ks2*16), (.., +8), (.., (ks2+1)*16), (.., +8)
          const int mi = lane >> 3;
          const uint32_t addr = sp_smem(ks + (nt * 8 + (lane & 7)) * PITCH + (ks2 + (mi >> 1)) * 16 + (mi & 1) * 8);
          uint32_t b0, b1, b2, b3;
          sp_ldmatrix_x4(addr, b0, b1, b2, b3);
#pragma unroll
          for (int t = 2; t >= 0; --t) {      // (the small terms first)
            sp_mma(s[nt], qa[t][ks2][0], qa[t][ks2][1], qa[t][ks2][2], qa[t][ks2][3], b0, b1);
            sp_mma(s[nt], qa[t][ks2 + 1][0], qa[t][ks2 + 1][1], qa[t][ks2 + 1][2], qa[t][ks2 + 1][3], b2, b3);
          }
        }
      }
      // ---- scale, mask, running max and sum (float32), scores in units of log 2
      const bool masked = pg * PAGE + PAGE - 1 > warp_min_limit || (pg * PAGE < warp_last_first && pg * PAGE + PAGE > keep);
      float mxA = -CUDART_INF_F, mxB = -CUDART_INF_F;
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
        const int key = pg * PAGE + nt * 8 + tig * 2;
        if (masked) {
          s[nt][0] = (key >= firstA || key < keep) && key <= limA ? s[nt][0] * scale2 : -CUDART_INF_F;
          s[nt][1] = (key + 1 >= firstA || key + 1 < keep) && key + 1 <= limA ? s[nt][1] * scale2 : -CUDART_INF_F;
          s[nt][2] = (key >= firstB || key < keep) && key <= limB ? s[nt][2] * scale2 : -CUDART_INF_F;
          s[nt][3] = (key + 1 >= firstB || key + 1 < keep) && key + 1 <= limB ? s[nt][3] * scale2 : -CUDART_INF_F;
        } else {
          s[nt][0] *= scale2;
          s[nt][1] *= scale2;
          s[nt][2] *= scale2;
          s[nt][3] *= scale2;
        }
        mxA = fmaxf(mxA, fmaxf(s[nt][0], s[nt][1]));
        mxB = fmaxf(mxB, fmaxf(s[nt][2], s[nt][3]));
      }
      mxA = fmaxf(mxA, __shfl_xor_sync(0xffffffffu, mxA, 1));
      mxA = fmaxf(mxA, __shfl_xor_sync(0xffffffffu, mxA, 2));
      mxB = fmaxf(mxB, __shfl_xor_sync(0xffffffffu, mxB, 1));
      mxB = fmaxf(mxB, __shfl_xor_sync(0xffffffffu, mxB, 2));
      const float nmA = fmaxf(mA, mxA), nmB = fmaxf(mB, mxB);
      const float refA = nmA == -CUDART_INF_F ? 0.f : nmA, refB = nmB == -CUDART_INF_F ? 0.f : nmB;  // a row that sees no key yet
      const float corrA = exp2f(mA - refA), corrB = exp2f(mB - refB);  // exp2(-inf) = 0 on the first page
      float sumA = 0.f, sumB = 0.f;
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
        s[nt][0] = exp2f(s[nt][0] - refA);
        s[nt][1] = exp2f(s[nt][1] - refA);
        s[nt][2] = exp2f(s[nt][2] - refB);
        s[nt][3] = exp2f(s[nt][3] - refB);
        sumA += s[nt][0] + s[nt][1];
        sumB += s[nt][2] + s[nt][3];
      }
      sumA += __shfl_xor_sync(0xffffffffu, sumA, 1);
      sumA += __shfl_xor_sync(0xffffffffu, sumA, 2);
      sumB += __shfl_xor_sync(0xffffffffu, sumB, 1);
      sumB += __shfl_xor_sync(0xffffffffu, sumB, 2);
      lA = lA * corrA + sumA;
      lB = lB * corrB + sumB;
      mA = nmA;
      mB = nmB;
      if (__any_sync(0xffffffffu, corrA != 1.f || corrB != 1.f)) {   // some row's maximum moved: rescale what is gathered
#pragma unroll
        for (int i = 0; i < VD / 8; ++i) {
          o[i][0] *= corrA;
          o[i][1] *= corrA;
          o[i][2] *= corrB;
          o[i][3] *= corrB;
        }
      }
      // ---- O += P V : 4 steps of 16 keys, three terms of every weight against every value fragment
#pragma unroll
      for (int kt = 0; kt < 4; ++kt) {
        uint32_t a[3][4];
        sp_split(s[2 * kt][0], s[2 * kt][1], a[0][0], a[1][0], a[2][0]);
        sp_split(s[2 * kt][2], s[2 * kt][3], a[0][1], a[1][1], a[2][1]);
        sp_split(s[2 * kt + 1][0], s[2 * kt + 1][1], a[0][2], a[1][2], a[2][2]);
        sp_split(s[2 * kt + 1][2], s[2 * kt + 1][3], a[0][3], a[1][3], a[2][3]);
#pragma unroll
        for (int dt = 0; dt < VD / 8; dt += 2) {
          // transposed 8x8 matrices: (keys kt*16.., d block dt), (keys +8, dt), (keys kt*16.., dt+1), (keys +8, dt+1)
          const int mi = lane >> 3;
          const uint32_t addr = sp_smem(vs + (kt * 16 + (mi & 1) * 8 + (lane & 7)) * VPITCH + (dt + (mi >> 1)) * 8);
          uint32_t b0, b1, b2, b3;
          sp_ldmatrix_x4_trans(addr, b0, b1, b2, b3);
#pragma unroll
          for (int t = 2; t >= 0; --t) {
            sp_mma(o[dt], a[t][0], a[t][1], a[t][2], a[t][3], b0, b1);
            sp_mma(o[dt + 1], a[t][0], a[t][1], a[t][2], a[t][3], b2, b3);
          }
        }
      }
    }
    group_sync();  // this stage is free for the page after next
  }
  if (NG > 1) {
    // ---- merge the groups: groups 1.. leave (max, sum, output) in shared memory, group 0 folds them in order
    __syncthreads();
    float* mg = reinterpret_cast<float*>(sp_raw);            // [NG - 1][64 rows][VD + 2]
    constexpr int MP = VD + 2;
    if (group > 0) {
      float* a = mg + ((size_t)(group - 1) * SP_ROWS + rowA) * MP;
      float* b = mg + ((size_t)(group - 1) * SP_ROWS + rowB) * MP;
#pragma unroll
      for (int dt = 0; dt < VD / 8; ++dt) {
        a[dt * 8 + tig * 2] = o[dt][0];
        a[dt * 8 + tig * 2 + 1] = o[dt][1];
        b[dt * 8 + tig * 2] = o[dt][2];
        b[dt * 8 + tig * 2 + 1] = o[dt][3];
      }
      if (tig == 0) {
        a[VD] = mA;
        a[VD + 1] = lA;
        b[VD] = mB;
        b[VD + 1] = lB;
      }
    }
    __syncthreads();
    if (group > 0) return;
    for (int gsrc = 1; gsrc < NG; ++gsrc) {
      const float* a = mg + ((size_t)(gsrc - 1) * SP_ROWS + rowA) * MP;
      const float* b = mg + ((size_t)(gsrc - 1) * SP_ROWS + rowB) * MP;
      const float nmA = fmaxf(mA, a[VD]), nmB = fmaxf(mB, b[VD]);
      const float refA = nmA == -CUDART_INF_F ? 0.f : nmA, refB = nmB == -CUDART_INF_F ? 0.f : nmB;
      const float fA0 = exp2f(mA - refA), fA1 = exp2f(a[VD] - refA), fB0 = exp2f(mB - refB), fB1 = exp2f(b[VD] - refB);
      lA = lA * fA0 + a[VD + 1] * fA1;
      lB = lB * fB0 + b[VD + 1] * fB1;
      mA = nmA;
      mB = nmB;
#pragma unroll
      for (int dt = 0; dt < VD / 8; ++dt) {
        o[dt][0] = o[dt][0] * fA0 + a[dt * 8 + tig * 2] * fA1;
        o[dt][1] = o[dt][1] * fA0 + a[dt * 8 + tig * 2 + 1] * fA1;
        o[dt][2] = o[dt][2] * fB0 + b[dt * 8 + tig * 2] * fB1;
        o[dt][3] = o[dt][3] * fB0 + b[dt * 8 + tig * 2 + 1] * fB1;
      }
    }
  }
  float fixA = 1.f, fixB = 1.f;
  if (sink != nullptr) {      // the sink: one more term of the denominator (in units of log 2, as the maxima are)
    const float s2 = sink[head] * 1.4426950408889634f, nmA = fmaxf(mA, s2), nmB = fmaxf(mB, s2);
    fixA = exp2f(mA - nmA);
    fixB = exp2f(mB - nmB);
    lA = lA * fixA + exp2f(s2 - nmA);
    lB = lB * fixB + exp2f(s2 - nmB);
  }
  float invA = lA > 0.f ? fixA / lA : 0.f, invB = lB > 0.f ? fixB / lB : 0.f;
  if (gate != nullptr && !gate_ch) {      // the head's output gate: sigmoid of its logit
    if (rowA < ntok) invA *= 1.0f / (1.0f + expf(-gate[(size_t)(tok0 + rowA) * ldg + head]));
    if (rowB < ntok) invB *= 1.0f / (1.0f + expf(-gate[(size_t)(tok0 + rowB) * ldg + head]));
  }
  if (gate != nullptr && gate_ch) {     // a gate per channel: all of a row's numbers are requested before the first is used
    float ga[VD / 8][4];
    const float* gA = gate + (size_t)(tok0 + min(rowA, ntok - 1)) * ldg + head * VD + tig * 2;
    const float* gB = gate + (size_t)(tok0 + min(rowB, ntok - 1)) * ldg + head * VD + tig * 2;
#pragma unroll
    for (int dt = 0; dt < VD / 8; ++dt) {
      ga[dt][0] = gA[dt * 8];
      ga[dt][1] = gA[dt * 8 + 1];
      ga[dt][2] = gB[dt * 8];
      ga[dt][3] = gB[dt * 8 + 1];
    }
#pragma unroll
    for (int dt = 0; dt < VD / 8; ++dt)
#pragma unroll
      for (int j = 0; j < 4; ++j) o[dt][j] *= 1.0f / (1.0f + expf(-ga[dt][j]));
  }
#pragma unroll
  for (int dt = 0; dt < VD / 8; ++dt) {
    const int d = head * VD + dt * 8 + tig * 2;
    if (rowA < ntok) {
      const __nv_bfloat162 v = __floats2bfloat162_rn(o[dt][0] * invA, o[dt][1] * invA);
      *reinterpret_cast<__nv_bfloat162*>(out + (size_t)(tok0 + rowA) * ldo + d) = v;
    }
    if (rowB < ntok) {
      const __nv_bfloat162 v = __floats2bfloat162_rn(o[dt][2] * invB, o[dt][3] * invB);
      *reinterpret_cast<__nv_bfloat162*>(out + (size_t)(tok0 + rowB) * ldo + d) = v;
    }
  }
}

struct SplitArgs {
  const float* q;
  int ldq;
  void* out;
  int ldo;
  const void *kc, *vc;
  const int32_t* page_table;
  int table_stride;
  const int32_t *tile_seq, *tile_tok0, *tile_ntok, *tile_pos0;
  int n_tiles, nh, nkv;
  float scale;
  const float* gate;
  int ldg, mask, mask_size;
  const float* sink;
  int keep, gate_ch;
};

template <int HDT, int VDT, int NG>
static int launch_split_ng(const SplitArgs& a, cudaStream_t stream) {
  constexpr int HD = HDT * 16, VD = VDT * 16;
  const size_t stages = (size_t)NG * 2 * PAGE * (HD + 8 + VD + 8) * 2, merge = (size_t)(NG - 1) * SP_ROWS * (VD + 2) * 4;
  const size_t smem = stages > merge ? stages : merge;
  auto kern = attn_prefill_split_kernel<HDT, VDT, NG>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) {
    set_error("attn_prefill_split: %zu bytes of shared memory refused: %s", smem, cudaGetErrorString(e));
    return -2;
  }
  kern<<<dim3(a.n_tiles, a.nh), SP_WARPS * 32 * NG, smem, stream>>>(a.q, a.ldq, (__nv_bfloat16*)a.out, a.ldo, (const __nv_bfloat16*)a.kc, (const __nv_bfloat16*)a.vc,
                                                                     a.page_table, a.table_stride, a.tile_seq, a.tile_tok0, a.tile_ntok, a.tile_pos0, a.nh, a.nkv,
                                                                     a.scale, a.gate, a.ldg, a.mask, a.mask_size, a.sink, a.keep, a.gate_ch);
  return 0;
}

template <int HDT, int VDT>
static int launch_split(int groups, const SplitArgs& a, cudaStream_t stream) {
  return groups == 2 ? launch_split_ng<HDT, VDT, 2>(a, stream) : launch_split_ng<HDT, VDT, 1>(a, stream);
}

static bool split_size(int hd) { return hd == 32 || hd == 64 || hd == 96 || hd == 128; }

}  // namespace edgelm

using namespace edgelm;

// Tokens per tile that the host must cut sequences into for this kernel.
extern "C" int edgelm_attn_prefill_split_tile_tokens() { return SP_ROWS; }

// 1 if the kernel takes these key and value head sizes, else 0.
extern "C" int edgelm_attn_prefill_split_takes(int dk, int dv) { return split_size(dk) && split_size(dv) && dv <= dk ? 1 : 0; }

// q [tokens][nh dk] float32 (row pitch ldq), out [tokens][nh dv] bfloat16 (row pitch ldo); keys and values bfloat16: the cache's
// pages [page][kv head][64][dk or dv] with `page_table` rows for the step's sequences (tile_seq indexes them), or, with `page_table`
// null, the step's own rows [token][kv head][dk or dv] (every sequence of the step starts at position 0); tiles of at most 64 new
// tokens of one sequence each.  `mask` 0 causal, 1 a window of `mask_size` keys, 2 chunks of `mask_size` positions.  `sink` (or
// null): float32 [nh].  `keep`: with a window, the sequence's first keys that stay visible.  `gate` (or null): float32 with row pitch
// ldg, a number per head (`gate_ch` 0) or per channel (`gate_ch` = dv).  `max_keys`: the most keys a tile attends over
// (a hint for how many warp groups share a tile's pages).
extern "C" int edgelm_attn_prefill_split(const float* q, int ldq, void* out, int ldo, const void* kcache, const void* vcache,
                                         const int32_t* page_table, int table_stride, const int32_t* tile_seq, const int32_t* tile_tok0,
                                         const int32_t* tile_ntok, const int32_t* tile_pos0, int n_tiles, int nh, int nkv, int dk, int dv,
                                         float scale, int mask, int mask_size, const float* sink, const float* gate, int ldg, int max_keys,
                                         int keep, int gate_ch, cudaStream_t stream) {
  if (n_tiles == 0) return 0;
  EL_REFUSE(nh > 0 && nkv > 0 && nh % nkv == 0, "attn_prefill_split: %d query heads are not a multiple of %d key/value heads", nh, nkv);
  EL_REFUSE(edgelm_attn_prefill_split_takes(dk, dv), "attn_prefill_split: head sizes %d / %d (takes 32, 64, 96, 128, values not larger than keys)", dk, dv);
  EL_REFUSE(ldq % 2 == 0 && ldo % 2 == 0 && (uintptr_t)q % 8 == 0 && (uintptr_t)out % 4 == 0, "attn_prefill_split: rows must be 8- and 4-byte aligned");
  EL_REFUSE((uintptr_t)kcache % 16 == 0 && (uintptr_t)vcache % 16 == 0, "attn_prefill_split: keys and values must be 16-byte aligned");
  EL_REFUSE(mask == SP_MASK_CAUSAL || ((mask == SP_MASK_WINDOW || mask == SP_MASK_CHUNK) && mask_size >= 1), "attn_prefill_split: mask %d of size %d", mask, mask_size);
  EL_REFUSE(keep >= 0 && (keep == 0 || mask == SP_MASK_WINDOW) && (gate_ch == 0 || gate_ch == dv), "attn_prefill_split: %d kept keys, a gate of %d channels", keep, gate_ch);
  EL_REFUSE(n_tiles > 0 && nh <= 65535, "attn_prefill_split: bad grid");
  const long long blocks = (long long)n_tiles * nh;
  if (mask != SP_MASK_CAUSAL && max_keys > mask_size + keep + SP_ROWS) max_keys = mask_size + keep + SP_ROWS;
  const int groups = ((max_keys + PAGE - 1) / PAGE >= 6 && blocks < 4 * 148 * 2) ? 2 : 1;
  const SplitArgs a{q, ldq, out, ldo, kcache, vcache, page_table, table_stride, tile_seq, tile_tok0, tile_ntok, tile_pos0, n_tiles, nh, nkv, scale,
                    gate, ldg, mask, mask_size, sink, keep, gate_ch};
  int rc = 0;
#define EL_SP(H, V) case (H) * 16 + (V): rc = launch_split<H, V>(groups, a, stream); break;
  switch (dk / 16 * 16 + dv / 16) {
    EL_SP(2, 2) EL_SP(4, 2) EL_SP(4, 4) EL_SP(6, 2) EL_SP(6, 4) EL_SP(6, 6) EL_SP(8, 2) EL_SP(8, 4) EL_SP(8, 6) EL_SP(8, 8)
  }
#undef EL_SP
  if (rc) return rc;
  EL_LAUNCH_CHECK("attn_prefill_split");
  return 0;
}
