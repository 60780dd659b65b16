// Attention of few rows of grouped heads on tensor cores (mma.sync m16n8k16), keys split over the warps of a CTA.
//
// The kernel of `attn_decode_mma.cu` gives every warp 16 of 64 (row, head) pairs and the whole key tile. A decoded row brings only the
// heads of one group (4 .. 8 of them), so one warp does all the arithmetic there and its latencies are the kernel's time, the more so
// where scores are softcapped. Here M is 16 pairs and a 64-key tile is cut over the four warps, 16 keys each: every warp keeps a softmax of
// its own (maximum, sum, unnormalised output), the four are joined once at the end. K and V stream through two cp.async stages.
//
// POOL: the means of the blocks before a row's window come first in the list of keys that the splits share, in tiles of their own (a tile of
// means is gathered row by row, since they lie in the pages of their blocks' last positions).
//
// grid (segments x row groups, kv heads, key splits). Rows see the keys up to their own, of a window or a chunk (`first_key`), scores may be
// softcapped, softmax weights enter the PV product as a bf16 value plus its bf16 remainder. A CTA leaves the record of its split
// (unnormalised o, maximum, sum) for the merges of `latent.cu`; the order of the joins is fixed, so results do not depend on scheduling.
#include "api.h"
#include "common.cuh"

namespace fb {

constexpr int DK_M = 16, DK_KEYS = 64, DK_WARPS = 4, DK_THREADS = DK_WARPS * 32;

__device__ __forceinline__ void dk_cp16(void* smem, const void* gmem, bool valid) {
  const int sz = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(smem)), "l"(gmem), "r"(sz) : "memory");
}
__device__ __forceinline__ void dk_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void dk_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void dk_ldsm(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void dk_ldsm_t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void dk_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

template <int HD, bool POOL>
__global__ void __launch_bounds__(DK_THREADS)
attn_decode_keys_kernel(float* __restrict__ o_part, float* __restrict__ ml_part, const __nv_bfloat16* __restrict__ q,
                        const __nv_bfloat16* __restrict__ k_cache, const __nv_bfloat16* __restrict__ v_cache, const int* __restrict__ seg_slot,
                        const int* __restrict__ seg_row0, const int* __restrict__ seg_nrows, const int* __restrict__ row_kvlen,
                        const int* __restrict__ block_table, int max_blocks, int kv_block, int nq, int nkv, int nsplit, int groups_per_seg,
                        int row_first, float scale_log2, int window, int chunk, float cap_log2, const __nv_bfloat16* __restrict__ k_mean,
                        const __nv_bfloat16* __restrict__ v_mean, int pool, int* status) {
  constexpr int LD = HD + 8;                    // padded row (elements): conflict-free ldmatrix
  constexpr int CPR = HD / 8;                   // 16-byte pieces per row
  extern __shared__ __align__(16) unsigned char dk_smem[];
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(dk_smem);           // [M][LD]
  __nv_bfloat16* sK = sQ + DK_M * LD;                                       // [2][KEYS][LD]
  __nv_bfloat16* sV = sK + 2 * DK_KEYS * LD;                                // [2][KEYS][LD]
  pdl_wait();
  const int G = nq / nkv, RG = DK_M / G;        // heads per kv head, rows of a segment per CTA
  const int seg = blockIdx.x / groups_per_seg, r_first = blockIdx.x % groups_per_seg * RG;
  const int kvh = blockIdx.y, split = blockIdx.z;
  const int n = seg_nrows[seg];
  if (r_first >= n) return;
  const int rows_here = min(RG, n - r_first), valid_m = rows_here * G;
  const int row0 = seg_row0[seg] - row_first + r_first;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, tid = threadIdx.x;
  const int* bt = block_table + (size_t)seg_slot[seg] * max_blocks;
  // rows of a segment follow one another: the last one sees the latest key, the first one the earliest
  const int kv_end = row_kvlen[row0 + rows_here - 1];
  const int first_lo = first_key(row_kvlen[row0] - 1, window, chunk), kv_lo = first_lo / DK_KEYS * DK_KEYS;
  // list of keys: place u < shift is mean u (those of the last row's blocks), the others are token u - shift + kv_lo
  const int nb = POOL ? first_key(kv_end - 1, window, 0) / pool : 0, shift = POOL ? (nb + DK_KEYS - 1) / DK_KEYS * DK_KEYS : 0;
  const int at0 = POOL ? 0 : kv_lo, list_end = POOL ? shift + kv_end - kv_lo : kv_end;
  int per = (list_end - at0 + nsplit - 1) / nsplit;
  per = (per + DK_KEYS - 1) / DK_KEYS * DK_KEYS;
  const int lo = at0 + split * per, hi = min(list_end, lo + per);
  // (row, head) pair m of this CTA -> its record
  auto record = [&](int m) { return ((size_t)(row0 + m / G) * nq + kvh * G + m % G) * nsplit + split; };
  if (lo >= hi) {                               // an empty split: the merge skips it
    if (tid < valid_m) { ml_part[record(tid) * 2] = -INFINITY; ml_part[record(tid) * 2 + 1] = 0.f; }
    return;
  }
  for (int c = tid; c < DK_M * CPR; c += DK_THREADS) {
    const int m = c / CPR, cc = c % CPR;
    const bool ok = m < valid_m;
    dk_cp16(sQ + m * LD + cc * 8, q + ((size_t)(row0 + (ok ? m / G : 0)) * nq + kvh * G + (ok ? m % G : 0)) * HD + cc * 8, ok);
  }
  auto load_tile = [&](int t0, int stage) {     // a tile lies in one page: both start on multiples of 64 keys
    if constexpr (POOL) {
      if (t0 < shift) {
        const int per_page = (kv_block + pool - 1) / pool;
#pragma unroll 4
        for (int i = 0; i < DK_KEYS * CPR / DK_THREADS; ++i) {
          const int c = tid + i * DK_THREADS, r = c / CPR, cc = c % CPR, e = (t0 + r) * pool + pool - 1;
          const int blk = t0 + r < nb ? bt[e / kv_block] : -1;
          if (blk < 0 && t0 + r < nb) set_status(status, ST_BOUNDS);
          const size_t off = blk < 0 ? 0 : (((size_t)blk * per_page + e % kv_block / pool) * nkv + kvh) * HD + cc * 8;
          dk_cp16(sK + (stage * DK_KEYS + r) * LD + cc * 8, k_mean + off, blk >= 0);
          dk_cp16(sV + (stage * DK_KEYS + r) * LD + cc * 8, v_mean + off, blk >= 0);
        }
        dk_commit();
        return;
      }
      t0 += kv_lo - shift;
    }
    const int blk = bt[t0 / kv_block];
    if (blk < 0 && tid == 0) set_status(status, ST_BOUNDS);
    const int live = blk < 0 ? 0 : min(DK_KEYS, (POOL ? min(kv_end, hi + kv_lo - shift) : hi) - t0);
    const size_t base = blk < 0 ? 0 : (((size_t)blk * kv_block + t0 % kv_block) * nkv + kvh) * HD;
    const size_t ld = (size_t)nkv * HD;
#pragma unroll
    for (int i = 0; i < DK_KEYS * CPR / DK_THREADS; ++i) {
      const int c = tid + i * DK_THREADS, r = c / CPR, cc = c % CPR;
      const size_t off = base + (r < live ? r * ld : 0) + cc * 8;
      dk_cp16(sK + (stage * DK_KEYS + r) * LD + cc * 8, k_cache + off, r < live);
      dk_cp16(sV + (stage * DK_KEYS + r) * LD + cc * 8, v_cache + off, r < live);
    }
    dk_commit();
  };
  load_tile(lo, 0);
  const int r_lo = lane / 4;                    // this thread's two M rows: r_lo, r_lo + 8
  const bool two = valid_m > 8;                 // ... the second only where some pair sits there
  int kvl[2], klo[2];
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int m = r_lo + 8 * h;
    kvl[h] = m < valid_m ? row_kvlen[row0 + m / G] : 0;
    klo[h] = m < valid_m ? first_key(kvl[h] - 1, window, chunk) : 0;
  }
  float o[HD / 8][4];
#pragma unroll
  for (int i = 0; i < HD / 8; ++i) { o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f; }
  float mrow[2] = {-INFINITY, -INFINITY}, lrow[2] = {0.f, 0.f};
  const int ntiles = (hi - lo + DK_KEYS - 1) / DK_KEYS;

  for (int tile = 0; tile < ntiles; ++tile) {
    const int stage = tile & 1;
    if (tile + 1 < ntiles) { load_tile(lo + (tile + 1) * DK_KEYS, stage ^ 1); dk_wait<1>(); }
    else dk_wait<0>();
    __syncthreads();
    const int t0 = lo + tile * DK_KEYS + warp * 16;          // this warp's 16 keys
    const bool means = POOL && t0 < shift;
    const int off = POOL && !means ? kv_lo - shift : 0;      // from the place in the list to the token
    if (t0 < hi && (means || t0 + off + 15 >= first_lo)) {
      const __nv_bfloat16* K = sK + (stage * DK_KEYS + warp * 16) * LD;
      const __nv_bfloat16* V = sV + (stage * DK_KEYS + warp * 16) * LD;
      float s[2][4] = {};
#pragma unroll
      for (int ks = 0; ks < HD / 16; ++ks) {
        uint32_t a[4], b[4];
        dk_ldsm(a, sQ + ((lane & 7) + ((lane >> 3) & 1) * 8) * LD + ks * 16 + (lane >> 4) * 8);
        dk_ldsm(b, K + ((lane >> 4) * 8 + (lane & 7)) * LD + ks * 16 + ((lane >> 3) & 1) * 8);
        dk_mma(s[0], a, b[0], b[1]);
        dk_mma(s[1], a, b[2], b[3]);
      }
      const int kbase = t0 + (lane & 3) * 2;
      float f[2] = {1.f, 1.f};
      uint32_t pa[4] = {0u, 0u, 0u, 0u}, px[4] = {0u, 0u, 0u, 0u};
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        if (h == 1 && !two) break;
        float mx = -INFINITY;
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int t = kbase + nt * 8 + e;
            float v = s[nt][2 * h + e] * scale_log2;
            if (cap_log2 > 0.f) v = cap_log2 * tanh_exp(v);
            if constexpr (POOL) {
              if (t >= hi || (means ? (t + 1) * pool > klo[h] : t + off >= kvl[h] || t + off < klo[h])) v = -INFINITY;
            } else {
              if (t >= kvl[h] || t < klo[h] || t >= hi) v = -INFINITY;
            }
            s[nt][2 * h + e] = v;
            mx = fmaxf(mx, v);
          }
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float mn = fmaxf(mrow[h], mx);
        f[h] = mn == -INFINITY ? 1.f : exp2f(mrow[h] - mn);
        mrow[h] = mn;
        const float ref = mn == -INFINITY ? 0.f : mn;
        float ls = 0.f;
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          const float p0 = exp2f(s[nt][2 * h] - ref), p1 = exp2f(s[nt][2 * h + 1] - ref);
          ls += p0 + p1;
          const uint32_t v = pack_bf2(p0, p1);
          pa[nt * 2 + h] = v;
          px[nt * 2 + h] = pack_bf2(p0 - bf_lo(v), p1 - bf_hi(v));
        }
        lrow[h] = lrow[h] * f[h] + ls;
      }
      if (__any_sync(0xffffffffu, f[0] != 1.f || f[1] != 1.f)) {
#pragma unroll
        for (int i = 0; i < HD / 8; ++i) { o[i][0] *= f[0]; o[i][1] *= f[0]; o[i][2] *= f[1]; o[i][3] *= f[1]; }
      }
#pragma unroll
      for (int np = 0; np < HD / 16; ++np) {
        uint32_t b[4];
        dk_ldsm_t(b, V + (((lane >> 3) & 1) * 8 + (lane & 7)) * LD + np * 16 + (lane >> 4) * 8);
        dk_mma(o[np * 2], pa, b[0], b[1]);
        dk_mma(o[np * 2 + 1], pa, b[2], b[3]);
        dk_mma(o[np * 2], px, b[0], b[1]);
        dk_mma(o[np * 2 + 1], px, b[2], b[3]);
      }
    }
    __syncthreads();                                         // the stage is free for the load after next
  }
  // join the warps: (maximum, sum) over the queries' place, outputs over the key tiles
  float* sml = reinterpret_cast<float*>(dk_smem);            // [WARPS][M][2]
  float* so = reinterpret_cast<float*>(sK);                  // [WARPS][M][HD]
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int m = r_lo + 8 * h;
    lrow[h] += __shfl_xor_sync(0xffffffffu, lrow[h], 1);
    lrow[h] += __shfl_xor_sync(0xffffffffu, lrow[h], 2);
    if ((lane & 3) == 0) { sml[(warp * DK_M + m) * 2] = mrow[h]; sml[(warp * DK_M + m) * 2 + 1] = lrow[h]; }
    if (m < valid_m) {
      float* dst = so + ((size_t)warp * DK_M + m) * HD + (lane & 3) * 2;
#pragma unroll
      for (int i = 0; i < HD / 8; ++i) *reinterpret_cast<float2*>(dst + i * 8) = make_float2(o[i][2 * h], o[i][2 * h + 1]);
    }
  }
  __syncthreads();
  for (int c = tid; c < valid_m * (HD / 4); c += DK_THREADS) {
    const int m = c / (HD / 4), d = c % (HD / 4) * 4;
    float M = -INFINITY, L = 0.f;
#pragma unroll
    for (int w = 0; w < DK_WARPS; ++w) M = fmaxf(M, sml[(w * DK_M + m) * 2]);
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int w = 0; w < DK_WARPS; ++w) {
      const float mw = sml[(w * DK_M + m) * 2];
      const float f = mw == -INFINITY ? 0.f : exp2f(mw - M);
      const float4 v = *reinterpret_cast<const float4*>(so + ((size_t)w * DK_M + m) * HD + d);
      acc.x = fmaf(v.x, f, acc.x); acc.y = fmaf(v.y, f, acc.y); acc.z = fmaf(v.z, f, acc.z); acc.w = fmaf(v.w, f, acc.w);
      L = fmaf(sml[(w * DK_M + m) * 2 + 1], f, L);
    }
    const size_t rec = record(m);
    *reinterpret_cast<float4*>(o_part + rec * HD + d) = acc;
    if (d == 0) { ml_part[rec * 2] = M; ml_part[rec * 2 + 1] = L; }
  }
}

}  // namespace fb

using namespace fb;

// Records of key splits as fb_attn_decode_mma leaves them (o_part [rows][nq][nsplit][hd], ml_part two floats each); scale of the scores; kb:
// window, chunk and softcap, or null; pool: means of the blocks before the window, or null. Returns -20 for shapes it does not take: heads of 64
// or 128 columns, max_rows * (nq / nkv) <= 16 (with means: nq / nkv <= 16), pages of a multiple of 64 keys.
extern "C" int fb_attn_decode_keys(float* o_part, float* ml_part, const void* q, const void* k_cache, const void* v_cache, const int* seg_slot,
                                   const int* seg_row0, const int* seg_nrows, const int* row_kvlen, const int* block_table, int max_blocks,
                                   int kv_block, int nseg, int max_rows, int rows, int nq, int nkv, int hd, int nsplit, float scale,
                                   const KeyBounds* kb, const PoolKeys* pool, int row_first, int* status, cudaStream_t s) {
  if (nseg <= 0 || rows <= 0) return 0;
  if (nkv <= 0 || nq % nkv || nsplit < 1) return -1;
  const int G = nq / nkv;
  if ((hd != 64 && hd != 128) || (pool ? G : (long)max_rows * G) > DK_M || kv_block % DK_KEYS) return -20;
  if (pool && (pool->size < 1 || !kb || !kb->window)) return -1;
  if (kb && (kb->window < 0 || kb->chunk < 0 || (kb->window && kb->chunk) || kb->cap < 0.f)) return -1;
  constexpr float LOG2E = 1.4426950408889634f;
  const float cap = kb ? kb->cap : 0.f;
  const int gps = (max_rows + DK_M / G - 1) / (DK_M / G);
  const dim3 grid(nseg * gps, nkv, nsplit);
  auto go = [&](auto kern) {
    const size_t smem = (size_t)(DK_M + 4 * DK_KEYS) * (hd + 8) * 2;
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    return (int)launch_pdl(kern, grid, dim3(DK_THREADS), smem, s, o_part, ml_part, (const __nv_bfloat16*)q, (const __nv_bfloat16*)k_cache,
                           (const __nv_bfloat16*)v_cache, seg_slot, seg_row0, seg_nrows, row_kvlen, block_table, max_blocks, kv_block, nq, nkv,
                           nsplit, gps, row_first, cap > 0.f ? scale / cap : scale * LOG2E, kb ? kb->window : 0, kb ? kb->chunk : 0, cap * LOG2E,
                           pool ? (const __nv_bfloat16*)pool->k : nullptr, pool ? (const __nv_bfloat16*)pool->v : nullptr, pool ? pool->size : 0,
                           status);
  };
  if (pool) return hd == 64 ? go(attn_decode_keys_kernel<64, true>) : go(attn_decode_keys_kernel<128, true>);
  return hd == 64 ? go(attn_decode_keys_kernel<64, false>) : go(attn_decode_keys_kernel<128, false>);
}
