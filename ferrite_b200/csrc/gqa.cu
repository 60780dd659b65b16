// Grouped-query attention of the models of listed layers: what happens between the fused projection and the attention kernels
// (`attn_prefill_tc.cu` for prompt segments, `attn_decode_mma.cu` for few rows, `latent.cu` in 32 bits).
//
//   proj row = [q heads | k heads (| v heads)] of `dim` columns each, fp32 sums without their biases; with v_off at the keys the
//   values are the projected keys themselves, before rotation and norm.
//
// One warp per head: bias, rotation of the pairs (0, 1), (2, 3), ... of the first `rot` columns, division by the root mean square
// over `dim` (no weight), q to [row][head][hp], k and v into their page rows [kv head][hp]; columns dim .. hp - 1 are zeros.
// Angles are formed and reduced to one turn in double: a position of millions keeps all its bits.
#include "api_ext.h"
#include "common.cuh"
#include "elem.cuh"

namespace fb {

constexpr int GP_WARPS = 8;

// NP: pairs of a head per lane (dim <= 64 NP)
template <typename T, int NP>
__global__ void __launch_bounds__(GP_WARPS * 32)
gqa_prep_kernel(T* __restrict__ q_out, T* __restrict__ k_cache, T* __restrict__ v_cache, const float* __restrict__ proj, long ldp,
                const float* __restrict__ bias, const double* __restrict__ inv_freq, const int* __restrict__ row_slot,
                const int* __restrict__ row_pos, const int* __restrict__ block_table, int max_blocks, int kv_block, int heads,
                int kv_heads, int dim, int hp, int rot, int v_off, int norm, float eps, int* status) {
  extern __shared__ float2 gp_turn[];                       // (cos, sin) of every rotated pair
  pdl_launch_dependents();
  const int row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_wait();
  proj = after_wait(proj);
  const int pos = row_pos[row];
  for (int i = threadIdx.x; i < rot / 2; i += blockDim.x) {
    constexpr double TURN = 6.283185307179586476925;
    double a = (double)pos * inv_freq[i];
    a -= TURN * rint(a / TURN);
    float s, c;
    sincosf((float)a, &s, &c);
    gp_turn[i] = make_float2(c, s);
  }
  __syncthreads();
  const int h = blockIdx.y * GP_WARPS + warp;
  if (h >= heads + kv_heads) return;
  const int col = h * dim;                                  // q heads, then k heads
  const float* src = proj + (size_t)row * ldp + col;
  const bool is_q = h < heads;
  float2 v[NP];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < NP; ++j) {
    const int d = 2 * (lane + 32 * j);
    float2 x = make_float2(0.f, 0.f);
    if (d < dim) x.x = src[d] + (bias ? bias[col + d] : 0.f);
    if (d + 1 < dim) x.y = src[d + 1] + (bias ? bias[col + d + 1] : 0.f);
    if (d < rot) {
      const float2 t = gp_turn[d / 2];
      x = make_float2(x.x * t.x - x.y * t.y, x.y * t.x + x.x * t.y);
    }
    v[j] = x;
    ss = fmaf(x.x, x.x, fmaf(x.y, x.y, ss));
  }
  ss = warp_sum(ss);
  const float r = norm ? 1.f / sqrtf(ss / (float)dim + eps) : 1.f;
  T* dst;
  if (is_q) {
    dst = q_out + ((size_t)row * heads + h) * hp;
  } else {
    const int blk = block_table[(size_t)row_slot[row] * max_blocks + pos / kv_block];
    if (blk < 0) { if (lane == 0) set_status(status, ST_BOUNDS); return; }
    const size_t at = (((size_t)blk * kv_block + pos % kv_block) * kv_heads + (h - heads)) * hp;
    dst = k_cache + at;
    const int vc = v_off + (h - heads) * dim;
    const float* vs = proj + (size_t)row * ldp + vc;
    for (int d = 2 * lane; d < hp; d += 64) {
      const float a = d < dim ? vs[d] + (bias ? bias[vc + d] : 0.f) : 0.f;
      const float b = d + 1 < dim ? vs[d + 1] + (bias ? bias[vc + d + 1] : 0.f) : 0.f;
      Elem<T>::store2(v_cache + at + d, a, b);
    }
  }
#pragma unroll
  for (int j = 0; j < NP; ++j) {
    const int d = 2 * (lane + 32 * j);
    if (d < hp) Elem<T>::store2(dst + d, v[j].x * r, v[j].y * r);
  }
}

// The form with norms over whole rows of queries and of keys (weights, before the rotation), a value width of its own and two maps per
// head. proj row = [heads x maps x dim | kv_heads x maps x dim | .. v_off: kv_heads x vdim]. A key row takes a head's maps side by side; a
// query goes to [row][head][map][hp] with zeros in the other map's columns, so that one product with the key row gives its map's score.
// HALF: the rotated pairs are (i, i + rot / 2). Without caches only queries are made (the layer reads another layer's keys).
// One CTA per row: sums of squares over the row, then one warp per head; of a few rows several CTAs, which form the same sums and share the heads.
// Positions, pages and angles do not come from the kernel before this one, so they are read while it drains.
template <typename T, bool EVEN, bool HALF>
__global__ void __launch_bounds__(512)
gqa_row_prep_kernel(T* __restrict__ q_out, T* __restrict__ k_cache, T* __restrict__ v_cache, const float* __restrict__ proj, long ldp,
                    const float* __restrict__ q_norm, const float* __restrict__ k_norm, const double* __restrict__ inv_freq,
                    const int* __restrict__ row_slot, const int* __restrict__ row_pos, const int* __restrict__ block_table, int max_blocks,
                    int kv_block, int heads, int kv_heads, int maps, int dim, int vdim, int hp, int rot, int v_off, float eps, int* status) {
  extern __shared__ float2 gr_turn[];                       // (cos, sin) of every rotated pair
  __shared__ float red[32];
  pdl_launch_dependents();
  const int row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int nq = heads * maps * dim, nk = kv_heads * maps * dim;
  const int pos = row_pos[row];
  for (int i = threadIdx.x; i < rot / 2; i += blockDim.x) {
    constexpr double TURN = 6.283185307179586476925;
    double a = (double)pos * inv_freq[i];
    a -= TURN * rint(a / TURN);
    float s, c;
    sincosf((float)a, &s, &c);
    gr_turn[i] = make_float2(c, s);
  }
  const int blk = block_table[(size_t)row_slot[row] * max_blocks + pos / kv_block];
  if (blk < 0 && threadIdx.x == 0) set_status(status, ST_BOUNDS);
  pdl_wait();
  proj = after_wait(proj);
  const float* pr = proj + (size_t)row * ldp;
  float rq = 1.f, rk = 1.f;
  if (q_norm) {
    auto squares = [&](const float* x, int n) {
      float s = 0.f;
      if (EVEN) {
        for (int i = 2 * threadIdx.x; i < n; i += 2 * blockDim.x) {
          const float2 v = *reinterpret_cast<const float2*>(x + i);
          s = fmaf(v.x, v.x, fmaf(v.y, v.y, s));
        }
      } else {
        for (int i = threadIdx.x; i < n; i += blockDim.x) s = fmaf(x[i], x[i], s);
      }
      return s;
    };
    const float sq = squares(pr, nq), sk = k_cache ? squares(pr + nq, nk) : 0.f;
    rq = 1.f / sqrtf(block_sum(sq, red) / (float)nq + eps);
    if (k_cache) rk = 1.f / sqrtf(block_sum(sk, red) / (float)nk + eps);
  } else {
    __syncthreads();
  }
  const size_t page_row = blk < 0 ? 0 : ((size_t)blk * kv_block + pos % kv_block) * kv_heads;
  // columns d, d + 1 of one map: src[0 .. dim), rotated; e counts from the map's first column and may leave it on either side
  auto pair = [&](const float* src, const float* w, float r, int e) {
    float2 x = make_float2(0.f, 0.f);
    if (EVEN) {                                             // both columns are inside or neither is
      if (e >= 0 && e < dim) {
        x = *reinterpret_cast<const float2*>(src + e);
        if (w) {
          const float2 ww = *reinterpret_cast<const float2*>(w + e);
          x.x *= r * ww.x; x.y *= r * ww.y;
        }
      }
    } else {
      if (e >= 0 && e < dim) x.x = w ? src[e] * r * w[e] : src[e];
      if (e + 1 >= 0 && e + 1 < dim) x.y = w ? src[e + 1] * r * w[e + 1] : src[e + 1];
    }
    if constexpr (HALF) {                                   // the other column of a pair lies rot / 2 further or back
      const int hr = rot / 2;
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const int c = e + k;
        if (c < 0 || c >= rot) continue;
        const int o = c < hr ? c + hr : c - hr;
        const float z = w ? src[o] * r * w[o] : src[o];
        const float2 t = gr_turn[c < hr ? c : o];
        float& v = k ? x.y : x.x;
        v = c < hr ? v * t.x - z * t.y : v * t.x + z * t.y;
      }
      return x;
    }
    if (e >= 0 && e < rot) {                                // rot is even, and so is e wherever something is rotated
      const float2 t = gr_turn[e >> 1];
      x = make_float2(x.x * t.x - x.y * t.y, x.y * t.x + x.x * t.y);
    }
    return x;
  };
  const int units = heads * maps + (k_cache ? 2 * kv_heads : 0);
  for (int u = blockIdx.y * (blockDim.x >> 5) + warp; u < units; u += gridDim.y * (blockDim.x >> 5)) {
    if (u < heads * maps) {
      const float* src = pr + u * dim;
      const float* w = q_norm ? q_norm + u * dim : nullptr;
      T* dst = q_out + ((size_t)row * heads * maps + u) * hp;
      const int off = (u % maps) * dim;
      for (int d = 2 * lane; d < hp; d += 64) {
        const float2 x = pair(src, w, rq, d - off);
        Elem<T>::store2(dst + d, x.x, x.y);
      }
    } else if (u < heads * maps + kv_heads) {
      const int g = u - heads * maps;
      if (blk < 0) continue;
      const float* src = pr + nq + g * maps * dim;
      const float* w = k_norm ? k_norm + g * maps * dim : nullptr;
      T* dst = k_cache + (page_row + g) * hp;
      for (int d = 2 * lane; d < hp; d += 64) {
        float2 x = pair(src, w, rk, d);
        if (maps == 2) {
          const float2 y = pair(src + dim, w ? w + dim : nullptr, rk, d - dim);
          x.x += y.x; x.y += y.y;                           // one of the two is zero in every column
        }
        Elem<T>::store2(dst + d, x.x, x.y);
      }
    } else {
      const int g = u - heads * maps - kv_heads;
      if (blk < 0) continue;
      const float* src = pr + v_off + g * vdim;
      T* dst = v_cache + (page_row + g) * hp;
      for (int d = 2 * lane; d < hp; d += 64) {
        float2 x = make_float2(0.f, 0.f);
        if (EVEN && d < vdim) x = *reinterpret_cast<const float2*>(src + d);
        else if (d < vdim) x = make_float2(src[d], d + 1 < vdim ? src[d + 1] : 0.f);
        Elem<T>::store2(dst + d, x.x, x.y);
      }
    }
  }
}

// ---- pooled blocks ------------------------------------------------------------------------------------------------------
// The mean of the cached keys (values) of every block of `pool` positions whose last one, e, is in the step: into the page of e, at row
// (e % kv_block) / pool of its mean rows [per_page][kv_heads][hp]. grid (blocks that can end in a segment, kv heads, segments); half of the
// CTA takes the keys, half the values.
constexpr int PK_THREADS = 128;

template <typename T>
__global__ void __launch_bounds__(PK_THREADS) pool_keys_kernel(T* __restrict__ k_mean, T* __restrict__ v_mean, const T* __restrict__ k_cache,
                                                               const T* __restrict__ v_cache, const int* __restrict__ seg_slot,
                                                               const int* __restrict__ seg_pos0, const int* __restrict__ seg_nrows,
                                                               const int* __restrict__ block_table, int max_blocks, int kv_block, int kv_heads, int hp,
                                                               int pool, int per_page, int* status) {
  pdl_launch_dependents();
  pdl_wait();
  k_cache = after_wait(k_cache); v_cache = after_wait(v_cache);
  const int seg = blockIdx.z, h = blockIdx.y, p0 = seg_pos0[seg], n = seg_nrows[seg];
  const int e = (p0 / pool + 1 + blockIdx.x) * pool - 1;                 // last position of the block
  if (e >= p0 + n) return;
  const int* bt = block_table + (size_t)seg_slot[seg] * max_blocks;
  const bool keys = threadIdx.x < PK_THREADS / 2;
  const T* cache = keys ? k_cache : v_cache;
  const int own = bt[e / kv_block];
  if (own < 0) { if (threadIdx.x == 0) set_status(status, ST_BOUNDS); return; }
  T* dst = (keys ? k_mean : v_mean) + (((size_t)own * per_page + e % kv_block / pool) * kv_heads + h) * hp;
  const float inv = 1.f / (float)pool;
  for (int d = (threadIdx.x % (PK_THREADS / 2)) * 4; d < hp; d += PK_THREADS / 2 * 4) {
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int t = e - pool + 1; t <= e; ++t) {
      const int blk = bt[t / kv_block];
      if (blk < 0) { set_status(status, ST_BOUNDS); continue; }
      const float4 v = Elem<T>::load4(cache + (((size_t)blk * kv_block + t % kv_block) * kv_heads + h) * hp + d);
      s.x += v.x; s.y += v.y; s.z += v.z; s.w += v.w;
    }
    Elem<T>::store4(dst + d, make_float4(s.x * inv, s.y * inv, s.z * inv, s.w * inv));
  }
}

// Mean rows of the blocks that a prompt's rows see, side by side: out rows [start[seg], start[seg] + count[seg]) of segment seg, zeros up to
// start[seg + 1]; grid (rows of out). A row is `width` elements of keys and as many of values.
__global__ void __launch_bounds__(128) pool_gather_kernel(__nv_bfloat16* __restrict__ k_out, __nv_bfloat16* __restrict__ v_out,
                                                          const __nv_bfloat16* __restrict__ k_mean, const __nv_bfloat16* __restrict__ v_mean,
                                                          const int* __restrict__ seg_slot, const int* __restrict__ start, const int* __restrict__ count,
                                                          int nseg, const int* __restrict__ block_table, int max_blocks, int kv_block, int width,
                                                          int pool, int per_page, int* status) {
  pdl_launch_dependents();
  pdl_wait();
  k_mean = after_wait(k_mean); v_mean = after_wait(v_mean);
  const int row = blockIdx.x;
  int seg = 0;
  while (seg + 1 < nseg && start[seg + 1] <= row) ++seg;
  const int b = row - start[seg], e = b * pool + pool - 1;
  int blk = -1;
  if (b < count[seg]) {
    blk = block_table[(size_t)seg_slot[seg] * max_blocks + e / kv_block];
    if (blk < 0 && threadIdx.x == 0) set_status(status, ST_BOUNDS);
  }
  const size_t src = blk < 0 ? 0 : ((size_t)blk * per_page + e % kv_block / pool) * width, dst = (size_t)row * width;
  for (int i = threadIdx.x * 8; i < width; i += 128 * 8) {
    const uint4 z = make_uint4(0, 0, 0, 0);
    *reinterpret_cast<uint4*>(k_out + dst + i) = blk < 0 ? z : *reinterpret_cast<const uint4*>(k_mean + src + i);
    *reinterpret_cast<uint4*>(v_out + dst + i) = blk < 0 ? z : *reinterpret_cast<const uint4*>(v_mean + src + i);
  }
}

}  // namespace fb

using namespace fb;

// Caches [page][kv_block][kv_heads][hp], means [page][per_page][kv_heads][hp]
extern "C" int fb_pool_keys(void* k_mean, void* v_mean, const void* k_cache, const void* v_cache, const int* seg_slot, const int* seg_pos0,
                            const int* seg_nrows, int nseg, int max_rows, const int* block_table, int max_blocks, int kv_block, int kv_heads, int hp,
                            int pool, int f32, int* status, cudaStream_t s) {
  if (nseg <= 0 || max_rows <= 0) return 0;
  if (pool < 1 || hp % 4 || kv_heads < 1 || kv_heads > 65535 || nseg > 65535) return -1;
  const dim3 grid((max_rows - 1) / pool + 1, kv_heads, nseg);
  const int per_page = (kv_block + pool - 1) / pool;
  auto go = [&](auto kern, auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    return (int)launch_pdl(kern, grid, dim3(PK_THREADS), 0, s, (T*)k_mean, (T*)v_mean, (const T*)k_cache, (const T*)v_cache, seg_slot, seg_pos0,
                           seg_nrows, block_table, max_blocks, kv_block, kv_heads, hp, pool, per_page, status);
  };
  return f32 ? go(pool_keys_kernel<float>, (float*)0) : go(pool_keys_kernel<__nv_bfloat16>, (__nv_bfloat16*)0);
}

extern "C" int fb_pool_gather(void* k_out, void* v_out, const void* k_mean, const void* v_mean, const int* seg_slot, const int* start,
                              const int* count, int nseg, int rows, const int* block_table, int max_blocks, int kv_block, int width, int pool,
                              int* status, cudaStream_t s) {
  if (nseg <= 0 || rows <= 0) return 0;
  if (pool < 1 || width % 8) return -1;
  return (int)launch_pdl(pool_gather_kernel, dim3(rows), dim3(128), 0, s, (__nv_bfloat16*)k_out, (__nv_bfloat16*)v_out, (const __nv_bfloat16*)k_mean,
                         (const __nv_bfloat16*)v_mean, seg_slot, start, count, nseg, block_table, max_blocks, kv_block, width, pool,
                         (kv_block + pool - 1) / pool, status);
}

extern "C" int fb_gqa_row_prep(void* q_out, void* k_cache, void* v_cache, const float* proj, long ldp, const float* q_norm,
                               const float* k_norm, const double* inv_freq, const int* row_slot, const int* row_pos, const int* block_table,
                               int max_blocks, int kv_block, int rows, int heads, int kv_heads, int maps, int dim, int vdim, int hp, int rot,
                               int v_off, int half, float eps, int f32, int* status, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (!k_cache != !v_cache || (half && maps != 1)) return -1;
  if (dim < 1 || vdim < 1 || maps < 1 || maps > 2 || maps * dim > hp || vdim > hp || hp % 64 || rot % 2 || rot > dim || (rot && !inv_freq) ||
      (rot && maps == 2 && dim % 2) || (k_cache && (!q_norm) != (!k_norm))) return -1;
  const size_t smem = (size_t)(rot / 2 + 1) * sizeof(float2);
  const int units = heads * maps + 2 * kv_heads, threads = units > 16 ? 512 : 256, share = rows <= 16 ? (units * 32 + threads - 1) / threads : 1;
  auto go = [&](auto kern, auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    return (int)launch_pdl(kern, dim3(rows, share), dim3(threads), smem, s, (T*)q_out, (T*)k_cache, (T*)v_cache, proj, ldp, q_norm, k_norm,
                           inv_freq, row_slot, row_pos, block_table, max_blocks, kv_block, heads, kv_heads, maps, dim, vdim, hp, rot, v_off, eps,
                           status);
  };
  using B = __nv_bfloat16;
  const bool even = dim % 2 == 0 && vdim % 2 == 0 && ldp % 2 == 0 && v_off % 2 == 0 &&
                    (((uintptr_t)proj | (uintptr_t)q_norm | (uintptr_t)k_norm) & 7) == 0;
  if (half) {
    if (even) return f32 ? go(gqa_row_prep_kernel<float, true, true>, (float*)0) : go(gqa_row_prep_kernel<B, true, true>, (B*)0);
    return f32 ? go(gqa_row_prep_kernel<float, false, true>, (float*)0) : go(gqa_row_prep_kernel<B, false, true>, (B*)0);
  }
  if (even) return f32 ? go(gqa_row_prep_kernel<float, true, false>, (float*)0) : go(gqa_row_prep_kernel<B, true, false>, (B*)0);
  return f32 ? go(gqa_row_prep_kernel<float, false, false>, (float*)0) : go(gqa_row_prep_kernel<B, false, false>, (B*)0);
}

extern "C" int fb_gqa_prep(void* q_out, void* k_cache, void* v_cache, const float* proj, long ldp, const float* bias,
                           const double* inv_freq, const int* row_slot, const int* row_pos, const int* block_table, int max_blocks,
                           int kv_block, int rows, int heads, int kv_heads, int dim, int hp, int rot, int v_off, int norm, float eps,
                           int f32, int* status, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (dim < 1 || dim > hp || hp % 64 || hp > 1024 || rot % 2 || rot > dim || (rot && !inv_freq)) return -1;
  const dim3 grid(rows, (heads + kv_heads + GP_WARPS - 1) / GP_WARPS);
  const size_t smem = (size_t)(rot / 2 + 1) * sizeof(float2);
  auto go = [&](auto kern, auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    return (int)launch_pdl(kern, grid, dim3(GP_WARPS * 32), smem, s, (T*)q_out, (T*)k_cache, (T*)v_cache, proj, ldp, bias, inv_freq,
                           row_slot, row_pos, block_table, max_blocks, kv_block, heads, kv_heads, dim, hp, rot, v_off, norm, eps, status);
  };
  using B = __nv_bfloat16;
  if (hp <= 64) return f32 ? go(gqa_prep_kernel<float, 1>, (float*)0) : go(gqa_prep_kernel<B, 1>, (B*)0);
  if (hp <= 128) return f32 ? go(gqa_prep_kernel<float, 2>, (float*)0) : go(gqa_prep_kernel<B, 2>, (B*)0);
  if (hp <= 256) return f32 ? go(gqa_prep_kernel<float, 4>, (float*)0) : go(gqa_prep_kernel<B, 4>, (B*)0);
  return f32 ? go(gqa_prep_kernel<float, 16>, (float*)0) : go(gqa_prep_kernel<B, 16>, (B*)0);
}
