// Kernels of the models whose layers are listed one by one: position-free latent attention, RMSNorm on the sublayers'
// outputs over a 32-bit residual stream, a hashed bigram embedding, softcapped logits.
//
//   embed_grams    x = table[token] * scale + grams[(prev * mul_prev + token * mul_cur) mod buckets] in 32 bits. The token of
//                  every cached position is kept in an int32 page next to the KV pages, so the token before a segment comes
//                  out of the cache: it moves with the pages (parking, forks, resumed prefixes, rejected drafts) for free.
//   latent_prep    both latents of a token from one fused projection: RMSNorm of the query latent, RMSNorm of the key / value
//                  latent into its page
//   latent_attn    few rows: every head attends the cached latents themselves (key projection folded into the query); the same
//                  kernel over separate keys and values of grouped heads, with a sink, is what grouped-query attention runs in 32
//                  bits and at head widths the tensor-core kernels do not take
//   add_normed     x += rms(y + bias) * w on the 32-bit residual stream, plus the next GEMM's operand: the new x or its norm
//   norm_rows      rms(x[idx]) * w for the rows whose logits are wanted; layer_norm_rows the same with the mean off and a bias
//   add_layer_norm x += y + weighted expert rows, plus the next GEMM's operand, the layer norm of the new x (parallel blocks)
//   softcap        logits <- cap * tanh(logits / cap)
//   gemm_f32       y = x W^T in 32 bits on the CUDA cores, optionally one product per head
//
// The row kernels are templates over the element type of activations and cache (bf16, or fp32 for full-precision runs).
#include "api_ext.h"
#include "common.cuh"
#include "elem.cuh"

namespace fb {

// ---- embedding -----------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) embed_grams_kernel(float* __restrict__ x, T* __restrict__ xb, int copies, const T* __restrict__ table,
                                                          const T* __restrict__ grams, const int* __restrict__ tok,
                                                          const int* __restrict__ slot, const int* __restrict__ pos,
                                                          const int* __restrict__ block_table, int max_blocks, int kv_block,
                                                          int* tok_pages, int width, int vocab, float scale,
                                                          unsigned long long buckets, unsigned long long mul_prev,
                                                          unsigned long long mul_cur, int* status) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x;
  int id = tok[row];
  if (id < 0 || id >= vocab) { if (threadIdx.x == 0) set_status(status, ST_BOUNDS); id = 0; }
  const T* gr = nullptr;
  if (grams) {
    const int p = pos[row], s = slot[row];
    const int* bt = block_table + (size_t)s * max_blocks;
    unsigned long long g = buckets;                       // a sequence's first token has the last row to itself
    if (p > 0) {
      int prev;
      if (row > 0 && slot[row - 1] == s && pos[row - 1] == p - 1) prev = tok[row - 1];
      else {
        const int blk = bt[(p - 1) / kv_block];
        if (blk < 0 && threadIdx.x == 0) set_status(status, ST_BOUNDS);
        prev = blk < 0 ? 0 : tok_pages[(size_t)blk * kv_block + (p - 1) % kv_block];
      }
      g = ((unsigned long long)prev * mul_prev + (unsigned long long)id * mul_cur) % buckets;
    }
    gr = grams + (size_t)g * width;
    if (threadIdx.x == 0) {
      const int blk = bt[p / kv_block];
      if (blk < 0) set_status(status, ST_BOUNDS);
      else tok_pages[(size_t)blk * kv_block + p % kv_block] = id;
    }
  }
  const T* tr = table + (size_t)id * width;
  for (int i = threadIdx.x * 4; i < width; i += blockDim.x * 4) {
    float4 v = Elem<T>::load4(tr + i);
    v.x *= scale; v.y *= scale; v.z *= scale; v.w *= scale;
    if (gr) {
      const float4 g = Elem<T>::load4(gr + i);
      v.x += g.x; v.y += g.y; v.z += g.z; v.w += g.w;
    }
    *reinterpret_cast<float4*>(x + (size_t)row * width + i) = v;
    for (int c = 0; c < copies; ++c) Elem<T>::store4(xb + ((size_t)row * copies + c) * width + i, v);
  }
}

// ---- row norms -------------------------------------------------------------------------------------------------------
// Sum of squares of a row of n floats (n % 4 == 0), over the whole CTA.
template <typename S>
__device__ __forceinline__ float row_rscale(const S* r, int n, int count, float eps, float* red) {
  float ss = 0.f;
  for (int i = threadIdx.x * 4; i < n; i += blockDim.x * 4) {
    const float4 v = Elem<S>::load4(r + i);
    ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
  }
  return 1.f / sqrtf(block_sum(ss, red) / (float)count + eps);
}

// x[row] += rms(y[row] + bias) * w (no w: x[row] = y[row] + bias); xb = the next operand: rms(x) * next_w, or x with next_w null. The
// row waits in shared memory between the passes (every thread reads what it wrote itself). `width` counts the true columns, `ld` the
// padded ones (zeros beyond width).
template <typename T, typename S>
__global__ void add_normed_kernel(float* __restrict__ x, T* __restrict__ xb, long ldb, const S* __restrict__ y,
                                  const float* __restrict__ bias, const float* __restrict__ w, const float* __restrict__ next_w,
                                  int width, int ld, long ldy, float eps) {
  extern __shared__ __align__(16) float an_row[];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  y = after_wait(y);
  const size_t row = blockIdx.x;
  const S* yr = y + row * ldy;
  float ss = 0.f;
  for (int i = threadIdx.x * 4; i < ld; i += blockDim.x * 4) {
    float4 v = Elem<S>::load4(yr + i);
    if (bias) {
      const float4 b = *reinterpret_cast<const float4*>(bias + i);
      v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w;
    }
    *reinterpret_cast<float4*>(an_row + i) = v;
    ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
  }
  const float r = w ? 1.f / sqrtf(block_sum(ss, red) / (float)width + eps) : 0.f;
  ss = 0.f;
  for (int i = threadIdx.x * 4; i < ld; i += blockDim.x * 4) {
    float4 a = *reinterpret_cast<const float4*>(an_row + i);
    if (w) {
      const float4 ww = *reinterpret_cast<const float4*>(w + i), xx = *reinterpret_cast<const float4*>(x + row * ld + i);
      a.x = xx.x + a.x * r * ww.x; a.y = xx.y + a.y * r * ww.y; a.z = xx.z + a.z * r * ww.z; a.w = xx.w + a.w * r * ww.w;
    }
    *reinterpret_cast<float4*>(x + row * ld + i) = a;
    if (next_w) *reinterpret_cast<float4*>(an_row + i) = a;
    else if (xb) Elem<T>::store4(xb + row * ldb + i, a);
    ss = fmaf(a.x, a.x, fmaf(a.y, a.y, fmaf(a.z, a.z, fmaf(a.w, a.w, ss))));
  }
  if (!next_w) return;
  const float r2 = 1.f / sqrtf(block_sum(ss, red) / (float)width + eps);
  for (int i = threadIdx.x * 4; i < ld; i += blockDim.x * 4) {
    float4 v = *reinterpret_cast<const float4*>(an_row + i);
    const float4 ww = *reinterpret_cast<const float4*>(next_w + i);
    v.x *= r2 * ww.x; v.y *= r2 * ww.y; v.z *= r2 * ww.z; v.w *= r2 * ww.w;
    Elem<T>::store4(xb + row * ldb + i, v);
  }
}

// out[r] = x[idx ? idx[r] : r] * rscale * w
template <typename T>
__global__ void norm_rows_kernel(T* __restrict__ out, const float* __restrict__ x, const int* __restrict__ idx,
                                 const float* __restrict__ w, int width, int ld, float eps) {
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  x = after_wait(x);
  const float* xr = x + (size_t)(idx ? idx[blockIdx.x] : (int)blockIdx.x) * ld;
  const float r = row_rscale<float>(xr, ld, width, eps, red);
  for (int i = threadIdx.x * 4; i < ld; i += blockDim.x * 4) {
    float4 v = *reinterpret_cast<const float4*>(xr + i);
    const float4 ww = *reinterpret_cast<const float4*>(w + i);
    v.x *= r * ww.x; v.y *= r * ww.y; v.z *= r * ww.z; v.w *= r * ww.w;
    Elem<T>::store4(out + (size_t)blockIdx.x * ld + i, v);
  }
}

// ---- layer norms (mean off, bias): rows of `width` true columns, zeros up to ld ------------------------------------------
// The row waits in shared memory (every thread reads what it wrote itself); mean first, then the squared deviations of the true columns.
__device__ __forceinline__ float2 ln_stats(const float* row, float sum, int width, int ld, float eps, float* red) {
  const float mean = block_sum(sum, red) / (float)width;
  float ss = 0.f;
  for (int i = threadIdx.x * 4; i < ld; i += blockDim.x * 4) {
    const float4 v = *reinterpret_cast<const float4*>(row + i);
    const float a = v.x - mean, b = v.y - mean, c = v.z - mean, d = v.w - mean;
    if (i + 3 < width) {
      ss = fmaf(a, a, fmaf(b, b, fmaf(c, c, fmaf(d, d, ss))));
    } else {
      if (i < width) ss = fmaf(a, a, ss);
      if (i + 1 < width) ss = fmaf(b, b, ss);
      if (i + 2 < width) ss = fmaf(c, c, ss);
    }
  }
  return make_float2(mean, 1.f / sqrtf(block_sum(ss, red) / (float)width + eps));
}
template <typename T>
__device__ __forceinline__ void ln_store(T* out, const float* row, float2 st, const float* w, const float* b, int ld) {
  for (int i = threadIdx.x * 4; i < ld; i += blockDim.x * 4) {
    float4 v = *reinterpret_cast<const float4*>(row + i);
    const float4 ww = *reinterpret_cast<const float4*>(w + i), bb = b ? *reinterpret_cast<const float4*>(b + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    v.x = (v.x - st.x) * st.y * ww.x + bb.x; v.y = (v.y - st.x) * st.y * ww.y + bb.y;
    v.z = (v.z - st.x) * st.y * ww.z + bb.z; v.w = (v.w - st.x) * st.y * ww.w + bb.w;
    Elem<T>::store4(out + i, v);
  }
}

// x[row] += y[row] + sum over `top` picks of wts[row][k] * yp[row * top + k]; xb = layer norm of the new x (no w: none)
template <typename T, typename S>
__global__ void add_layer_norm_kernel(float* __restrict__ x, T* __restrict__ xb, const S* __restrict__ y, long ldy, const float* __restrict__ yp,
                                      const float* __restrict__ wts, int top, const float* __restrict__ w, const float* __restrict__ b,
                                      int width, int ld, float eps) {
  extern __shared__ __align__(16) float al_row[];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  y = after_wait(y); yp = after_wait(yp); wts = after_wait(wts);
  const size_t row = blockIdx.x;
  const S* yr = y + row * ldy;
  float* xr = x + row * ld;
  float sum = 0.f;
  for (int i = threadIdx.x * 4; i < ld; i += blockDim.x * 4) {
    float4 a = *reinterpret_cast<const float4*>(xr + i);
    const float4 v = Elem<S>::load4(yr + i);
    float4 s = v;
    for (int k = 0; k < top; ++k) {
      const float g = wts[row * top + k];
      const float4 e = *reinterpret_cast<const float4*>(yp + (row * top + k) * ld + i);
      s.x = fmaf(g, e.x, s.x); s.y = fmaf(g, e.y, s.y); s.z = fmaf(g, e.z, s.z); s.w = fmaf(g, e.w, s.w);
    }
    a.x += s.x; a.y += s.y; a.z += s.z; a.w += s.w;
    *reinterpret_cast<float4*>(xr + i) = a;
    if (w) *reinterpret_cast<float4*>(al_row + i) = a;
    sum += (a.x + a.y) + (a.z + a.w);
  }
  if (!w) return;
  const float2 st = ln_stats(al_row, sum, width, ld, eps, red);
  ln_store<T>(xb + row * ld, al_row, st, w, b, ld);
}

template <typename T>
__global__ void layer_norm_rows_kernel(T* __restrict__ out, const float* __restrict__ x, const int* __restrict__ idx,
                                       const float* __restrict__ w, const float* __restrict__ b, int width, int ld, float eps) {
  extern __shared__ __align__(16) float al_row[];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  x = after_wait(x);
  const float* xr = x + (size_t)(idx ? idx[blockIdx.x] : (int)blockIdx.x) * ld;
  float sum = 0.f;
  for (int i = threadIdx.x * 4; i < ld; i += blockDim.x * 4) {
    const float4 v = *reinterpret_cast<const float4*>(xr + i);
    *reinterpret_cast<float4*>(al_row + i) = v;
    sum += (v.x + v.y) + (v.z + v.w);
  }
  const float2 st = ln_stats(al_row, sum, width, ld, eps, red);
  ln_store<T>(out + (size_t)blockIdx.x * ld, al_row, st, w, b, ld);
}

// proj row = [query latent (qr columns, q_rank true) | key / value latent (lat columns, kv_rank true)], fp32.
template <typename T>
__global__ void __launch_bounds__(256) latent_prep_kernel(T* __restrict__ cq, T* __restrict__ cache, const float* __restrict__ proj,
                                                          long ldp, const float* __restrict__ q_norm,
                                                          const float* __restrict__ kv_norm, const int* __restrict__ row_slot,
                                                          const int* __restrict__ row_pos, const int* __restrict__ block_table,
                                                          int max_blocks, int kv_block, int q_rank, int qr, int kv_rank, int lat,
                                                          float eps, int* status) {
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  proj = after_wait(proj);
  const size_t row = blockIdx.x;
  const float* pr = proj + row * ldp;
  float r = row_rscale<float>(pr, qr, q_rank, eps, red);
  for (int i = threadIdx.x * 4; i < qr; i += blockDim.x * 4) {
    float4 v = *reinterpret_cast<const float4*>(pr + i);
    const float4 w = *reinterpret_cast<const float4*>(q_norm + i);
    v.x *= r * w.x; v.y *= r * w.y; v.z *= r * w.z; v.w *= r * w.w;
    Elem<T>::store4(cq + row * qr + i, v);
  }
  if (!kv_norm) return;                                   // the layer reads another layer's latents
  const int p = row_pos[row];
  const int blk = block_table[(size_t)row_slot[row] * max_blocks + p / kv_block];
  if (blk < 0) { if (threadIdx.x == 0) set_status(status, ST_BOUNDS); return; }
  T* dst = cache + ((size_t)blk * kv_block + p % kv_block) * lat;
  pr += qr;
  r = row_rscale<float>(pr, lat, kv_rank, eps, red);
  for (int i = threadIdx.x * 4; i < lat; i += blockDim.x * 4) {
    float4 v = *reinterpret_cast<const float4*>(pr + i);
    const float4 w = *reinterpret_cast<const float4*>(kv_norm + i);
    v.x *= r * w.x; v.y *= r * w.y; v.z *= r * w.z; v.w *= r * w.w;
    Elem<T>::store4(dst + i, v);
  }
}

// The form with a rotated key part: proj row = [heads x (dim | rot) | latent (kv_rank) | key part (rot)], fp32. Queries go to [row][head][hp] with
// their last rot columns rotated (pairs (0, 1), (2, 3), ..), the normed latent and the rotated key part to the token's cache row, zeros beyond.
// Angles are formed and reduced to one turn in double.
// grid (rows, 1 + groups of LR_HEADS heads): the first CTA of a row makes its cache row, the others heads of its query.
constexpr int LR_HEADS = 8;

template <typename T>
__global__ void __launch_bounds__(256) latent_rot_prep_kernel(T* __restrict__ q_out, T* __restrict__ cache, const float* __restrict__ proj, long ldp,
                                                              const float* __restrict__ kv_norm, const double* __restrict__ inv_freq,
                                                              const int* __restrict__ row_slot, const int* __restrict__ row_pos,
                                                              const int* __restrict__ block_table, int max_blocks, int kv_block, int heads, int dim,
                                                              int rot, int hp, int kv_rank, int lat, float eps, int* status) {
  extern __shared__ float2 lr_turn[];
  __shared__ float red[32];
  pdl_launch_dependents();
  const size_t row = blockIdx.x;
  const int pos = row_pos[row];
  for (int i = threadIdx.x; i < rot / 2; i += blockDim.x) {
    constexpr double TURN = 6.283185307179586476925;
    double a = (double)pos * inv_freq[i];
    a -= TURN * rint(a / TURN);
    float s, c;
    sincosf((float)a, &s, &c);
    lr_turn[i] = make_float2(c, s);
  }
  const int blk = block_table[(size_t)row_slot[row] * max_blocks + pos / kv_block];
  pdl_wait();
  proj = after_wait(proj);
  const float* pr = proj + row * ldp;
  const int kd = dim + rot;
  auto turned = [&](const float* src, int e) {               // column e of a rotated part
    const float2 t = lr_turn[e >> 1];
    const float u = src[e & ~1], v = src[e | 1];
    return e & 1 ? v * t.x + u * t.y : u * t.x - v * t.y;
  };
  if (blockIdx.y == 0) {
    const float* pc = pr + (size_t)heads * kd;
    float ss = 0.f;
    for (int i = threadIdx.x; i < kv_rank; i += blockDim.x) ss = fmaf(pc[i], pc[i], ss);
    const float r = 1.f / sqrtf(block_sum(ss, red) / (float)kv_rank + eps);    // (its barriers publish the angles)
    if (blk < 0) {
      if (threadIdx.x == 0) set_status(status, ST_BOUNDS);
      return;
    }
    T* dst = cache + ((size_t)blk * kv_block + pos % kv_block) * lat;
    for (int i = threadIdx.x; i < lat; i += blockDim.x)
      dst[i] = Elem<T>::from(i < kv_rank ? pc[i] * r * kv_norm[i] : i < kv_rank + rot ? turned(pc + kv_rank, i - kv_rank) : 0.f);
    return;
  }
  __syncthreads();
  const int h = (blockIdx.y - 1) * LR_HEADS + (threadIdx.x >> 5);            // one warp per head
  if (h >= heads) return;
  const float* src = pr + h * kd;
  T* dst = q_out + (row * heads + h) * (size_t)hp;
  for (int d = 2 * (threadIdx.x & 31); d < hp; d += 64) {
    float o[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) o[e] = d + e < dim ? src[d + e] : d + e < kd ? turned(src + dim, d + e - dim) : 0.f;
    Elem<T>::store2(dst + d, o[0], o[1]);
  }
}

__global__ void softcap_kernel(float* __restrict__ y, long ld, int n, float cap) {
  pdl_launch_dependents();
  pdl_wait();
  float* r = y + (size_t)blockIdx.y * ld;
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) r[i] = cap * tanhf(r[i] / cap);
}

// y = relu(x)^2 where the product that made x has no such epilogue (packed weights)
__global__ void relu2_kernel(__nv_bfloat16* __restrict__ y, const __nv_bfloat16* __restrict__ x, long ldx, int n) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const float v = fmaxf(bf2f(x[(size_t)blockIdx.y * ldx + i]), 0.f);
  y[(size_t)blockIdx.y * n + i] = f2bf(v * v);
}

// ---- attention over the cached latents, CUDA cores ---------------------------------------------------------------------
// grid (rows, heads, splits), 4 warps striding over the keys with an online softmax; a lane owns columns 64 j + 2 lane, + 1.
// lat = 64 nl with nl <= NJ. One split writes the normalised output itself, more leave partials for the merge. KV: cache rows are
// [kv_heads][lat] of keys with the values in v_cache (else one latent row, keys and values alike); sink: a number per head that
// joins the denominator; window / chunk bound the keys a row sees, cap > 0 softcaps the scores (scale_log2 is then scale / cap).
// `records`: one split leaves its partial as well. Rows of out are ldo elements apart and have vl columns per head (latents: the first ones of
// a cache row). pool > 0 (KV): the means of the blocks before the window come first in the list of keys.
constexpr int LA_WARPS = 4;
constexpr float LOG2E = 1.4426950408889634f;

template <typename T, int NJ, bool KV>
__global__ void __launch_bounds__(LA_WARPS * 32) latent_attn_kernel(T* __restrict__ out, float* __restrict__ o_part,
                                                                    float* __restrict__ ml_part, const T* __restrict__ q,
                                                                    const T* __restrict__ cache, const T* __restrict__ v_cache,
                                                                    const float* __restrict__ sink, const int* __restrict__ row_slot,
                                                                    const int* __restrict__ row_kvlen,
                                                                    const int* __restrict__ block_table, int max_blocks,
                                                                    int kv_block, int heads, int kv_heads, int lat, int nsplit,
                                                                    float scale_log2, int window, int chunk, float cap, long ldo, int records,
                                                                    int vl, const T* __restrict__ k_mean, const T* __restrict__ v_mean, int pool,
                                                                    int* status) {
  extern __shared__ float so[];                            // [warps][lat]
  __shared__ float sml[LA_WARPS][2];
  pdl_launch_dependents();
  pdl_wait();
  q = after_wait(q); cache = after_wait(cache); v_cache = after_wait(v_cache); k_mean = after_wait(k_mean); v_mean = after_wait(v_mean);
  const int nl = lat / 64;
  const int row = blockIdx.x, h = blockIdx.y, split = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kvlen = row_kvlen[row];
  const int* bt = block_table + (size_t)row_slot[row] * max_blocks;
  const int kv_lo = first_key(kvlen - 1, window, chunk);
  // list of keys: nb means, then the tokens from kv_lo on
  const int nb = KV && pool > 0 ? kv_lo / pool : 0, keys = nb + kvlen - kv_lo, per_page = KV && pool > 0 ? (kv_block + pool - 1) / pool : 1;
  int per = (keys + nsplit - 1) / nsplit;
  per = (per + 31) / 32 * 32;
  const int lo = split * per, hi = min(keys, lo + per);
  const T* qr = q + ((size_t)row * heads + h) * lat;
  float2 qf[NJ], o[NJ];
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    o[j] = make_float2(0.f, 0.f);
    qf[j] = j < nl ? Elem<T>::load2(qr + 64 * j + 2 * lane) : make_float2(0.f, 0.f);
    qf[j].x *= scale_log2; qf[j].y *= scale_log2;
  }
  float m = -INFINITY, l = 0.f;
  for (int u = lo + warp; u < hi; u += LA_WARPS) {
    const bool mean = u < nb;
    const int t = mean ? u * pool + pool - 1 : u - nb + kv_lo;
    const int blk = bt[t / kv_block];
    if (blk < 0) { if (lane == 0) set_status(status, ST_BOUNDS); break; }
    size_t at = mean ? (size_t)blk * per_page + t % kv_block / pool : (size_t)blk * kv_block + t % kv_block;
    if constexpr (KV) at = at * kv_heads + h / (heads / kv_heads);
    const T* kr = (mean ? k_mean : cache) + at * lat + 2 * lane;
    float2 k[NJ];
#pragma unroll
    for (int j = 0; j < NJ; ++j) k[j] = j < nl ? Elem<T>::load2(kr + 64 * j) : make_float2(0.f, 0.f);
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < NJ; ++j) s = fmaf(qf[j].x, k[j].x, fmaf(qf[j].y, k[j].y, s));
    s = warp_sum(s);
    if constexpr (KV) { if (cap > 0.f) s = cap * LOG2E * tanhf(s); }
    const float mn = fmaxf(m, s);
    const float a = exp2f(m - mn), p = exp2f(s - mn);
    l = l * a + p;
    if constexpr (KV) {
      const T* vr = (mean ? v_mean : v_cache) + at * lat + 2 * lane;
#pragma unroll
      for (int j = 0; j < NJ; ++j) k[j] = j < nl ? Elem<T>::load2(vr + 64 * j) : make_float2(0.f, 0.f);
    }
#pragma unroll
    for (int j = 0; j < NJ; ++j) { o[j].x = fmaf(p, k[j].x, o[j].x * a); o[j].y = fmaf(p, k[j].y, o[j].y * a); }
    m = mn;
  }
#pragma unroll
  for (int j = 0; j < NJ; ++j)
    if (j < nl) *reinterpret_cast<float2*>(so + (size_t)warp * lat + 64 * j + 2 * lane) = o[j];
  if (lane == 0) { sml[warp][0] = m; sml[warp][1] = l; }
  __syncthreads();
  float M = -INFINITY, f[LA_WARPS], Ls = 0.f;
#pragma unroll
  for (int w = 0; w < LA_WARPS; ++w) M = fmaxf(M, sml[w][0]);
#pragma unroll
  for (int w = 0; w < LA_WARPS; ++w) {
    f[w] = sml[w][0] == -INFINITY ? 0.f : exp2f(sml[w][0] - M);
    Ls += sml[w][1] * f[w];
  }
  const size_t pidx = ((size_t)row * heads + h) * nsplit + split;
  const float den = Ls + (sink && nsplit == 1 ? exp2f(sink[h] * LOG2E - M) : 0.f);
  const bool final_rows = nsplit == 1 && !records;
  const float inv = final_rows ? (den > 0.f ? 1.f / den : 0.f) : 1.f;
  for (int d = threadIdx.x; d < vl; d += blockDim.x) {
    float acc = 0.f;
#pragma unroll
    for (int w = 0; w < LA_WARPS; ++w) acc += so[(size_t)w * lat + d] * f[w];
    if (final_rows) out[(size_t)row * ldo + (size_t)h * vl + d] = Elem<T>::from(acc * inv);
    else o_part[pidx * vl + d] = acc;
  }
  if (!final_rows && threadIdx.x == 0) { ml_part[pidx * 2] = M; ml_part[pidx * 2 + 1] = Ls; }
}

// Merge of the splits; grid (rows, heads). LG_GROUPS groups of 128 threads take every LG_GROUPS-th split each (all loads of a
// group in flight together) and are added in group order, so the result does not depend on scheduling.
constexpr int LG_GROUPS = 4;

template <typename T>
__global__ void __launch_bounds__(128 * LG_GROUPS) latent_merge_kernel(T* __restrict__ out, long ldo, const float* __restrict__ o_part,
                                                                       const float* __restrict__ ml_part,
                                                                       const float* __restrict__ sink, int heads, int nsplit, int lat) {
  extern __shared__ float sf[];                            // [nsplit] factors, then [groups][lat] partial sums
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  o_part = after_wait(o_part); ml_part = after_wait(ml_part);
  const size_t rh = (size_t)blockIdx.x * heads + blockIdx.y, pbase = rh * nsplit;
  const int tid = threadIdx.x, grp = tid / 128, col = (tid % 128) * 4;
  float M = -INFINITY, Ls = 0.f;
  for (int s = tid; s < nsplit; s += blockDim.x) M = fmaxf(M, ml_part[(pbase + s) * 2]);
  M = block_max(M, red);
  for (int s = tid; s < nsplit; s += blockDim.x) {
    const float ms = ml_part[(pbase + s) * 2];
    const float f = ms == -INFINITY ? 0.f : exp2f(ms - M);          // an empty split wrote no rows
    sf[s] = f;
    Ls += f == 0.f ? 0.f : ml_part[(pbase + s) * 2 + 1] * f;
  }
  Ls = block_sum(Ls, red);                                 // (its barriers publish the factors)
  if (sink) Ls += exp2f(sink[blockIdx.y] * LOG2E - M);
  const float inv = Ls > 0.f ? 1.f / Ls : 0.f;
  float* sums = sf + nsplit;
  for (int d = col; d < lat; d += 512) {
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int s = grp; s < nsplit; s += LG_GROUPS) {
      const float f = sf[s];
      if (f == 0.f) continue;
      const float4 v = *reinterpret_cast<const float4*>(o_part + (pbase + s) * lat + d);
      acc.x = fmaf(v.x, f, acc.x); acc.y = fmaf(v.y, f, acc.y); acc.z = fmaf(v.z, f, acc.z); acc.w = fmaf(v.w, f, acc.w);
    }
    float* p = sums + grp * lat + d;
    p[0] = acc.x; p[1] = acc.y; p[2] = acc.z; p[3] = acc.w;
  }
  __syncthreads();
  if (tid < lat / 4)
    for (int d = tid * 4; d < lat; d += 512 * 4) {
      float v[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int g = 0; g < LG_GROUPS; ++g)
#pragma unroll
        for (int e = 0; e < 4; ++e) v[e] += sums[g * lat + d + e];
      Elem<T>::store4(out + (size_t)blockIdx.x * ldo + (size_t)blockIdx.y * lat + d, make_float4(v[0] * inv, v[1] * inv, v[2] * inv, v[3] * inv));
    }
}

// ---- heads' outputs: difference of two maps, norm, output gate -----------------------------------------------------------
// o = a1 - lam a2, divided by its root mean square over vdim and scaled (two maps), times sigmoid(gate): from the records of key splits
// (one CTA per row and head; half of it per map) or from normalised rows (one warp per row and head).
constexpr int MX_THREADS = 256;

template <typename T, int MAPS>
__global__ void __launch_bounds__(MX_THREADS) attn_merge_mix_kernel(T* __restrict__ out, long ldo, const float* __restrict__ o_part,
                                                                    const float* __restrict__ ml_part, const float* __restrict__ lam,
                                                                    const float* __restrict__ gate, long ldg, float mix_scale, int heads,
                                                                    int nsplit, int vdim, int hd, float eps) {
  constexpr int PER = MX_THREADS / MAPS;                   // threads of a map
  extern __shared__ __align__(16) float mx_s[];            // [MAPS][nsplit] factors, [MAPS] 1 / row sum, [MAPS][groups][hd] sums
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  o_part = after_wait(o_part); ml_part = after_wait(ml_part); gate = after_wait(gate);
  const int tid = threadIdx.x, map = tid / PER, t = tid % PER, warp = tid >> 5, lane = tid & 31;
  const size_t row = blockIdx.x;
  const int h = blockIdx.y;
  const size_t pbase = ((row * heads + h) * MAPS + map) * nsplit;
  float* fac = mx_s + map * nsplit;
  float* inv = mx_s + MAPS * nsplit;
  float* sums = mx_s + (MAPS * nsplit + MAPS + 3) / 4 * 4;
  if (warp < MAPS) {                                       // one warp per map turns the maxima into factors
    const size_t pb = ((row * heads + h) * MAPS + warp) * nsplit;
    float M = -INFINITY, L = 0.f;
    for (int s = lane; s < nsplit; s += 32) M = fmaxf(M, ml_part[(pb + s) * 2]);
    M = warp_max(M);
    for (int s = lane; s < nsplit; s += 32) {
      const float ms = ml_part[(pb + s) * 2];
      const float f = ms == -INFINITY ? 0.f : exp2f(ms - M);         // an empty split wrote no rows
      mx_s[warp * nsplit + s] = f;
      if (f != 0.f) L += ml_part[(pb + s) * 2 + 1] * f;
    }
    L = warp_sum(L);
    if (lane == 0) inv[warp] = L > 0.f ? 1.f / L : 0.f;
  }
  __syncthreads();
  const int cols = hd / 4, groups = max(1, PER / cols);    // groups of threads take every groups-th split
  for (int i = t; i < cols * groups; i += PER) {
    const int g = i / cols, d = (i % cols) * 4;
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int s = g; s < nsplit; s += groups) {
      const float f = fac[s];
      if (f == 0.f) continue;
      const float4 v = *reinterpret_cast<const float4*>(o_part + (pbase + s) * hd + d);
      acc.x = fmaf(v.x, f, acc.x); acc.y = fmaf(v.y, f, acc.y); acc.z = fmaf(v.z, f, acc.z); acc.w = fmaf(v.w, f, acc.w);
    }
    *reinterpret_cast<float4*>(sums + ((size_t)map * groups + g) * hd + d) = acc;
  }
  __syncthreads();
  const float l2 = MAPS == 2 ? lam[0] : 0.f;
  float ss = 0.f;
  for (int d = tid; d < hd; d += MX_THREADS) {
    float a[MAPS];
#pragma unroll
    for (int m = 0; m < MAPS; ++m) {
      a[m] = 0.f;
      for (int g = 0; g < groups; ++g) a[m] += sums[((size_t)m * groups + g) * hd + d];
      a[m] *= inv[m];
    }
    const float o = MAPS == 2 ? a[0] - l2 * a[MAPS - 1] : a[0];
    sums[d] = o;                                           // this thread's own column of group 0
    ss = fmaf(o, o, ss);
  }
  const float r = MAPS == 2 ? mix_scale / sqrtf(block_sum(ss, red) / (float)vdim + eps) : 1.f;
  for (int d = tid; d < hd; d += MX_THREADS) {
    float o = sums[d] * r;
    if (gate && d < vdim) o *= 1.f / (1.f + expf(-gate[row * ldg + (size_t)h * vdim + d]));
    out[row * ldo + (size_t)h * hd + d] = Elem<T>::from(o);
  }
}

// in [rows][heads * MAPS][hd] fp32, zeros beyond vdim
template <typename T, int MAPS>
__global__ void __launch_bounds__(256) head_mix_kernel(T* __restrict__ out, long ldo, const float* __restrict__ in, const float* __restrict__ lam,
                                                       const float* __restrict__ gate, long ldg, float mix_scale, int heads, int vdim, int hd,
                                                       float eps) {
  pdl_launch_dependents();
  pdl_wait();
  in = after_wait(in); gate = after_wait(gate);
  const size_t row = blockIdx.x;
  const int h = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h >= heads) return;
  const float* a = in + (row * heads + h) * MAPS * hd;
  T* dst = out + row * ldo + (size_t)h * hd;
  const float l2 = MAPS == 2 ? lam[0] : 0.f;
  float ss = 0.f;
  auto value = [&](int d) {
    float4 v = *reinterpret_cast<const float4*>(a + d);
    if constexpr (MAPS == 2) {
      const float4 b = *reinterpret_cast<const float4*>(a + hd + d);
      v.x -= l2 * b.x; v.y -= l2 * b.y; v.z -= l2 * b.z; v.w -= l2 * b.w;
    }
    return v;
  };
  float r = 1.f;
  if constexpr (MAPS == 2) {
    for (int d = lane * 4; d < hd; d += 128) {
      const float4 v = value(d);
      ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
    }
    r = mix_scale / sqrtf(warp_sum(ss) / (float)vdim + eps);
  }
  for (int d = lane * 4; d < hd; d += 128) {
    const float4 v = value(d);
    float o[4] = {v.x * r, v.y * r, v.z * r, v.w * r};
    if (gate) {
      const float* g = gate + row * ldg + (size_t)h * vdim + d;
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (d + e < vdim) o[e] *= 1.f / (1.f + expf(-g[e]));
    }
    Elem<T>::store4(dst + d, make_float4(o[0], o[1], o[2], o[3]));
  }
}

// ---- attention over the cached latents, tensor cores ---------------------------------------------------------------------
// bf16. The M dimension is (row of the segment, head): all of them read the same latents, so one pass over a key tile
// serves 64 of them. grid (segments x M tiles, splits), 8 warps. Scores: warp = 16 M rows x 32 of the tile's 64 keys over the
// whole latent (16 keys when at most 32 M rows are in use, so that no warp idles). Values are the same shared-memory tile read
// transposed: warp = all 64 M rows x lat / 8 columns. The softmax weights go through shared memory as a bf16 value plus its bf16
// remainder, two products each, so they keep 16 bits of mantissa instead of 8; scores, maxima, exponentials and row sums are
// 32-bit.
// A cache row has 64 NJ columns; values are its first 64 VJ (the rest is a key part). M is 64, or 32 where rows are so wide that two key
// tiles and 64 queries do not fit.
constexpr int LM_KEYS = 64, LM_THREADS = 256, LM_LDP = LM_KEYS + 8;

__device__ __forceinline__ void lm_cp16(void* smem, const void* gmem, bool valid) {
  const int sz = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(smem)), "l"(gmem), "r"(sz) : "memory");
}
__device__ __forceinline__ void lm_ldsm(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void lm_ldsm_t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void lm_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

template <int NJ>
struct Lm {
  static constexpr int LM_M = NJ <= 8 ? 64 : 32, VJ = NJ <= 8 ? NJ : 8;
  static constexpr int LAT = NJ * 64, LD = LAT + 8;
  static constexpr size_t SMEM = (size_t)(LM_M + 2 * LM_KEYS) * LD * 2 + (size_t)2 * LM_M * LM_LDP * 2 + 6 * LM_M * 4;
};

template <int NJ>
__global__ void __launch_bounds__(LM_THREADS, 1)
latent_mma_kernel(__nv_bfloat16* __restrict__ out, float* __restrict__ o_part, float* __restrict__ ml_part,
                  const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ cache, const int* __restrict__ seg_slot,
                  const int* __restrict__ seg_row0, const int* __restrict__ seg_nrows, const int* __restrict__ row_kvlen,
                  const int* __restrict__ block_table, int max_blocks, int kv_block, int heads, int row_base, int tiles_per_seg,
                  int nsplit, float scale_log2, int window, int* status) {
  constexpr int LAT = Lm<NJ>::LAT, LD = Lm<NJ>::LD, CPR = LAT / 8, LM_M = Lm<NJ>::LM_M, MT = LM_M / 16, VJ = Lm<NJ>::VJ, VL = VJ * 64;
  extern __shared__ __align__(16) unsigned char lm_smem[];
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(lm_smem);           // [M][LD]
  __nv_bfloat16* sK = sQ + LM_M * LD;                                      // [2][KEYS][LD]
  __nv_bfloat16* sP = sK + 2 * LM_KEYS * LD;                               // [value | remainder][M][LDP]
  float* smx = reinterpret_cast<float*>(sP + 2 * LM_M * LM_LDP);           // [4][M] maxima of the key groups, then sums
  float* sfac = smx + 4 * LM_M;                                            // [M] rescale factor of the tile
  float* sinv = sfac + LM_M;                                               // [M] 1 / row sum
  pdl_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int seg = blockIdx.x / tiles_per_seg, tile_m = blockIdx.x % tiles_per_seg, split = blockIdx.y;
  const int n = seg_nrows[seg], m_all = n * heads, m0 = tile_m * LM_M;
  if (m0 >= m_all) return;
  const int valid_m = min(LM_M, m_all - m0);
  const int row0 = seg_row0[seg];
  const int* bt = block_table + (size_t)seg_slot[seg] * max_blocks;
  const int kv_end = row_kvlen[row0 + (m0 + valid_m - 1) / heads - row_base];          // rows of a segment see ever more keys
  const int kv_lo = first_key(row_kvlen[row0 + m0 / heads - row_base] - 1, window, 0) / LM_KEYS * LM_KEYS;
  int per = (kv_end - kv_lo + nsplit - 1) / nsplit;
  per = (per + LM_KEYS - 1) / LM_KEYS * LM_KEYS;
  const int lo = kv_lo + split * per, hi = min(kv_end, lo + per);
  // (row, head) flat index of an M row in q / out, which start at row row_base of the step
  const size_t flat0 = (size_t)(row0 - row_base) * heads + m0;
  if (lo >= hi) {
    if (nsplit > 1)
      for (int m = tid; m < valid_m; m += LM_THREADS) {
        float* ml = ml_part + ((flat0 + m) * nsplit + split) * 2;
        ml[0] = -INFINITY; ml[1] = 0.f;
      }
    return;
  }
  for (int c = tid; c < LM_M * CPR; c += LM_THREADS) {
    const int m = c / CPR, cc = c % CPR;
    const bool ok = m < valid_m;
    lm_cp16(sQ + m * LD + cc * 8, q + (flat0 + (ok ? m : 0)) * LAT + cc * 8, ok);
  }
  auto load_tile = [&](int t0, int stage) {                  // a tile lies in one page: both start on multiples of 64 keys
    const int blk = bt[t0 / kv_block];
    if (blk < 0 && tid == 0) set_status(status, ST_BOUNDS);
    const int live = blk < 0 ? 0 : min(LM_KEYS, hi - t0);
    const __nv_bfloat16* src = cache + (blk < 0 ? 0 : ((size_t)blk * kv_block + t0 % kv_block) * LAT);
    __nv_bfloat16* dst = sK + stage * LM_KEYS * LD;
#pragma unroll 4
    for (int c = tid; c < LM_KEYS * CPR; c += LM_THREADS) {
      const int r = c / CPR, cc = c % CPR;
      lm_cp16(dst + r * LD + cc * 8, src + (r < live ? c * 8 : 0), r < live);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load_tile(lo, 0);

  // score role: 16 M rows at mw * 16, keys [key0, key0 + 16 npairs) of the tile
  const bool few = valid_m <= 32;
  const int mw = few ? warp & 1 : warp & 3, nw = few ? warp >> 1 : warp >> 2, kgroups = few ? 4 : 2;
  const int npairs = few ? 1 : 2, key0 = nw * 16 * npairs;
  const int r_lo = mw * 16 + lane / 4;                       // this thread's two M rows: r_lo, r_lo + 8
  int kvl[2], klo[2];
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int m = r_lo + 8 * h;
    kvl[h] = m < valid_m ? row_kvlen[row0 + (m0 + m) / heads - row_base] : 0;
    klo[h] = m < valid_m ? first_key(kvl[h] - 1, window, 0) : 0;
  }
  float mrow[2] = {-INFINITY, -INFINITY}, lrow[2] = {0.f, 0.f};
  float o[MT][VJ][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < VJ; ++j) { o[i][j][0] = o[i][j][1] = o[i][j][2] = o[i][j][3] = 0.f; }
  const int ntiles = (hi - lo + LM_KEYS - 1) / LM_KEYS;
  const bool score_on = mw * 16 < valid_m;

  for (int tile = 0; tile < ntiles; ++tile) {
    const int stage = tile & 1;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                         // the tile has landed; everyone is done with the other buffer
    if (tile + 1 < ntiles) load_tile(lo + (tile + 1) * LM_KEYS, stage ^ 1);
    const __nv_bfloat16* K = sK + stage * LM_KEYS * LD;
    float s[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i) { s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f; }
    float mx[2] = {-INFINITY, -INFINITY};
    if (score_on) {
      // fragments are loaded one k step ahead of the products
      const __nv_bfloat16* pa = sQ + (mw * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LD + (lane >> 4) * 8;
      const __nv_bfloat16* pb = K + (key0 + (lane >> 4) * 8 + (lane & 7)) * LD + ((lane >> 3) & 1) * 8;
      uint32_t a[2][4], b[2][2][4];
      lm_ldsm(a[0], pa);
      lm_ldsm(b[0][0], pb);
      if (!few) lm_ldsm(b[0][1], pb + 16 * LD);
#pragma unroll 4
      for (int ks = 0; ks < LAT / 16; ++ks) {
        const int cur = ks & 1;
        if (ks + 1 < LAT / 16) {
          lm_ldsm(a[cur ^ 1], pa + (ks + 1) * 16);
          lm_ldsm(b[cur ^ 1][0], pb + (ks + 1) * 16);
          if (!few) lm_ldsm(b[cur ^ 1][1], pb + 16 * LD + (ks + 1) * 16);
        }
        lm_mma(s[0], a[cur], b[cur][0][0], b[cur][0][1]);
        lm_mma(s[1], a[cur], b[cur][0][2], b[cur][0][3]);
        if (!few) {
          lm_mma(s[2], a[cur], b[cur][1][0], b[cur][1][1]);
          lm_mma(s[3], a[cur], b[cur][1][2], b[cur][1][3]);
        }
      }
      const int kbase = lo + tile * LM_KEYS + key0 + (lane & 3) * 2;
#pragma unroll
      for (int nt = 0; nt < 4; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int t = kbase + nt * 8 + (e & 1), h = e >> 1;
          const float v = (nt < 2 * npairs && t < kvl[h] && t >= klo[h] && t < hi) ? s[nt][e] * scale_log2 : -INFINITY;
          s[nt][e] = v;
          mx[h] = fmaxf(mx[h], v);
        }
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
        mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
        if ((lane & 3) == 0) smx[nw * LM_M + r_lo + 8 * h] = mx[h];
      }
    }
    __syncthreads();
    if (score_on) {
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int r = r_lo + 8 * h;
        float mn = fmaxf(mrow[h], fmaxf(smx[r], smx[LM_M + r]));
        if (few) mn = fmaxf(mn, fmaxf(smx[2 * LM_M + r], smx[3 * LM_M + r]));
        const float f = mn == -INFINITY ? 1.f : exp2f(mrow[h] - mn);
        mrow[h] = mn;
        float ls = 0.f;
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
          if (nt >= 2 * npairs) break;
          const float p0 = mn == -INFINITY ? 0.f : exp2f(s[nt][2 * h] - mn);
          const float p1 = mn == -INFINITY ? 0.f : exp2f(s[nt][2 * h + 1] - mn);
          ls += p0 + p1;
          const uint32_t v = pack_bf2(p0, p1);
          const int at = r * LM_LDP + key0 + nt * 8 + (lane & 3) * 2;
          *reinterpret_cast<uint32_t*>(sP + at) = v;
          *reinterpret_cast<uint32_t*>(sP + LM_M * LM_LDP + at) = pack_bf2(p0 - bf_lo(v), p1 - bf_hi(v));
        }
        lrow[h] = lrow[h] * f + ls;
        if (nw == 0 && (lane & 3) == 0) sfac[r] = f;
      }
    }
    __syncthreads();
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      if (mt * 16 >= valid_m) break;
      const float f0 = sfac[mt * 16 + lane / 4], f1 = sfac[mt * 16 + lane / 4 + 8];
      if (!__any_sync(0xffffffffu, f0 != 1.f || f1 != 1.f)) continue;
#pragma unroll
      for (int j = 0; j < VJ; ++j) { o[mt][j][0] *= f0; o[mt][j][1] *= f0; o[mt][j][2] *= f1; o[mt][j][3] *= f1; }
    }
#pragma unroll
    for (int kp = 0; kp < 2; ++kp) {
      uint32_t b[VJ][4];                                     // 8 columns x 32 keys each: two k steps
#pragma unroll
      for (int j = 0; j < VJ; ++j) lm_ldsm_t(b[j], K + (kp * 32 + lane) * LD + (warp * VJ + j) * 8);
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        if (mt * 16 >= valid_m) break;
#pragma unroll
        for (int k2 = 0; k2 < 2; ++k2) {
#pragma unroll
          for (int part = 0; part < 2; ++part) {
            uint32_t a[4];
            lm_ldsm(a, sP + (part * LM_M + mt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LM_LDP + (kp * 2 + k2) * 16 + (lane >> 4) * 8);
#pragma unroll
            for (int j = 0; j < VJ; ++j) lm_mma(o[mt][j], a, b[j][2 * k2], b[j][2 * k2 + 1]);
          }
        }
      }
    }
  }
  __syncthreads();                                           // the maxima buffer takes the row sums now
  if (score_on) {
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      lrow[h] += __shfl_xor_sync(0xffffffffu, lrow[h], 1);
      lrow[h] += __shfl_xor_sync(0xffffffffu, lrow[h], 2);
      if ((lane & 3) == 0) smx[nw * LM_M + r_lo + 8 * h] = lrow[h];
    }
  }
  __syncthreads();
  if (score_on && nw == 0 && (lane & 3) == 0) {
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int r = r_lo + 8 * h;
      if (r >= valid_m) continue;
      float l = 0.f;
      for (int g = 0; g < kgroups; ++g) l += smx[g * LM_M + r];
      if (nsplit == 1) sinv[r] = l > 0.f ? 1.f / l : 0.f;
      else {
        float* ml = ml_part + ((flat0 + r) * nsplit + split) * 2;
        ml[0] = mrow[h]; ml[1] = l;
      }
    }
  }
  __syncthreads();
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int r = mt * 16 + lane / 4 + 8 * h;
      if (r >= valid_m) continue;
      const float inv = nsplit == 1 ? sinv[r] : 1.f;
#pragma unroll
      for (int j = 0; j < VJ; ++j) {
        const int d = (warp * VJ + j) * 8 + (lane & 3) * 2;
        if (nsplit == 1)
          *reinterpret_cast<uint32_t*>(out + (flat0 + r) * VL + d) = pack_bf2(o[mt][j][2 * h] * inv, o[mt][j][2 * h + 1] * inv);
        else
          *reinterpret_cast<float2*>(o_part + ((flat0 + r) * nsplit + split) * VL + d) = make_float2(o[mt][j][2 * h], o[mt][j][2 * h + 1]);
      }
    }
}

// ---- y = x W^T in 32 bits -----------------------------------------------------------------------------------------------
// 64 x 64 tile per CTA of 256 threads (4 x 4 outputs each), K in steps of 16; grid.z = batch (one product per head).
__global__ void __launch_bounds__(256) gemm_f32_kernel(float* __restrict__ y, const float* __restrict__ x,
                                                       const float* __restrict__ w, int M, int N, int K, long ldx, long ldy,
                                                       long x_bs, long w_bs, long y_bs, int act) {
  __shared__ float sx[16][64 + 4], sw[16][64 + 4];
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64, tid = threadIdx.x;
  x += (size_t)blockIdx.z * x_bs; w += (size_t)blockIdx.z * w_bs; y += (size_t)blockIdx.z * y_bs;
  const int lr = tid / 4, lk = (tid % 4) * 4;                // loader: row of the tile, 4 k values
  const int tx = tid % 16, ty = tid / 16;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += 16) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b = a;
    if (m0 + lr < M && k0 + lk < K) a = *reinterpret_cast<const float4*>(x + (size_t)(m0 + lr) * ldx + k0 + lk);
    if (n0 + lr < N && k0 + lk < K) b = *reinterpret_cast<const float4*>(w + (size_t)(n0 + lr) * K + k0 + lk);
    __syncthreads();
    sx[lk][lr] = a.x; sx[lk + 1][lr] = a.y; sx[lk + 2][lr] = a.z; sx[lk + 3][lr] = a.w;
    sw[lk][lr] = b.x; sw[lk + 1][lr] = b.y; sw[lk + 2][lr] = b.z; sw[lk + 3][lr] = b.w;
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      const float4 av = *reinterpret_cast<const float4*>(&sx[k][ty * 4]), bv = *reinterpret_cast<const float4*>(&sw[k][tx * 4]);
      const float am[4] = {av.x, av.y, av.z, av.w}, bn[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(am[i], bn[j], acc[i][j]);
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m < M && n < N) y[(size_t)m * ldy + n] = epilogue_act(acc[i][j], act);
    }
}

}  // namespace fb

using namespace fb;
using bf16 = __nv_bfloat16;

static int row_threads(int width) { return width >= 4096 ? 512 : width >= 1024 ? 256 : 128; }

extern "C" int fb_embed_grams(float* x, void* xb, int copies, const void* table, const void* grams, const int* tok, const int* slot,
                              const int* pos, const int* block_table, int max_blocks, int kv_block, int* tok_pages, int rows,
                              int width, int vocab, float scale, long buckets, long mul_prev, long mul_cur, int f32, int* status,
                              cudaStream_t s) {
  if (rows <= 0) return 0;
  if (width % 4 || (grams && (buckets <= 0 || !tok_pages))) return -1;
  if (f32)
    return (int)launch_pdl(embed_grams_kernel<float>, dim3(rows), dim3(256), 0, s, x, (float*)xb, copies, (const float*)table,
                           (const float*)grams, tok, slot, pos, block_table, max_blocks, kv_block, tok_pages, width, vocab, scale,
                           (unsigned long long)buckets, (unsigned long long)mul_prev, (unsigned long long)mul_cur, status);
  return (int)launch_pdl(embed_grams_kernel<bf16>, dim3(rows), dim3(256), 0, s, x, (bf16*)xb, copies, (const bf16*)table, (const bf16*)grams,
                         tok, slot, pos, block_table, max_blocks, kv_block, tok_pages, width, vocab, scale,
                         (unsigned long long)buckets, (unsigned long long)mul_prev, (unsigned long long)mul_cur, status);
}

// y: fp32 (y_f32) or bf16 rows of stride ldy; xb: rows of stride ldb in the operand type (xb_f32), or null; bias, w, next_w: ld
// floats or null
extern "C" int fb_add_normed(float* x, void* xb, int xb_f32, long ldb, const void* y, int y_f32, const float* bias, const float* w,
                             const float* next_w, int rows, int width, int ld, long ldy, float eps, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (ld % 4 || ldy % 4 || ldb % 4 || (next_w && !xb) || ld > 49152) return -1;
  const dim3 g(rows), b(row_threads(ld));
  const size_t smem = (size_t)ld * 4;
  auto go = [&](auto kern, auto* xo, const auto* yi) {
    if (smem > 40 * 1024) {
      const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return (int)e;
    }
    return (int)launch_pdl(kern, g, b, smem, s, x, xo, ldb, yi, bias, w, next_w, width, ld, ldy, eps);
  };
  if (xb_f32) {
    if (!y_f32) return -1;
    return go(add_normed_kernel<float, float>, (float*)xb, (const float*)y);
  }
  if (y_f32) return go(add_normed_kernel<bf16, float>, (bf16*)xb, (const float*)y);
  return go(add_normed_kernel<bf16, bf16>, (bf16*)xb, (const bf16*)y);
}

template <typename Kern>
static int row_smem(Kern kern, size_t smem) {
  return smem > 40 * 1024 ? (int)cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) : 0;
}

// mean: layer norm (b: its bias, or null), else the root mean square norm
extern "C" int fb_norm_rows(void* out, const float* x, const int* idx, const float* w, const float* b, int mean, int rows, int width, int ld,
                            float eps, int f32, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (ld % 4 || ld > 49152) return -1;
  const dim3 g(rows), t(row_threads(ld));
  if (b || mean) {
    auto go = [&](auto kern, auto* o) {
      if (const int e = row_smem(kern, (size_t)ld * 4)) return e;
      return (int)launch_pdl(kern, g, t, (size_t)ld * 4, s, o, x, idx, w, b, width, ld, eps);
    };
    return f32 ? go(layer_norm_rows_kernel<float>, (float*)out) : go(layer_norm_rows_kernel<bf16>, (bf16*)out);
  }
  if (f32) return (int)launch_pdl(norm_rows_kernel<float>, g, t, 0, s, (float*)out, x, idx, w, width, ld, eps);
  return (int)launch_pdl(norm_rows_kernel<bf16>, g, t, 0, s, (bf16*)out, x, idx, w, width, ld, eps);
}

// y: fp32 (y_f32) or bf16 rows of stride ldy; yp / wts: rows of a token's `top` experts and their weights (top 0: none); next_w, next_b:
// ld floats, or null for no operand
extern "C" int fb_add_layer_norm(float* x, void* xb, int f32, const void* y, int y_f32, long ldy, const float* yp, const float* wts, int top,
                                 const float* next_w, const float* next_b, int rows, int width, int ld, float eps, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (ld % 4 || ldy % 4 || ld > 49152 || (next_w && (!xb || !next_b)) || (top && (!yp || !wts)) || (f32 && !y_f32)) return -1;
  const dim3 g(rows), b(row_threads(ld));
  auto go = [&](auto kern, auto* xo, const auto* yi) {
    if (const int e = row_smem(kern, (size_t)ld * 4)) return e;
    return (int)launch_pdl(kern, g, b, (size_t)ld * 4, s, x, xo, yi, ldy, yp, wts, top, next_w, next_b, width, ld, eps);
  };
  if (f32) return go(add_layer_norm_kernel<float, float>, (float*)xb, (const float*)y);
  if (y_f32) return go(add_layer_norm_kernel<bf16, float>, (bf16*)xb, (const float*)y);
  return go(add_layer_norm_kernel<bf16, bf16>, (bf16*)xb, (const bf16*)y);
}

extern "C" int fb_latent_prep(void* cq, void* cache, const float* proj, long ldp, const float* q_norm, const float* kv_norm,
                              const int* row_slot, const int* row_pos, const int* block_table, int max_blocks, int kv_block,
                              int rows, int q_rank, int qr, int kv_rank, int lat, float eps, int f32, int* status, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (qr % 4 || lat % 4 || ldp % 4) return -1;
  const dim3 g(rows), b(qr + lat >= 512 ? 256 : 128);
  if (f32)
    return (int)launch_pdl(latent_prep_kernel<float>, g, b, 0, s, (float*)cq, (float*)cache, proj, ldp, q_norm, kv_norm, row_slot,
                           row_pos, block_table, max_blocks, kv_block, q_rank, qr, kv_rank, lat, eps, status);
  return (int)launch_pdl(latent_prep_kernel<bf16>, g, b, 0, s, (bf16*)cq, (bf16*)cache, proj, ldp, q_norm, kv_norm, row_slot, row_pos,
                         block_table, max_blocks, kv_block, q_rank, qr, kv_rank, lat, eps, status);
}

// proj: rows of heads * (dim + rot) + kv_rank + rot floats, ldp apart; kv_norm: kv_rank floats; lat >= kv_rank + rot, hp >= dim + rot
extern "C" int fb_latent_rot_prep(void* q_out, void* cache, const float* proj, long ldp, const float* kv_norm, const double* inv_freq,
                                  const int* row_slot, const int* row_pos, const int* block_table, int max_blocks, int kv_block, int rows, int heads,
                                  int dim, int rot, int hp, int kv_rank, int lat, float eps, int f32, int* status, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (rot % 2 || rot < 0 || dim < 0 || dim + rot > hp || hp % 2 || kv_rank < 1 || kv_rank + rot > lat) return -1;
  auto go = [&](auto kern, auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    return (int)launch_pdl(kern, dim3(rows, 1 + (heads + LR_HEADS - 1) / LR_HEADS), dim3(LR_HEADS * 32), (size_t)(rot / 2 + 1) * sizeof(float2), s,
                           (T*)q_out, (T*)cache, proj, ldp, kv_norm, inv_freq,
                           row_slot, row_pos, block_table, max_blocks, kv_block, heads, dim, rot, hp, kv_rank, lat, eps, status);
  };
  return f32 ? go(latent_rot_prep_kernel<float>, (float*)0) : go(latent_rot_prep_kernel<bf16>, (bf16*)0);
}

extern "C" int fb_softcap(float* y, int rows, int n, long ld, float cap, cudaStream_t s) {
  if (rows <= 0 || n <= 0) return 0;
  if (rows > 65535) return -1;
  return (int)launch_pdl(softcap_kernel, dim3((n + 255) / 256, rows), dim3(256), 0, s, y, ld, n, cap);
}

extern "C" int fb_relu2(void* y, const void* x, long ldx, int rows, int n, cudaStream_t s) {
  if (rows <= 0 || n <= 0) return 0;
  if (rows > 65535) return -1;
  relu2_kernel<<<dim3((n + 255) / 256, rows), 256, 0, s>>>((bf16*)y, (const bf16*)x, ldx, n);
  return (int)cudaGetLastError();
}

template <typename T>
static int latent_merge(void* out, long ldo, const float* o_part, const float* ml_part, const float* sink, int rows, int heads, int nsplit, int lat,
                        cudaStream_t s) {
  return (int)launch_pdl(latent_merge_kernel<T>, dim3(rows, heads), dim3(128 * LG_GROUPS),
                         (size_t)(nsplit + LG_GROUPS * lat) * 4, s, (T*)out, ldo, o_part, ml_part, sink, heads, nsplit, lat);
}

template <typename T, bool KV>
static int latent_attn(void* out, float* o_part, float* ml_part, const void* q, const void* cache, const void* v_cache, const float* sink,
                       const int* row_slot, const int* row_kvlen, const int* block_table, int max_blocks, int kv_block, int rows, int heads,
                       int kv_heads, int lat, int vl, int nsplit, float scale, const KeyBounds* kb, const PoolKeys* pool, long ldo, bool records,
                       int* status, cudaStream_t s) {
  const KeyBounds none{0, 0, 0.f};
  const KeyBounds& b = kb ? *kb : none;
  if (b.window < 0 || b.chunk < 0 || (b.window && b.chunk) || b.cap < 0.f || (pool && (pool->size < 1 || !b.window))) return -1;
  const float scale_log2 = b.cap > 0.f ? scale / b.cap : scale * LOG2E;
  const dim3 grid(rows, heads, nsplit);
  const size_t smem = (size_t)LA_WARPS * lat * 4;
  auto go = [&](auto kern) {
    return (int)launch_pdl(kern, grid, dim3(LA_WARPS * 32), smem, s, (T*)out, o_part, ml_part, (const T*)q, (const T*)cache,
                           (const T*)v_cache, sink, row_slot, row_kvlen, block_table, max_blocks, kv_block, heads, kv_heads, lat, nsplit,
                           scale_log2, b.window, b.chunk, b.cap, ldo, records ? 1 : 0, vl, pool ? (const T*)pool->k : nullptr,
                           pool ? (const T*)pool->v : nullptr, pool ? pool->size : 0, status);
  };
  int rc;
  if (lat <= 128) rc = go(latent_attn_kernel<T, 2, KV>);
  else if (lat <= 256) rc = go(latent_attn_kernel<T, 4, KV>);
  else if (lat <= 512) rc = go(latent_attn_kernel<T, 8, KV>);
  else rc = go(latent_attn_kernel<T, 16, KV>);
  if (rc || nsplit == 1 || records) return rc;
  return latent_merge<T>(out, ldo, o_part, ml_part, sink, rows, heads, nsplit, vl, s);
}

// out [rows][heads][vl] (the first vl columns of the rows; 64 | vl); window: keys that a row sees, 0 = all; partials (nsplit > 1): o_part rows * heads * nsplit * lat floats, ml_part two per record
extern "C" int fb_latent_attn(void* out, float* o_part, float* ml_part, const void* q, const void* cache, const int* row_slot,
                              const int* row_kvlen, const int* block_table, int max_blocks, int kv_block, int rows, int heads, int lat,
                              int vl, int window, int nsplit, float scale, int f32, int* status, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (vl % 64 || vl > lat || window < 0) return -1;
  const KeyBounds kb{window, 0, 0.f};
  if (lat % 64 || lat > 1024 || heads > 65535 || nsplit < 1 || nsplit > 4096) return -1;
  const long ldo = (long)heads * vl;
  return f32 ? latent_attn<float, false>(out, o_part, ml_part, q, cache, nullptr, nullptr, row_slot, row_kvlen, block_table, max_blocks,
                                         kv_block, rows, heads, 1, lat, vl, nsplit, scale, &kb, nullptr, ldo, false, status, s)
             : latent_attn<bf16, false>(out, o_part, ml_part, q, cache, nullptr, nullptr, row_slot, row_kvlen, block_table, max_blocks,
                                        kv_block, rows, heads, 1, lat, vl, nsplit, scale, &kb, nullptr, ldo, false, status, s);
}

// The same over separate keys and values: caches [page][kv_block][kv_heads][hd], q / out [rows][heads][hd] (rows of out ldo elements
// apart); sink: heads floats or null; kb: window, chunk, softcap, or null; pool: means of the blocks before the window, or null; out null: the records of the splits stay for the caller
extern "C" int fb_gqa_attn(void* out, float* o_part, float* ml_part, const void* q, const void* k_cache, const void* v_cache,
                           const float* sink, const int* row_slot, const int* row_kvlen, const int* block_table, int max_blocks,
                           int kv_block, int rows, int heads, int kv_heads, int hd, int nsplit, float scale, const KeyBounds* kb,
                           const PoolKeys* pool, long ldo, int f32, int* status, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (hd % 64 || hd > 1024 || heads > 65535 || kv_heads <= 0 || heads % kv_heads || nsplit < 1 || nsplit > 4096) return -1;
  if (ldo % 4 || (!out && sink)) return -1;
  return f32 ? latent_attn<float, true>(out, o_part, ml_part, q, k_cache, v_cache, sink, row_slot, row_kvlen, block_table, max_blocks,
                                        kv_block, rows, heads, kv_heads, hd, hd, nsplit, scale, kb, pool, ldo, !out, status, s)
             : latent_attn<bf16, true>(out, o_part, ml_part, q, k_cache, v_cache, sink, row_slot, row_kvlen, block_table, max_blocks,
                                       kv_block, rows, heads, kv_heads, hd, hd, nsplit, scale, kb, pool, ldo, !out, status, s);
}

// Merge of key splits alone (records as fb_attn_decode_mma leaves them), sink: heads floats or null
extern "C" int fb_attn_merge(void* out, long ldo, const float* o_part, const float* ml_part, const float* sink, int rows, int heads, int nsplit,
                             int hd, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (hd % 64 || hd > 1024 || heads > 65535 || nsplit < 1 || nsplit > 4096 || ldo % 4) return -1;
  return latent_merge<bf16>(out, ldo, o_part, ml_part, sink, rows, heads, nsplit, hd, s);
}

// Merge of key splits with what follows it: maps 2: the difference of a head's two maps (records [rows][heads][2]), its norm over vdim,
// mix_scale; gate: rows of heads * vdim logits ldg floats apart, or null. out [rows][heads][hd], rows ldo elements apart.
extern "C" int fb_attn_merge_mix(void* out, long ldo, const float* o_part, const float* ml_part, const float* lam, const float* gate, long ldg,
                                 float mix_scale, int maps, int rows, int heads, int nsplit, int vdim, int hd, float eps, int f32,
                                 cudaStream_t s) {
  if (rows <= 0) return 0;
  if (hd % 64 || hd > 1024 || heads > 65535 || nsplit < 1 || nsplit > 256 || maps < 1 || maps > 2 || (maps == 2 && !lam) || vdim < 1 ||
      vdim > hd) return -1;
  const int per = MX_THREADS / maps, groups = per / (hd / 4) > 1 ? per / (hd / 4) : 1;
  const size_t smem = ((size_t)(maps * nsplit + maps + 3) / 4 * 4 + (size_t)maps * groups * hd) * 4;
  auto go = [&](auto kern, auto* o) {
    return (int)launch_pdl(kern, dim3(rows, heads), dim3(MX_THREADS), smem, s, o, ldo, o_part, ml_part, lam, gate, ldg, mix_scale, heads, nsplit,
                           vdim, hd, eps);
  };
  if (f32) return maps == 2 ? go(attn_merge_mix_kernel<float, 2>, (float*)out) : go(attn_merge_mix_kernel<float, 1>, (float*)out);
  return maps == 2 ? go(attn_merge_mix_kernel<bf16, 2>, (bf16*)out) : go(attn_merge_mix_kernel<bf16, 1>, (bf16*)out);
}

// The same for rows that need no merge: in [rows][heads * maps][hd] fp32
extern "C" int fb_head_mix(void* out, long ldo, const float* in, const float* lam, const float* gate, long ldg, float mix_scale, int maps,
                           int rows, int heads, int vdim, int hd, float eps, int f32, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (hd % 64 || ldo % 4 || maps < 1 || maps > 2 || (maps == 2 && !lam) || vdim < 1 || vdim > hd || (heads + 7) / 8 > 65535) return -1;
  auto go = [&](auto kern, auto* o) {
    return (int)launch_pdl(kern, dim3(rows, (heads + 7) / 8), dim3(256), 0, s, o, ldo, in, lam, gate, ldg, mix_scale, heads, vdim, hd, eps);
  };
  if (f32) return maps == 2 ? go(head_mix_kernel<float, 2>, (float*)out) : go(head_mix_kernel<float, 1>, (float*)out);
  return maps == 2 ? go(head_mix_kernel<bf16, 2>, (bf16*)out) : go(head_mix_kernel<bf16, 1>, (bf16*)out);
}

// The same on tensor cores for bf16, lat <= 512 with vl = lat, or 576 with vl = 512, and pages of a multiple of 64 keys (-20 otherwise). Rows come in
// segments (consecutive rows of one slot); seg_row0 counts the rows of the step, of which q / out / row_kvlen hold those from row_base on.
extern "C" int fb_latent_mma(void* out, float* o_part, float* ml_part, const void* q, const void* cache, const int* seg_slot,
                             const int* seg_row0, const int* seg_nrows, int nseg, int max_rows, const int* row_kvlen,
                             const int* block_table, int max_blocks, int kv_block, int rows, int row_base, int heads, int lat,
                             int vl, int window, int nsplit, float scale, int* status, cudaStream_t s) {
  if (rows <= 0 || nseg <= 0) return 0;
  if (lat % 64 || lat > 576 || vl != (lat <= 512 ? lat : 512) || kv_block % LM_KEYS) return -20;
  if (nsplit < 1 || nsplit > 4096 || window < 0) return -1;
  const int m_tile = lat <= 512 ? 64 : 32, tps = (max_rows * heads + m_tile - 1) / m_tile;
  const dim3 grid(nseg * tps, nsplit);
  const float sl = scale * 1.4426950408889634f;
  int rc = 0;
#define FB_LM(NJ)                                                                                                              \
  case NJ: {                                                                                                                   \
    auto kern = latent_mma_kernel<NJ>;                                                                                         \
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Lm<NJ>::SMEM);                \
    if (e != cudaSuccess) return (int)e;                                                                                       \
    rc = (int)launch_pdl(kern, grid, dim3(LM_THREADS), Lm<NJ>::SMEM, s, (bf16*)out, o_part, ml_part, (const bf16*)q,           \
                         (const bf16*)cache, seg_slot, seg_row0, seg_nrows, row_kvlen, block_table, max_blocks, kv_block, heads, \
                         row_base, tps, nsplit, sl, window, status);                                                           \
    break;                                                                                                                     \
  }
  switch (lat / 64) { FB_LM(1) FB_LM(2) FB_LM(3) FB_LM(4) FB_LM(5) FB_LM(6) FB_LM(7) FB_LM(8) FB_LM(9) }
#undef FB_LM
  if (rc || nsplit == 1) return rc;
  return latent_merge<bf16>(out, (long)heads * vl, o_part, ml_part, nullptr, rows, heads, nsplit, vl, s);
}

// y [batch][M][N] = act(x [batch][M][K] w [batch][N][K]^T); row strides ldx / ldy, batch strides x_bs / w_bs / y_bs (elements)
extern "C" int fb_gemm_f32(float* y, const float* x, const float* w, int M, int N, int K, long ldx, long ldy, int batch, long x_bs,
                           long w_bs, long y_bs, int act, cudaStream_t s) {
  if (M <= 0 || N <= 0 || batch <= 0) return 0;
  if (K % 4 || ldx % 4 || x_bs % 4 || w_bs % 4 || batch > 65535 || (M + 63) / 64 > 65535) return -1;
  gemm_f32_kernel<<<dim3((N + 63) / 64, (M + 63) / 64, batch), 256, 0, s>>>(y, x, w, M, N, K, ldx, ldy, x_bs, w_bs, y_bs, act);
  return (int)cudaGetLastError();
}
