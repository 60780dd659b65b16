// State-space layers (Mamba-2) of few rows: one launch per group of segments from the projection to the heads' outputs, one for the gated
// norm behind it.
//
//   projection row = [z: inner | x: inner | B: groups * N | C: groups * N | dt: heads], inner = heads * V
//   x, B, C: causal convolution over the slot's tail, bias, silu;  dt = softplus(dt + dt_bias)
//   S = exp(A dt) S + dt B x^T  (S [N][V] per head, fp32),  y = S^T C + skip x
//
// grid (segments, heads, V / 16): the columns of a state are independent, so a CTA owns 16 of them, keeps its part of the state in
// registers over the rows of the segment (four columns per thread, every 32nd row of N) and sums S^T C over threads in a fixed order. The
// state lives in 32 bits; convolved values are rounded to the operand type, as the chunked form of prompts does.
#include "api_listed.h"
#include "common.cuh"
#include "elem.cuh"

namespace fb {

using bf16 = __nv_bfloat16;

constexpr int SS_THREADS = 128, SS_COLS = 16;

template <typename T, int NR>
__global__ void __launch_bounds__(SS_THREADS) ssm_step_kernel(float* __restrict__ y, long ldy, float* __restrict__ rec, const T* __restrict__ tails,
                                                              long tail_step, const T* __restrict__ proj, long ldp, const float* __restrict__ conv_w,
                                                              const float* __restrict__ conv_b, const float* __restrict__ A,
                                                              const float* __restrict__ dt_bias, const float* __restrict__ skip,
                                                              const int* __restrict__ seg_slot, const int* __restrict__ seg_row0,
                                                              const int* __restrict__ seg_nrows, int heads, int groups, int N, int V, int taps,
                                                              int commit) {
  extern __shared__ __align__(16) float ss_s[];              // [2][16 x | N B | N C]
  __shared__ float4 red[2][4][4];
  pdl_launch_dependents();
  const int h = blockIdx.y, v0 = blockIdx.z * SS_COLS, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = h / (heads / groups), inner = heads * V, ch = inner + 2 * groups * N, vals = SS_COLS + 2 * N;
  const float a_h = A[h], db = dt_bias[h], sk = skip[h];
  pdl_wait();
  proj = after_wait(proj); tails = after_wait(tails);
  const int slot = seg_slot[blockIdx.x], row0 = seg_row0[blockIdx.x], n = seg_nrows[blockIdx.x];
  if (n <= 0) return;
  const int q = tid & 3, ng = tid >> 2, v = v0 + 4 * q;      // this thread's columns v .. v + 3, rows ng, ng + 32, ...
  float* st = rec + ((size_t)slot * heads + h) * N * V;
  const bool vec = V % 4 == 0;
  float S[NR][4];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int r = ng + 32 * i;
    if (r < N && vec && v < V) {
      const float4 f = *reinterpret_cast<const float4*>(st + (size_t)r * V + v);
      S[i][0] = f.x; S[i][1] = f.y; S[i][2] = f.z; S[i][3] = f.w;
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) S[i][e] = r < N && v + e < V ? st[(size_t)r * V + v + e] : 0.f;
    }
  }
  const T* tail = tails + (size_t)slot * tail_step;
  for (int t = 0; t < n; ++t) {
    float* s = ss_s + (t & 1) * ((vals + 3) & ~3);
    const T* pr = proj + (size_t)(row0 + t) * ldp + inner;
    for (int i = tid; i < vals; i += SS_THREADS) {           // convolved x (own columns), B, C
      int c;
      if (i < SS_COLS) c = v0 + i < V ? h * V + v0 + i : -1;
      else if (i < SS_COLS + N) c = inner + g * N + i - SS_COLS;
      else c = inner + (groups + g) * N + i - SS_COLS - N;
      float acc = 0.f;
      if (c >= 0) {
        acc = conv_b[c];
        for (int j = 0; j < taps; ++j) {
          const int back = taps - 1 - j;
          const float in = back <= t ? Elem<T>::to(pr[c - (long)back * ldp]) : Elem<T>::to(tail[(size_t)(taps - 1 - (back - t)) * ch + c]);
          acc = fmaf(conv_w[(size_t)j * ch + c], in, acc);
        }
        acc = Elem<T>::to(Elem<T>::from(acc / (1.f + expf(-acc))));
      }
      s[i] = acc;
    }
    const float draw = Elem<T>::to(pr[ch + h]) + db;
    const float dt = draw > 20.f ? draw : log1pf(expf(draw)), decay = expf(a_h * dt);
    __syncthreads();
    const float4 x4 = *reinterpret_cast<const float4*>(s + 4 * q);
    const float* B = s + SS_COLS;
    const float* C = B + N;
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int r = ng + 32 * i;
      if (r >= N) break;
      const float b = dt * B[r], c = C[r];
      S[i][0] = fmaf(decay, S[i][0], b * x4.x); S[i][1] = fmaf(decay, S[i][1], b * x4.y);
      S[i][2] = fmaf(decay, S[i][2], b * x4.z); S[i][3] = fmaf(decay, S[i][3], b * x4.w);
      o.x = fmaf(c, S[i][0], o.x); o.y = fmaf(c, S[i][1], o.y); o.z = fmaf(c, S[i][2], o.z); o.w = fmaf(c, S[i][3], o.w);
    }
#pragma unroll
    for (int m = 4; m < 32; m <<= 1) {
      o.x += __shfl_xor_sync(0xffffffffu, o.x, m); o.y += __shfl_xor_sync(0xffffffffu, o.y, m);
      o.z += __shfl_xor_sync(0xffffffffu, o.z, m); o.w += __shfl_xor_sync(0xffffffffu, o.w, m);
    }
    if (lane < 4) red[t & 1][warp][lane] = o;
    __syncthreads();
    if (tid < SS_COLS && v0 + tid < V) {
      const float* p = reinterpret_cast<const float*>(red[t & 1]);
      y[(size_t)(row0 + t) * ldy + (size_t)h * V + v0 + tid] = (p[tid] + p[16 + tid]) + (p[32 + tid] + p[48 + tid]) + sk * s[tid];
    }
  }
  if (!commit) return;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int r = ng + 32 * i;
    if (r >= N) break;
    if (vec && v < V) *reinterpret_cast<float4*>(st + (size_t)r * V + v) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
    else
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (v + e < V) st[(size_t)r * V + v + e] = S[i][e];
  }
}

// out = y * silu(z), an RMS norm over each of `parts` equal parts of the row, times w; grid (rows, parts (+ tail blocks)). With
// `tails` (one row per segment) CTAs behind the parts move the slot's tail on by the row's inputs: nobody reads the old one any more.
// VEC: four columns at a time.
constexpr int GN_THREADS = 256, GN_TAIL = 1024;              // channels of a tail per CTA

template <typename T, int VEC>
__global__ void __launch_bounds__(GN_THREADS) group_norm_gated_kernel(T* __restrict__ out, long ldo, const float* __restrict__ y, long ldy,
                                                                      const T* __restrict__ proj, long ldp, const float* __restrict__ w, int inner,
                                                                      int parts, int ko, float eps, T* __restrict__ tails, long tail_step, int taps,
                                                                      int ch, const int* __restrict__ row_slot) {
  extern __shared__ __align__(16) float gn_s[];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  y = after_wait(y); proj = after_wait(proj);
  const size_t row = blockIdx.x;
  const int part = blockIdx.y, size = inner / parts, c0 = part * size;
  if (part >= parts) {                                       // a piece of the tail
    const int lo = (part - parts) * GN_TAIL, hi = min(ch, lo + GN_TAIL);
    T* t = tails + row_slot[row] * tail_step;
    for (int j0 = 0; j0 + 1 < taps; ++j0)
#pragma unroll
      for (int k = 0; k < GN_TAIL / GN_THREADS; ++k) {
        const int c = lo + k * GN_THREADS + threadIdx.x;
        if (c < hi) t[(size_t)j0 * ch + c] = j0 + 2 < taps ? t[(size_t)(j0 + 1) * ch + c] : proj[row * ldp + inner + c];
      }
    return;
  }
  float ss = 0.f;
  for (int i = threadIdx.x * VEC; i < size; i += GN_THREADS * VEC) {
    if constexpr (VEC == 4) {
      const float4 z = Elem<T>::load4(proj + row * ldp + c0 + i), a = *reinterpret_cast<const float4*>(y + row * ldy + c0 + i);
      const float4 v = make_float4(a.x * siluf_(z.x), a.y * siluf_(z.y), a.z * siluf_(z.z), a.w * siluf_(z.w));
      *reinterpret_cast<float4*>(gn_s + i) = v;
      ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
    } else {
      const float v = y[row * ldy + c0 + i] * siluf_(Elem<T>::to(proj[row * ldp + c0 + i]));
      gn_s[i] = v;
      ss = fmaf(v, v, ss);
    }
  }
  const float r = 1.f / sqrtf(block_sum(ss, red) / (float)size + eps);
  for (int i = threadIdx.x * VEC; i < size; i += GN_THREADS * VEC) {
    if constexpr (VEC == 4) {
      const float4 v = *reinterpret_cast<const float4*>(gn_s + i), ww = *reinterpret_cast<const float4*>(w + c0 + i);
      Elem<T>::store4(out + row * ldo + c0 + i, make_float4(v.x * r * ww.x, v.y * r * ww.y, v.z * r * ww.z, v.w * r * ww.w));
    } else {
      out[row * ldo + c0 + i] = Elem<T>::from(gn_s[i] * r * w[c0 + i]);
    }
  }
  if (part == parts - 1)
    for (int i = inner + threadIdx.x; i < ko; i += GN_THREADS) out[row * ldo + i] = Elem<T>::from(0.f);
}

}  // namespace fb

using namespace fb;

// y: fp32 rows of heads * V, ldy apart; conv_w [taps][channels]; A = -exp(A_log). Returns -20 for a state of more than 512 rows.
extern "C" int fb_ssm_step(float* y, long ldy, float* rec, const void* tails, long tail_step, const void* proj, long ldp, const float* conv_w,
                           const float* conv_b, const float* A, const float* dt_bias, const float* skip, const int* seg_slot, const int* seg_row0,
                           const int* seg_nrows, int nseg, int heads, int groups, int N, int V, int taps, int commit, int f32, cudaStream_t s) {
  if (nseg <= 0) return 0;
  if (heads < 1 || groups < 1 || heads % groups || N < 1 || V < 1 || taps < 1 || heads > 65535) return -1;
  if (N > 512) return -20;
  const dim3 grid(nseg, heads, (V + SS_COLS - 1) / SS_COLS);
  const size_t smem = (size_t)2 * ((SS_COLS + 2 * N + 3) & ~3) * 4;
  auto go = [&](auto kern, auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    return (int)launch_pdl(kern, grid, dim3(SS_THREADS), smem, s, y, ldy, rec, (const T*)tails, tail_step, (const T*)proj, ldp, conv_w, conv_b, A,
                           dt_bias, skip, seg_slot, seg_row0, seg_nrows, heads, groups, N, V, taps, commit);
  };
#define FB_SS(NR) (f32 ? go(ssm_step_kernel<float, NR>, (float*)0) : go(ssm_step_kernel<bf16, NR>, (bf16*)0))
  return N <= 32 ? FB_SS(1) : N <= 64 ? FB_SS(2) : N <= 128 ? FB_SS(4) : N <= 256 ? FB_SS(8) : FB_SS(16);
#undef FB_SS
}

// proj: rows ldp apart, z in the first `inner` columns, the convolution's inputs in the next `ch`; out [rows][ko] with zeros beyond inner.
// tails: null, or the tails that every row joins
extern "C" int fb_group_norm_gated(void* out, long ldo, const float* y, long ldy, const void* proj, long ldp, const float* w, int rows, int inner,
                                   int parts, int ko, float eps, void* tails, long tail_step, int taps, int ch, const int* row_slot, int f32,
                                   cudaStream_t s) {
  if (rows <= 0) return 0;
  if (parts < 1 || inner % parts || ko < inner || parts > 65535 || (long)inner / parts > 49152 || (tails && (taps < 2 || !row_slot))) return -1;
  const int size = inner / parts, blocks = parts + (tails ? (ch + GN_TAIL - 1) / GN_TAIL : 0);
  const size_t smem = (size_t)size * 4, item = f32 ? 4 : 2;
  const bool vec = size % 4 == 0 && ldo % 4 == 0 && ldy % 4 == 0 && ldp % 4 == 0 && (((uintptr_t)y | (uintptr_t)w) & 15) == 0 &&
                   (((uintptr_t)out | (uintptr_t)proj) & (4 * item - 1)) == 0;
  auto go = [&](auto kern, auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    if (smem > 40 * 1024) {
      const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return (int)e;
    }
    return (int)launch_pdl(kern, dim3(rows, blocks), dim3(GN_THREADS), smem, s, (T*)out, ldo, y, ldy, (const T*)proj, ldp, w, inner,
                           parts, ko, eps, (T*)tails, tail_step, taps, ch, row_slot);
  };
  if (vec) return f32 ? go(group_norm_gated_kernel<float, 4>, (float*)0) : go(group_norm_gated_kernel<bf16, 4>, (bf16*)0);
  return f32 ? go(group_norm_gated_kernel<float, 1>, (float*)0) : go(group_norm_gated_kernel<bf16, 1>, (bf16*)0);
}
