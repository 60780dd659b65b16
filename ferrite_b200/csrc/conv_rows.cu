// Row kernels of the models of listed layers whose sublayers read convolved operands (ops/latent.py states what each of them does):
//
//   add_conv_normed  x = x_in + layer norm of the sublayer's output (its 32-bit sums and the weighted rows of the chosen experts), the
//                    weighted sum over the results of all layers so far, the layer norm for the next sublayer and, where every segment is
//                    one row, the causal convolution on top of it: everything between two sublayers in one pass over a row
//   conv_rows        causal convolution per channel of a step's rows of any segments: plus the row itself, or with bias and silu
//   conv_tail        the last taps - 1 inputs of every segment's sequence become its slot's tail
//
// What lies before a segment comes out of the slot's tail [taps - 1][channels], oldest first, zeros before a sequence's start. Inputs
// are kept in the operand type, in the tail as in the step, so where a prompt is cut does not show.
#include "api_listed.h"
#include "common.cuh"
#include "elem.cuh"

namespace fb {

using bf16 = __nv_bfloat16;

// mean and 1 / deviation of a row of `width` true columns (zeros up to ld) that waits in shared memory
__device__ __forceinline__ float2 cr_stats(const float* row, float sum, int width, int ld, float eps, float* red) {
  const float mean = block_sum(sum, red) / (float)width;
  float ss = 0.f;
  for (int i = threadIdx.x * 4; i < ld; i += blockDim.x * 4) {
    const float4 v = *reinterpret_cast<const float4*>(row + i);
    const float d[4] = {v.x - mean, v.y - mean, v.z - mean, v.w - mean};
#pragma unroll
    for (int e = 0; e < 4; ++e)
      if (i + e < width) ss = fmaf(d[e], d[e], ss);
  }
  return make_float2(mean, 1.f / sqrtf(block_sum(ss, red) / (float)width + eps));
}

template <typename T>
__global__ void add_conv_normed_kernel(const float* __restrict__ x_in, float* __restrict__ x, const float* __restrict__ y, long ldy,
                                       const float* __restrict__ yp, const float* __restrict__ wts, int top, const float* __restrict__ w,
                                       float* __restrict__ xs, long xs_step, int place, const float* __restrict__ dwa,
                                       const float* __restrict__ next_w, T* __restrict__ h_out, T* __restrict__ xb, const float* __restrict__ cw,
                                       int taps, T* __restrict__ tails, long tail_step, const int* __restrict__ row_slot, int commit, int width,
                                       int ld, float eps) {
  extern __shared__ __align__(16) float cr_row[];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  x_in = after_wait(x_in); y = after_wait(y); yp = after_wait(yp); wts = after_wait(wts);
  const size_t row = blockIdx.x;
  const float* xi = x_in + row * ld;
  float sum = 0.f;
  if (w) {                                                   // the sublayer's output, its norm, the residual sum
    for (int i = threadIdx.x * 4; i < ld; i += blockDim.x * 4) {
      float4 s = y ? *reinterpret_cast<const float4*>(y + row * ldy + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      for (int k = 0; k < top; ++k) {
        const float g = wts[row * top + k];
        const float4 e = *reinterpret_cast<const float4*>(yp + (row * top + k) * ld + i);
        s.x = fmaf(g, e.x, s.x); s.y = fmaf(g, e.y, s.y); s.z = fmaf(g, e.z, s.z); s.w = fmaf(g, e.w, s.w);
      }
      *reinterpret_cast<float4*>(cr_row + i) = s;
      sum += (s.x + s.y) + (s.z + s.w);
    }
    const float2 st = cr_stats(cr_row, sum, width, ld, eps, red);
    sum = 0.f;
    const float last = xs ? dwa[place] : 1.f;
    for (int i = threadIdx.x * 4; i < ld; i += blockDim.x * 4) {
      const float4 f = *reinterpret_cast<const float4*>(cr_row + i), ww = *reinterpret_cast<const float4*>(w + i);
      float4 v = *reinterpret_cast<const float4*>(xi + i);
      v.x += (f.x - st.x) * st.y * ww.x; v.y += (f.y - st.x) * st.y * ww.y;
      v.z += (f.z - st.x) * st.y * ww.z; v.w += (f.w - st.x) * st.y * ww.w;
      if (xs) {                                              // this layer's result, then the sum over depth
        *reinterpret_cast<float4*>(xs + place * xs_step + row * ld + i) = v;
        v.x *= last; v.y *= last; v.z *= last; v.w *= last;
#pragma unroll 4
        for (int j = 0; j < place; ++j) {
          const float g = dwa[j];
          const float4 r = *reinterpret_cast<const float4*>(xs + j * xs_step + row * ld + i);
          v.x = fmaf(g, r.x, v.x); v.y = fmaf(g, r.y, v.y); v.z = fmaf(g, r.z, v.z); v.w = fmaf(g, r.w, v.w);
        }
      }
      *reinterpret_cast<float4*>(x + row * ld + i) = v;
      *reinterpret_cast<float4*>(cr_row + i) = v;
      sum += (v.x + v.y) + (v.z + v.w);
    }
  } else {
    for (int i = threadIdx.x * 4; i < ld; i += blockDim.x * 4) {
      const float4 v = *reinterpret_cast<const float4*>(xi + i);
      *reinterpret_cast<float4*>(cr_row + i) = v;
      sum += (v.x + v.y) + (v.z + v.w);
    }
  }
  if (!next_w) return;
  const float2 st = cr_stats(cr_row, sum, width, ld, eps, red);
  T* tail = xb ? tails + row_slot[row] * tail_step : nullptr;
  for (int i = threadIdx.x * 4; i < ld; i += blockDim.x * 4) {
    const float4 v = *reinterpret_cast<const float4*>(cr_row + i), ww = *reinterpret_cast<const float4*>(next_w + i);
    T h4[4] = {Elem<T>::from((v.x - st.x) * st.y * ww.x), Elem<T>::from((v.y - st.x) * st.y * ww.y),
               Elem<T>::from((v.z - st.x) * st.y * ww.z), Elem<T>::from((v.w - st.x) * st.y * ww.w)};
    const float4 h = make_float4(Elem<T>::to(h4[0]), Elem<T>::to(h4[1]), Elem<T>::to(h4[2]), Elem<T>::to(h4[3]));
    if (h_out) Elem<T>::store4(h_out + row * ld + i, h);
    if (!xb) continue;
    const float4 c = *reinterpret_cast<const float4*>(cw + (size_t)(taps - 1) * ld + i);
    float4 o = make_float4(fmaf(c.x, h.x, h.x), fmaf(c.y, h.y, h.y), fmaf(c.z, h.z, h.z), fmaf(c.w, h.w, h.w));
    for (int j = 0; j + 1 < taps; ++j) {
      const float4 p = Elem<T>::load4(tail + (size_t)j * ld + i), g = *reinterpret_cast<const float4*>(cw + (size_t)j * ld + i);
      o.x = fmaf(g.x, p.x, o.x); o.y = fmaf(g.y, p.y, o.y); o.z = fmaf(g.z, p.z, o.z); o.w = fmaf(g.w, p.w, o.w);
      if (commit && j > 0) Elem<T>::store4(tail + (size_t)(j - 1) * ld + i, p);
    }
    if (commit && taps > 1) Elem<T>::store4(tail + (size_t)(taps - 2) * ld + i, h);
    Elem<T>::store4(xb + row * ld + i, o);
  }
}

// grid (column blocks, strips of CR_ROWS rows). A row's predecessors are those of the step while slot and position go on, the tail's beyond.
constexpr int CR_ROWS = 8;

template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(256) conv_rows_kernel(T* __restrict__ out, long ldo, const T* __restrict__ x, long ldx, const float* __restrict__ w,
                                                        int taps_rt, int C, const T* __restrict__ tails, long tail_step,
                                                        const int* __restrict__ row_slot, const int* __restrict__ row_pos,
                                                        const float* __restrict__ bias, int silu, int residual, int rows) {
  const int taps = TAPS ? TAPS : taps_rt;
  __shared__ int before[CR_ROWS], slots[CR_ROWS];            // rows of the step that precede a row, up to taps - 1
  pdl_launch_dependents();
  pdl_wait();
  x = after_wait(x); tails = after_wait(tails);
  const int r0 = blockIdx.y * CR_ROWS, here = min(CR_ROWS, rows - r0);
  if (threadIdx.x < here) {
    const int r = r0 + threadIdx.x, s = row_slot[r], p = row_pos[r];
    int n = 0;
    while (n + 1 < taps && r - n - 1 >= 0 && row_slot[r - n - 1] == s && row_pos[r - n - 1] == p - n - 1) ++n;
    before[threadIdx.x] = n;
    slots[threadIdx.x] = s;
  }
  __syncthreads();
  const int c0 = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  if (c0 >= C) return;
  auto load = [&](const T* p, float (&v)[VEC]) {
    if constexpr (VEC == 4) {
      const float4 f = Elem<T>::load4(p);
      v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
    } else {
      v[0] = Elem<T>::to(*p);
    }
  };
  float wt[TAPS ? TAPS : 1][VEC], bs[VEC];
  if constexpr (TAPS > 0) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
      for (int e = 0; e < VEC; ++e) wt[j][e] = w[(size_t)j * C + c0 + e];
  }
#pragma unroll
  for (int e = 0; e < VEC; ++e) bs[e] = bias ? bias[c0 + e] : 0.f;
  for (int i = 0; i < here; ++i) {
    const int r = r0 + i, n = before[i];
    float acc[VEC], cur[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) acc[e] = bs[e];
#pragma unroll
    for (int j = 0; j < taps; ++j) {                         // tap j meets the row taps - 1 - j back
      const int back = taps - 1 - j;
      float v[VEC];
      load(back <= n ? x + (size_t)(r - back) * ldx + c0 : tails + slots[i] * tail_step + (size_t)(taps - 1 - (back - n)) * C + c0, v);
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[e] = fmaf(TAPS ? wt[TAPS ? j : 0][e] : w[(size_t)j * C + c0 + e], v[e], acc[e]);
      if (back == 0) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) cur[e] = v[e];
      }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      if (silu) acc[e] = acc[e] / (1.f + expf(-acc[e]));
      if (residual) acc[e] += cur[e];
    }
    if constexpr (VEC == 4) Elem<T>::store4(out + (size_t)r * ldo + c0, make_float4(acc[0], acc[1], acc[2], acc[3]));
    else out[(size_t)r * ldo + c0] = Elem<T>::from(acc[0]);
  }
}

template <typename T>
__global__ void __launch_bounds__(256) conv_tail_kernel(T* __restrict__ tails, long tail_step, int taps, const T* __restrict__ x, long ldx, int C,
                                                        const int* __restrict__ seg_slot, const int* __restrict__ seg_row0,
                                                        const int* __restrict__ seg_nrows) {
  pdl_launch_dependents();
  pdl_wait();
  x = after_wait(x);
  const int c = blockIdx.x * blockDim.x + threadIdx.x, s = blockIdx.y, n = seg_nrows[s], K = taps - 1;
  if (c >= C || n <= 0) return;
  T* t = tails + seg_slot[s] * tail_step + c;
  const T* xr = x + (size_t)seg_row0[s] * ldx + c;
  for (int j = 0; j < K; ++j) t[(size_t)j * C] = n + j < K ? t[(size_t)(n + j) * C] : xr[(size_t)(n + j - K) * ldx];
}

}  // namespace fb

using namespace fb;

// y: rows ldy floats apart, or null; yp / wts: rows of a token's `top` experts and their weights (top 0: none); w: weights of the output's
// norm, null: x stays and x_in is what is normed. xs: results of the layers, xs_step floats apart, and the weights dwa of the first place + 1
// of them, or null. next_w null: no operand. h_out: the next norm's rows, or null; xb: the convolved operand (cw [taps][ld], tails of every
// slot tail_step elements apart, one row per segment), or null.
extern "C" int fb_add_conv_normed(const float* x_in, float* x, const float* y, long ldy, const float* yp, const float* wts, int top, const float* w,
                                  float* xs, long xs_step, int place, const float* dwa, const float* next_w, void* h_out, void* xb,
                                  const float* cw, int taps, void* tails, long tail_step, const int* row_slot, int commit, int rows, int width,
                                  int ld, float eps, int f32, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (ld % 4 || ldy % 4 || ld > 49152 || width < 1 || width > ld || (top && (!yp || !wts)) || (w && !y && !top) || (xs && (!dwa || !w || place < 0)) ||
      (next_w && !h_out && !xb) || (xb && (!cw || taps < 1 || !row_slot || (taps > 1 && (!tails || tail_step % 4))))) return -1;
  const size_t smem = (size_t)ld * 4;
  const dim3 g(rows), b(ld >= 4096 ? 512 : ld >= 1024 ? 256 : 128);
  auto go = [&](auto kern, auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    if (smem > 40 * 1024) {
      const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return (int)e;
    }
    return (int)launch_pdl(kern, g, b, smem, s, x_in, x, y, ldy, yp, wts, top, w, xs, xs_step, place, dwa, next_w, (T*)h_out, (T*)xb, cw, taps,
                           (T*)tails, tail_step, row_slot, commit, width, ld, eps);
  };
  return f32 ? go(add_conv_normed_kernel<float>, (float*)0) : go(add_conv_normed_kernel<bf16>, (bf16*)0);
}

// out [rows][C] (ldo elements apart) from x (ldx), w [taps][C]; bias: C floats or null
extern "C" int fb_conv_rows(void* out, long ldo, const void* x, long ldx, const float* w, int taps, int C, const void* tails, long tail_step,
                            const int* row_slot, const int* row_pos, const float* bias, int silu, int residual, int rows, int f32,
                            cudaStream_t s) {
  if (rows <= 0) return 0;
  if (taps < 1 || C < 1 || (taps > 1 && !tails) || (rows + CR_ROWS - 1) / CR_ROWS > 65535) return -1;
  const size_t item = f32 ? 4 : 2;
  const bool vec = C % 4 == 0 && ldx % 4 == 0 && ldo % 4 == 0 && tail_step % 4 == 0 &&
                   (((uintptr_t)x | (uintptr_t)out | (uintptr_t)tails) & (4 * item - 1)) == 0;
  auto go = [&](auto kern, auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    const int per = 256 * (vec ? 4 : 1);
    return (int)launch_pdl(kern, dim3((C + per - 1) / per, (rows + CR_ROWS - 1) / CR_ROWS), dim3(256), 0, s, (T*)out, ldo, (const T*)x, ldx, w, taps,
                           C, (const T*)tails, tail_step, row_slot, row_pos, bias, silu, residual, rows);
  };
  if (vec && taps == 4) return f32 ? go(conv_rows_kernel<float, 4, 4>, (float*)0) : go(conv_rows_kernel<bf16, 4, 4>, (bf16*)0);
  if (vec) return f32 ? go(conv_rows_kernel<float, 4, 0>, (float*)0) : go(conv_rows_kernel<bf16, 4, 0>, (bf16*)0);
  return f32 ? go(conv_rows_kernel<float, 1, 0>, (float*)0) : go(conv_rows_kernel<bf16, 1, 0>, (bf16*)0);
}

extern "C" int fb_conv_tail(void* tails, long tail_step, int taps, const void* x, long ldx, int C, const int* seg_slot, const int* seg_row0,
                            const int* seg_nrows, int nseg, int f32, cudaStream_t s) {
  if (nseg <= 0 || taps <= 1) return 0;
  if (C < 1 || nseg > 65535) return -1;
  const dim3 g((C + 255) / 256, nseg);
  if (f32) return (int)launch_pdl(conv_tail_kernel<float>, g, dim3(256), 0, s, (float*)tails, tail_step, taps, (const float*)x, ldx, C, seg_slot, seg_row0, seg_nrows);
  return (int)launch_pdl(conv_tail_kernel<bf16>, g, dim3(256), 0, s, (bf16*)tails, tail_step, taps, (const bf16*)x, ldx, C, seg_slot, seg_row0, seg_nrows);
}
