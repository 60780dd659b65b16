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

// Count, mean and sum of squared deviations of a part of a row; parts are joined pairwise, so nothing cancels.
struct RowStats { float n, mean, m2; };
__device__ __forceinline__ RowStats cr_join(RowStats a, RowStats b) {
  const float n = a.n + b.n, f = n > 0.f ? b.n / n : 0.f, d = b.mean - a.mean;
  return {n, fmaf(d, f, a.mean), a.m2 + b.m2 + d * d * a.n * f};
}
__device__ __forceinline__ RowStats cr_warp(RowStats s) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1)
    s = cr_join(s, {__shfl_xor_sync(0xffffffffu, s.n, o), __shfl_xor_sync(0xffffffffu, s.mean, o), __shfl_xor_sync(0xffffffffu, s.m2, o)});
  return s;
}
// ... of four columns, of which `left` are inside the row's true width
__device__ __forceinline__ RowStats cr_quad(const float4& v, int left) {
  const float c[4] = {v.x, v.y, v.z, v.w};
  RowStats t{0.f, 0.f, 0.f};
  if (left >= 4) {
    t.n = 4.f;
    t.mean = 0.25f * ((c[0] + c[1]) + (c[2] + c[3]));
#pragma unroll
    for (int e = 0; e < 4; ++e) t.m2 = fmaf(c[e] - t.mean, c[e] - t.mean, t.m2);
  } else {
#pragma unroll
    for (int e = 0; e < 3; ++e)
      if (e < left) t = cr_join(t, {1.f, c[e], 0.f});
  }
  return t;
}
// (mean, 1 / deviation) of what all threads of the CTA hold
__device__ __forceinline__ float2 cr_block(RowStats s, int width, float eps, RowStats* red) {
  s = cr_warp(s);
  const int lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  __syncthreads();
  if (lane == 0) red[threadIdx.x >> 5] = s;
  __syncthreads();
  s = cr_warp(lane < warps ? red[lane] : RowStats{0.f, 0.f, 0.f});
  return make_float2(s.mean, 1.f / sqrtf(s.m2 / (float)width + eps));
}
// columns i + e < width, i = 4 (threadIdx.x + k blockDim.x), in v[k]
template <int NV>
__device__ __forceinline__ float2 cr_stats(const float4 (&v)[NV], int width, float eps, RowStats* red) {
  RowStats s = cr_quad(v[0], width - 4 * (int)threadIdx.x);
#pragma unroll
  for (int k = 1; k < NV; ++k) s = cr_join(s, cr_quad(v[k], width - 4 * (int)(threadIdx.x + k * blockDim.x)));
  return cr_block(s, width, eps, red);
}

// The pass of steps whose segments have several rows: many small CTAs, the row waits in shared memory between the norms (every thread reads what
// it wrote itself), so that one CTA's barriers hide behind another's loads.
constexpr int CN_ROW_THREADS = 256;

__device__ __forceinline__ float2 cr_row_stats(const float* row, int width, int ld, float eps, RowStats* red) {
  RowStats s{0.f, 0.f, 0.f};
  for (int i = threadIdx.x * 4; i < ld; i += CN_ROW_THREADS * 4) {
    s = cr_join(s, cr_quad(*reinterpret_cast<const float4*>(row + i), width - i));
  }
  return cr_block(s, width, eps, red);
}

template <typename T>
__global__ void __launch_bounds__(CN_ROW_THREADS)
add_rows_normed_kernel(const float* __restrict__ x_in, float* __restrict__ x, const float* __restrict__ y, long ldy, const float* __restrict__ yp,
                       const float* __restrict__ wts, int top, const float* __restrict__ w, float* __restrict__ xs, long xs_step, int place,
                       const float* __restrict__ dwa, const float* __restrict__ next_w, T* __restrict__ h_out, int width, int ld, float eps) {
  extern __shared__ __align__(16) float cr_row[];
  __shared__ RowStats red[32];
  pdl_launch_dependents();
  pdl_wait();
  x_in = after_wait(x_in); y = after_wait(y); yp = after_wait(yp); wts = after_wait(wts);
  const size_t row = blockIdx.x;
  const float* xi = x_in + row * ld;
  if (w) {
    for (int i = threadIdx.x * 4; i < ld; i += CN_ROW_THREADS * 4) {
      float4 s = y ? *reinterpret_cast<const float4*>(y + row * ldy + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      for (int k = 0; k < top; ++k) {
        const float g = wts[row * top + k];
        const float4 e = *reinterpret_cast<const float4*>(yp + (row * top + k) * ld + i);
        s.x = fmaf(g, e.x, s.x); s.y = fmaf(g, e.y, s.y); s.z = fmaf(g, e.z, s.z); s.w = fmaf(g, e.w, s.w);
      }
      *reinterpret_cast<float4*>(cr_row + i) = s;
    }
    const float2 st = cr_row_stats(cr_row, width, ld, eps, red);
    const float last = xs ? dwa[place] : 1.f;
    for (int i = threadIdx.x * 4; i < ld; i += CN_ROW_THREADS * 4) {
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
    }
  } else {
    for (int i = threadIdx.x * 4; i < ld; i += CN_ROW_THREADS * 4)
      *reinterpret_cast<float4*>(cr_row + i) = *reinterpret_cast<const float4*>(xi + i);
  }
  if (!next_w) return;
  const float2 st = cr_row_stats(cr_row, width, ld, eps, red);
  for (int i = threadIdx.x * 4; i < ld; i += CN_ROW_THREADS * 4) {
    const float4 v = *reinterpret_cast<const float4*>(cr_row + i), ww = *reinterpret_cast<const float4*>(next_w + i);
    Elem<T>::store4(h_out + row * ld + i, make_float4((v.x - st.x) * st.y * ww.x, (v.y - st.x) * st.y * ww.y, (v.z - st.x) * st.y * ww.z,
                                                      (v.w - st.x) * st.y * ww.w));
  }
}

// The pass of steps whose segments are one row each, with the convolution on it. NV: groups of four columns per thread, the whole row in
// registers. What does not come from the kernel before this one (weights) is read while that drains, what no norm has to wait for (results,
// tails) before the norms.
constexpr int cn_threads(int nv) { return nv == 16 ? 1024 : 512; }

template <typename T, int NV>
__global__ void __launch_bounds__(cn_threads(NV))
add_conv_normed_kernel(const float* __restrict__ x_in, float* __restrict__ x, const float* __restrict__ y, long ldy, const float* __restrict__ yp,
                       const float* __restrict__ wts, int top, const float* __restrict__ w, float* __restrict__ xs, long xs_step, int place,
                       const float* __restrict__ dwa, const float* __restrict__ next_w, T* __restrict__ h_out, T* __restrict__ xb,
                       const float* __restrict__ cw, int taps, T* __restrict__ tails, long tail_step, const int* __restrict__ row_slot, int commit,
                       int width, int ld, float eps) {
  constexpr bool EARLY = NV == 1;
  constexpr int PART = 4;                                    // expert rows, results and taps read at a time
  __shared__ RowStats red[32];
  pdl_launch_dependents();
  const size_t row = blockIdx.x;
  auto col = [&](int k) { return 4 * (threadIdx.x + k * (int)blockDim.x); };
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  auto load = [&](const float* p, int i) { return i < ld ? *reinterpret_cast<const float4*>(p + i) : zero; };
  auto axpy = [](float4& a, float g, const float4& b) {
    a.x = fmaf(g, b.x, a.x); a.y = fmaf(g, b.y, a.y); a.z = fmaf(g, b.z, a.z); a.w = fmaf(g, b.w, a.w);
  };
  float4 w_own = zero, next_own = zero, conv_own[EARLY ? PART : 1];
  if (EARLY) {
    if (w) w_own = load(w, col(0));
    if (next_w) next_own = load(next_w, col(0));
#pragma unroll
    for (int j = 0; j < PART; ++j) conv_own[EARLY ? j : 0] = j < taps && taps <= PART ? load(cw + (size_t)j * ld, col(0)) : zero;
  }
  const float last = xs ? dwa[place] : 1.f;
  const int slot = row_slot[row];
  T* tail = tails + slot * tail_step;
#pragma unroll
  for (int k = 0; k < NV; ++k) {                             // lines that nobody has touched since the last step
    const int i = col(k);
    if (i >= ld) break;
    if (i % 32 == 0) {
      if (!EARLY) {
        if (w) prefetch_l2(w + i);
        if (next_w) prefetch_l2(next_w + i);
        for (int j = 0; j < taps; ++j) prefetch_l2(cw + (size_t)j * ld + i);
      }
      if (xs)
        for (int j = 0; j < place; ++j) prefetch_l2(xs + j * xs_step + row * ld + i);
    }
    if (i % (128 / (int)sizeof(T)) == 0)
      for (int j = 0; j + 1 < taps; ++j) prefetch_l2(tail + (size_t)j * ld + i);
  }
  pdl_wait();
  x_in = after_wait(x_in); y = after_wait(y); yp = after_wait(yp); wts = after_wait(wts);
  float4 v[NV], f[NV], past[NV];
  float4 tail_own[EARLY ? PART - 1 : 1];
  if (EARLY && next_w) {
#pragma unroll
    for (int j = 0; j < PART - 1; ++j)
      tail_own[EARLY ? j : 0] = j + 1 < taps && taps <= PART && col(0) < ld ? Elem<T>::load4(tail + (size_t)j * ld + col(0)) : zero;
  }
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int i = col(k);
    v[k] = load(x_in + row * ld, i);
    f[k] = w && y ? load(y + row * ldy, i) : zero;
    past[k] = zero;
    for (int p0 = 0; p0 < top; p0 += PART) {
      float g[PART];
      float4 e[PART];
#pragma unroll
      for (int j = 0; j < PART; ++j) {
        const size_t r = row * top + p0 + j;
        g[j] = p0 + j < top ? wts[r] : 0.f;
        e[j] = p0 + j < top ? load(yp + r * ld, i) : zero;
      }
#pragma unroll
      for (int j = 0; j < PART; ++j) axpy(f[k], g[j], e[j]);
    }
    if (xs && i < ld) {                                      // earlier results
      const float* xr = xs + row * ld + i;
      for (int j0 = 0; j0 < place; j0 += PART) {
        float4 r[PART];
#pragma unroll
        for (int j = 0; j < PART; ++j) r[j] = j0 + j < place ? *reinterpret_cast<const float4*>(xr + (j0 + j) * xs_step) : zero;
#pragma unroll
        for (int j = 0; j < PART; ++j) axpy(past[k], j0 + j < place ? dwa[j0 + j] : 0.f, r[j]);
      }
    }
  }
  if (w) {                                                   // the sublayer's output, its norm, the residual sum
    const float2 st = cr_stats<NV>(f, width, eps, red);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int i = col(k);
      const float4 ww = EARLY ? w_own : load(w, i);
      v[k].x += (f[k].x - st.x) * st.y * ww.x; v[k].y += (f[k].y - st.x) * st.y * ww.y;
      v[k].z += (f[k].z - st.x) * st.y * ww.z; v[k].w += (f[k].w - st.x) * st.y * ww.w;
      if (i >= ld) continue;
      if (xs) {                                              // this layer's result, then the sum over depth
        *reinterpret_cast<float4*>(xs + place * xs_step + row * ld + i) = v[k];
        axpy(past[k], last, v[k]);
        v[k] = past[k];
      }
      *reinterpret_cast<float4*>(x + row * ld + i) = v[k];
    }
  }
  if (!next_w) return;
  const float2 st = cr_stats<NV>(v, width, eps, red);
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int i = col(k);
    if (i >= ld) continue;
    const float4 nw = EARLY ? next_own : load(next_w, i);
    T h4[4] = {Elem<T>::from((v[k].x - st.x) * st.y * nw.x), Elem<T>::from((v[k].y - st.x) * st.y * nw.y),
               Elem<T>::from((v[k].z - st.x) * st.y * nw.z), Elem<T>::from((v[k].w - st.x) * st.y * nw.w)};
    const float4 h = make_float4(Elem<T>::to(h4[0]), Elem<T>::to(h4[1]), Elem<T>::to(h4[2]), Elem<T>::to(h4[3]));
    if (h_out) Elem<T>::store4(h_out + row * ld + i, h);
    float4 o = h;
    auto tap = [&](int j, const float4& c, const float4& p) {
      o.x = fmaf(c.x, p.x, o.x); o.y = fmaf(c.y, p.y, o.y); o.z = fmaf(c.z, p.z, o.z); o.w = fmaf(c.w, p.w, o.w);
      if (commit && j > 0) Elem<T>::store4(tail + (size_t)(j - 1) * ld + i, p);
    };
    if (EARLY && taps <= PART) {
#pragma unroll
      for (int j = 0; j < PART; ++j)
        if (j < taps) tap(j, conv_own[EARLY ? j : 0], j + 1 < taps ? tail_own[EARLY && j < PART - 1 ? j : 0] : h);
    } else {
      for (int j = 0; j < taps; ++j) {
        const float4 p = j + 1 < taps ? Elem<T>::load4(tail + (size_t)j * ld + i) : h;
        tap(j, *reinterpret_cast<const float4*>(cw + (size_t)j * ld + i), p);
      }
    }
    Elem<T>::store4(xb + row * ld + i, o);
  }
}

// TAPS: taps known at compile time, 0 = any. grid (column blocks, strips of CR_ROWS rows). A row's predecessors are those of the step while slot and position go on, the tail's beyond.
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
  float bs[VEC];
#pragma unroll
  for (int e = 0; e < VEC; ++e) bs[e] = bias ? bias[c0 + e] : 0.f;
  auto finish = [&](int r, float (&acc)[VEC], const float (&cur)[VEC]) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      if (silu) acc[e] = acc[e] / (1.f + __expf(-acc[e]));
      if (residual) acc[e] += cur[e];
    }
    if constexpr (VEC == 4) Elem<T>::store4(out + (size_t)r * ldo + c0, make_float4(acc[0], acc[1], acc[2], acc[3]));
    else out[(size_t)r * ldo + c0] = Elem<T>::from(acc[0]);
  };
  if constexpr (TAPS > 0) {
    // all rows of the strip and the TAPS - 1 before it are read at once, those of another segment or of a tail replaced where one starts
    using Raw = std::conditional_t<VEC == 1, T, std::conditional_t<sizeof(T) == 4, float4, uint2>>;      // VEC values as they lie in memory
    float wt[TAPS][VEC];
    Raw in[TAPS - 1 + CR_ROWS];
    auto fetch = [](const T* p) { return *reinterpret_cast<const Raw*>(p); };
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
      for (int e = 0; e < VEC; ++e) wt[j][e] = w[(size_t)j * C + c0 + e];
#pragma unroll
    for (int j = 0; j < TAPS - 1 + CR_ROWS; ++j) {
      const int r = r0 + j - (TAPS - 1);
      if (r >= 0 && r < rows) in[j] = fetch(x + (size_t)r * ldx + c0);
    }
#pragma unroll
    for (int i = 0; i < CR_ROWS; ++i) {
      if (i >= here) break;
      const int n = before[i];
      if (n < TAPS - 1) {                                    // close behind a segment's start: the rows before it are the tail's
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) {
          const int back = TAPS - 1 - j;
          if (back > n) in[i + j] = fetch(tails + slots[i] * tail_step + (size_t)(TAPS - 1 - (back - n)) * C + c0);
        }
      }
      float acc[VEC], cur[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[e] = bs[e];
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        load(reinterpret_cast<const T*>(&in[i + j]), cur);
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc[e] = fmaf(wt[j][e], cur[e], acc[e]);
      }
      finish(r0 + i, acc, cur);
    }
  } else {
    for (int i = 0; i < here; ++i) {
      const int r = r0 + i, n = before[i];
      float acc[VEC], cur[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[e] = bs[e];
      for (int j = 0; j < taps; ++j) {                       // tap j meets the row taps - 1 - j back
        const int back = taps - 1 - j;
        load(back <= n ? x + (size_t)(r - back) * ldx + c0 : tails + slots[i] * tail_step + (size_t)(taps - 1 - (back - n)) * C + c0, cur);
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc[e] = fmaf(w[(size_t)j * C + c0 + e], cur[e], acc[e]);
      }
      finish(r, acc, cur);
    }
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
  if (!xb) {
    const size_t smem = (size_t)ld * 4;
    auto go = [&](auto kern, auto* tag) {
      using T = std::remove_pointer_t<decltype(tag)>;
      if (smem > 40 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
      }
      return (int)launch_pdl(kern, dim3(rows), dim3(CN_ROW_THREADS), smem, s, x_in, x, y, ldy, yp, wts, top, w, xs, xs_step, place, dwa, next_w,
                             (T*)h_out, width, ld, eps);
    };
    return f32 ? go(add_rows_normed_kernel<float>, (float*)0) : go(add_rows_normed_kernel<bf16>, (bf16*)0);
  }
  const int quads = ld / 4;
  int nv = 1;
  while (nv < 16 && quads > cn_threads(nv) * nv) nv *= 2;
  if (quads > cn_threads(nv) * nv) return -1;
  const dim3 g(rows), b(((quads + nv - 1) / nv + 31) / 32 * 32);
  auto go = [&](auto kern, auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    return (int)launch_pdl(kern, g, b, 0, s, x_in, x, y, ldy, yp, wts, top, w, xs, xs_step, place, dwa, next_w, (T*)h_out, (T*)xb, cw, taps,
                           (T*)tails, tail_step, row_slot, commit, width, ld, eps);
  };
#define FB_CN(NV) (f32 ? go(add_conv_normed_kernel<float, NV>, (float*)0) : go(add_conv_normed_kernel<bf16, NV>, (bf16*)0))
  return nv == 1 ? FB_CN(1) : nv == 2 ? FB_CN(2) : nv == 4 ? FB_CN(4) : nv == 8 ? FB_CN(8) : FB_CN(16);
#undef FB_CN
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
