// Shared pieces of the channel-delta kernels (`cdelta.cu`, `cdelta_chunk.cu`): the gated delta rule with one decay per head and
// key channel,
//   S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q,
// q, k unit vectors per head (q also times dim^-1/2) of short-convolved projections, v a short-convolved projection,
// g = exp(-exp(A_log) softplus(decay + dt_bias)), beta = sigmoid(b). Everything but the projections and the convolutions with
// their activations is 32-bit.
#pragma once
#include "common.cuh"
#include "elem.cuh"

namespace fb {

constexpr int CD_TAPS = 8;              // most taps of a short convolution; kernels come with room for NT = 4 and for all of them
constexpr float CD_UNIT_EPS = 1e-6f;

// Columns of the fused projection row [a1 (ra) | g1 (rg) | q (kv_heads dim) | k | v (heads vdim) | b (heads)]
struct CdLayer {
  int heads, kv_heads, dim, vdim, taps;
  int q_off;                            // ra + rg
  __host__ __device__ int channels() const { return 2 * kv_heads * dim + heads * vdim; }
  __host__ __device__ int k_off() const { return q_off + kv_heads * dim; }
  __host__ __device__ int v_off() const { return q_off + 2 * kv_heads * dim; }
  __host__ __device__ int b_off() const { return q_off + channels(); }
};

__device__ __forceinline__ float cd_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float cd_silu(float x) { return x / (1.f + expf(-x)); }
// log of a decay
__device__ __forceinline__ float cd_log_decay(float expA, float z) { return -expA * (fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)))); }

// Taps of channel c, right-aligned in NT registers
template <int NT>
__device__ __forceinline__ void cd_load_taps(float (&w)[NT], const float* conv_w, int c, int taps) {
#pragma unroll
  for (int j = 0; j < NT; ++j) {
    const int i = j - (NT - taps);
    w[j] = i >= 0 ? conv_w[(size_t)c * taps + i] : 0.f;
  }
}
// Raw input of channel c at row r of a segment; r < 0 reaches into the slot's tail (taps - 1 rows, oldest first)
template <typename T>
__device__ __forceinline__ float cd_input(const T* proj, long ldp, int q_off, const T* tail, int channels, int taps, int row0, int r, int c) {
  if (r >= 0) return Elem<T>::to(proj[(size_t)(row0 + r) * ldp + q_off + c]);
  return r >= 1 - taps ? Elem<T>::to(tail[(size_t)(taps - 1 + r) * channels + c]) : 0.f;
}
// One step of the sliding window: the activated convolution, rounded to the type that the prompt kernels keep it in
template <typename T, int NT>
__device__ __forceinline__ float cd_conv_step(const float (&w)[NT], float (&win)[NT - 1], float x) {
  float a = w[NT - 1] * x;
#pragma unroll
  for (int j = 0; j < NT - 1; ++j) a = fmaf(w[j], win[j], a);
#pragma unroll
  for (int j = 0; j < NT - 2; ++j) win[j] = win[j + 1];
  win[NT - 2] = x;
  return Elem<T>::to(Elem<T>::from(cd_silu(a)));
}

}  // namespace fb
