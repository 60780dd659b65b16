// Channel-delta layers, prompt segments: the recurrence of cdelta.cuh over chunks of C = 64 rows. With G_t = sum_{i <= t} log g_i (a
// vector over the key channels, inside the chunk) and S_0 the state the chunk starts from:
//   (I + A) D = diag(beta) B,   B = V - K~ S_0,   K~_t = k_t e^{G_t},   A[t][i] = beta_t sum_c k_t[c] k_i[c] e^{G_t[c] - G_i[c]}  (i < t)
//   O = Q~ S_0 + P D,                             Q~_t = q_t e^{G_t},   P[t][i] = sum_c q_t[c] k_i[c] e^{G_t[c] - G_i[c]}         (i <= t)
//   S_C = diag(e^{G_C}) S_0 + sum_i k_i e^{G_C - G_i} d_i^T
// prep (parallel over chunks x heads) forms K~, Q~, k e^{G_C - G}, T' = (I + A)^{-1} diag(beta) and P T'; scan (serial over the chunks of
// a segment, parallel over heads x slices of state columns) runs the products with S: [K~; Q~] S, then D = T' B and O beside one
// another, then the new state.
//
// The weights e^{G_t - G_i} need care: decays may be as strong as e^{-200} per token, so neither e^{-G_i} nor a difference of long sums
// of logarithms will do. Every pair (t, i) has one level L in {32, 16, 8, 4, 2, 1} at which t lies in the upper and i in the lower half
// of an aligned block of 2 L rows; with m the last row of the lower half the weight is e^{sum(m+1 .. t)} e^{sum(i+1 .. m)}: two factors
// in [0, 1], each from a short sum of terms of one sign, one exponential per row, channel and level.
//
// Products run in fp32 FMA: the state carries hundreds of chunks. Convolutions and activations happen in place (prep: q and k of its
// head; scan: its slice of v), so nothing of them goes through memory.
#include "api_ext.h"
#include "cdelta.cuh"

#include <type_traits>

namespace fb {

constexpr int CC = 64;                  // rows per chunk
constexpr int CP_THREADS = 512;

__device__ __forceinline__ void cc_cp16(void* smem, const void* gmem) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem)), "l"(gmem) : "memory");
}
__device__ __forceinline__ void cc_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cc_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// One (chunk, head) of the scratch: floats Kt [C][DKP] | Qt [C][DKP] | Kh [C][DKP] | T' [C][C] | P T' [C][C] | eC [DKP]
__host__ __device__ constexpr long cc_rec_floats(int dkp) { return 3l * CC * dkp + 2l * CC * CC + dkp; }

// ---- prep --------------------------------------------------------------------------------------------------------------------
template <typename T, int DKP>
struct PrepSmem {
  static constexpr int LDR = DKP + 16 / sizeof(T);          // raw rows
  static constexpr int LDK = DKP + 4, LDA = CC + 4;
  static constexpr size_t BYTES = (size_t)2 * CC * LDR * sizeof(T) + ((size_t)3 * CC * LDK + 2 * CC * LDA + 3 * CC) * 4;
};

// Pairs of level LV: a thread takes TT upper rows against one lower row over its share of the channels.
template <int DKP, int LDK, int LDA, int LV>
__device__ __forceinline__ void cc_level_pairs(float* Am, float* Pm, const float* Ks, const float* Qs, const float* rk, const float* rq,
                                               const float* bs) {
  constexpr int TT = LV < 4 ? LV : 4, UNITS = CC / 2 * LV / TT, LANES = CP_THREADS / UNITS, STEPS = DKP / 4 / LANES > 0 ? DKP / 4 / LANES : 1;
  static_assert(UNITS * LANES == CP_THREADS && STEPS * LANES >= DKP / 4, "shares");
  const int sub = threadIdx.x % LANES, u = threadIdx.x / LANES;
  const int blk = u / (LV * LV / TT), in = u % (LV * LV / TT);
  const int t0 = blk * 2 * LV + LV + in / LV * TT, i = blk * 2 * LV + in % LV;
  float a[TT] = {}, b[TT] = {};
#pragma unroll
  for (int st = 0; st < STEPS; ++st) {
    const int c = (sub + st * LANES) * 4;
    if (STEPS * LANES > DKP / 4 && c >= DKP) break;
    const float4 z = *reinterpret_cast<const float4*>(Ks + i * LDK + c);
#pragma unroll
    for (int e = 0; e < TT; ++e) {
      const float4 x = *reinterpret_cast<const float4*>(Ks + (t0 + e) * LDK + c), y = *reinterpret_cast<const float4*>(Qs + (t0 + e) * LDK + c);
      a[e] = fmaf(x.x, z.x, fmaf(x.y, z.y, fmaf(x.z, z.z, fmaf(x.w, z.w, a[e]))));
      b[e] = fmaf(y.x, z.x, fmaf(y.y, z.y, fmaf(y.z, z.z, fmaf(y.w, z.w, b[e]))));
    }
  }
#pragma unroll
  for (int e = 0; e < TT; ++e) {
#pragma unroll
    for (int o = LANES / 2; o > 0; o >>= 1) {
      a[e] += __shfl_xor_sync(0xffffffffu, a[e], o);
      b[e] += __shfl_xor_sync(0xffffffffu, b[e], o);
    }
    if (sub == e % LANES) {
      const int t = t0 + e;
      Am[t * LDA + i] = bs[t] * rk[t] * rk[i] * a[e];
      Pm[t * LDA + i] = rq[t] * rk[i] * b[e];
    }
  }
}

template <typename T, int DKP, int NT>
__global__ void __launch_bounds__(CP_THREADS)
cd_chunk_prep_kernel(float* __restrict__ scratch, const T* __restrict__ proj, long ldp, const float* __restrict__ decay, long ldd,
                     const float* __restrict__ conv_w, const float* __restrict__ A_log, const float* __restrict__ dt_bias,
                     const T* __restrict__ conv_state, const int* __restrict__ seg_slot, const int* __restrict__ seg_row0,
                     const int* __restrict__ seg_nrows, CdLayer L) {
  using M = PrepSmem<T, DKP>;
  constexpr int LDR = M::LDR, LDK = M::LDK, LDA = M::LDA, GROUPS = CP_THREADS / DKP;
  extern __shared__ __align__(16) unsigned char cp_smem[];
  T* Kr = reinterpret_cast<T*>(cp_smem);                    // [C][LDR] convolved k, q
  T* Qr = Kr + CC * LDR;
  float* lg = reinterpret_cast<float*>(Qr + CC * LDR);      // [C][LDK] log decays
  float* Ks = lg + CC * LDK;                                // [C][LDK] weighted k, q of a level (later: T by 16-row blocks)
  float* Qs = Ks + CC * LDK;
  float* Am = Qs + CC * LDK;                                // [C][LDA]
  float* Pm = Am + CC * LDA;                                // [C][LDA]
  float* rk = Pm + CC * LDA;                                // [C] row factors of k, q, and beta
  float* rq = rk + CC;
  float* bs = rq + CC;
  pdl_launch_dependents();
  pdl_wait();
  const int chunk = blockIdx.x, h = blockIdx.y, seg = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int n = seg_nrows[seg];
  if (chunk * CC >= n) return;
  const int seg0 = seg_row0[seg], r0 = chunk * CC, valid = min(CC, n - r0);
  const int kh = h / (L.heads / L.kv_heads), C = L.channels();
  const T* tail = conv_state + (size_t)seg_slot[seg] * (L.taps - 1) * C;
  float* rec = scratch + ((size_t)(seg0 / CC + seg + chunk) * L.heads + h) * cc_rec_floats(DKP);

  // convolved q and k of the head: a thread walks down its share of one channel's rows, eight loads ahead (rows past the segment's
  // end are read again from its last row and dropped)
  {
    constexpr int SHARES = CP_THREADS / (2 * DKP), ROWS = CC / SHARES, B = 8;
    static_assert(ROWS % B == 0, "batches");
    const int c2 = tid % (2 * DKP), t0 = tid / (2 * DKP) * ROWS, c = c2 % DKP;
    const bool is_k = c2 >= DKP;
    T* dst = (is_k ? Kr : Qr) + c;
    if (c < L.dim) {
      const int ch = (is_k ? L.kv_heads + kh : kh) * L.dim + c;
      const T* src = proj + (size_t)seg0 * ldp + L.q_off + ch;
      T raw[2][B];
      auto fetch = [&](T (&x)[B], int t) {
#pragma unroll
        for (int e = 0; e < B; ++e) x[e] = src[(size_t)min(r0 + t + e, n - 1) * ldp];
      };
      fetch(raw[0], t0);
      float w[NT], win[NT - 1];
      cd_load_taps(w, conv_w, ch, L.taps);
#pragma unroll
      for (int j = 0; j < NT - 1; ++j) {
        const int r = r0 + t0 + j - (NT - 1);
        win[j] = cd_input(proj, ldp, L.q_off, tail, C, L.taps, seg0, min(r, n - 1), ch);
      }
#pragma unroll
      for (int b = 0; b < ROWS / B; ++b) {
        if (b + 1 < ROWS / B) fetch(raw[(b + 1) & 1], t0 + (b + 1) * B);
#pragma unroll
        for (int e = 0; e < B; ++e) {
          const int t = t0 + b * B + e;
          const float v = cd_conv_step<T, NT>(w, win, Elem<T>::to(raw[b & 1][e]));
          dst[t * LDR] = Elem<T>::from(t < valid ? v : 0.f);
        }
      }
    } else {
      for (int t = t0; t < t0 + ROWS; ++t) dst[t * LDR] = Elem<T>::from(0.f);
    }
  }
  {
    const float expA = expf(A_log[h]);
    const int c = tid % DKP, cl = min(c, L.dim - 1);
    const float dtb = dt_bias[h * L.dim + cl];
    const float* src = decay + (size_t)(seg0 + r0) * ldd + h * L.dim + cl;
    constexpr int N = CC / GROUPS;
#pragma unroll
    for (int b = 0; b < N; b += 8) {
      float z[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) z[e] = src[(size_t)min(tid / DKP + (b + e) * GROUPS, valid - 1) * ldd];
#pragma unroll
      for (int e = 0; e < 8; ++e) {                         // rows past the segment's end leave the state as it is
        const int t = tid / DKP + (b + e) * GROUPS;
        lg[t * LDK + c] = t < valid && c < L.dim ? cd_log_decay(expA, z[e] + dtb) : 0.f;
      }
    }
  }
  if (tid < CC) bs[tid] = tid < valid ? cd_sigmoid(Elem<T>::to(proj[(size_t)(seg0 + r0 + tid) * ldp + L.b_off() + h])) : 0.f;
  for (int i = tid; i < 2 * CC * LDA; i += CP_THREADS) Am[i] = 0.f;                    // Am and Pm
  __syncthreads();
#pragma unroll
  for (int t = warp; t < CC; t += CP_THREADS / 32) {
    float sq = 0.f, sk = 0.f, qk = 0.f;
#pragma unroll
    for (int c = 2 * lane; c < DKP; c += 64) {
      const float2 q = Elem<T>::load2(Qr + t * LDR + c), k = Elem<T>::load2(Kr + t * LDR + c);
      sq = fmaf(q.x, q.x, fmaf(q.y, q.y, sq)); sk = fmaf(k.x, k.x, fmaf(k.y, k.y, sk)); qk = fmaf(q.x, k.x, fmaf(q.y, k.y, qk));
    }
    sq = warp_sum(sq); sk = warp_sum(sk); qk = warp_sum(qk);
    if (lane == 0) {
      const float fq = 1.f / (sqrtf(sq + CD_UNIT_EPS) * sqrtf((float)L.dim)), fk = 1.f / sqrtf(sk + CD_UNIT_EPS);
      rq[t] = fq; rk[t] = fk;
      Pm[t * LDA + t] = qk * fq * fk;
    }
  }
  __syncthreads();

  // what the scan multiplies with the state: K~ and Q~ down the rows (groups 0, 1: the halves of the chunk), k e^{G_C - G} up the rows
  // (groups 2, 3); more groups idle
  {
    const int c = tid % DKP, g = tid / DKP;
    float* gKt = rec;
    float* gQt = gKt + CC * DKP;
    float* gKh = gQt + CC * DKP;
    constexpr int HC = CC / 2;
    float acc = 0.f;
    if (g < 2) {
      if (g == 1)
#pragma unroll 8
        for (int t = 0; t < HC; ++t) acc += lg[t * LDK + c];
#pragma unroll 8
      for (int t = g * HC; t < (g + 1) * HC; ++t) {
        acc += lg[t * LDK + c];
        const float f = __expf(acc);
        gKt[t * DKP + c] = Elem<T>::to(Kr[t * LDR + c]) * rk[t] * f;
        gQt[t * DKP + c] = Elem<T>::to(Qr[t * LDR + c]) * rq[t] * f;
      }
      if (g == 1) rec[3 * CC * DKP + 2 * CC * CC + c] = __expf(acc);
    } else if (g < 4) {
      if (g == 2)
#pragma unroll 8
        for (int t = CC - 1; t >= HC; --t) acc += lg[t * LDK + c];
#pragma unroll 8
      for (int t = (g - 1) * HC - 1; t >= (g - 2) * HC; --t) {
        gKh[t * DKP + c] = Elem<T>::to(Kr[t * LDR + c]) * rk[t] * __expf(acc);
        acc += lg[t * LDK + c];
      }
    }
  }
  // A and P, level by level
  auto weigh = [&](auto level) {                            // runs of LV rows: even = lower half, odd = upper half
    constexpr int LV = decltype(level)::value;
    const int c = tid % DKP;
    for (int run = tid / DKP; run < CC / LV; run += GROUPS) {
      float acc = 0.f;
      if (run & 1) {
#pragma unroll(LV < 8 ? LV : 8)
        for (int j = 0; j < LV; ++j) {
          const int t = run * LV + j;
          acc += lg[t * LDK + c];
          const float f = __expf(acc);
          Ks[t * LDK + c] = Elem<T>::to(Kr[t * LDR + c]) * f;
          Qs[t * LDK + c] = Elem<T>::to(Qr[t * LDR + c]) * f;
        }
      } else {
#pragma unroll(LV < 8 ? LV : 8)
        for (int j = 0; j < LV; ++j) {
          const int t = (run + 1) * LV - 1 - j;
          Ks[t * LDK + c] = Elem<T>::to(Kr[t * LDR + c]) * __expf(acc);
          acc += lg[t * LDK + c];
        }
      }
    }
    __syncthreads();
    cc_level_pairs<DKP, LDK, LDA, LV>(Am, Pm, Ks, Qs, rk, rq, bs);
    __syncthreads();
  };
  weigh(std::integral_constant<int, 32>());
  weigh(std::integral_constant<int, 16>());
  weigh(std::integral_constant<int, 8>());
  weigh(std::integral_constant<int, 4>());
  weigh(std::integral_constant<int, 2>());
  weigh(std::integral_constant<int, 1>());
  // T = (I + A)^{-1} by blocks of 16: the diagonal blocks column by column, then block row b from the ones above it,
  // T[b][a] = -T[b][b] sum_{a <= m < b} A[b][m] T[m][a]
  float* Ti = Ks;                                           // [C][LDA]
  float* Xs = Qs;                                           // [16][48]
  for (int i = tid; i < CC * LDA; i += CP_THREADS) Ti[i] = 0.f;
  __syncthreads();
  if (tid < CC) {
    const int b0 = tid / 16 * 16, j = tid % 16;
    float x[16];
#pragma unroll
    for (int t = 0; t < 16; ++t) {
      float v = t == j ? 1.f : 0.f;
#pragma unroll
      for (int i = 0; i < t; ++i) v = fmaf(-Am[(b0 + t) * LDA + b0 + i], x[i], v);
      x[t] = v;
      Ti[(b0 + t) * LDA + b0 + j] = v;
    }
  }
  __syncthreads();
#pragma unroll 1
  for (int b0 = 16; b0 < CC; b0 += 16) {
    for (int o = tid; o < 16 * b0; o += CP_THREADS) {
      const int t = o / b0, j = o % b0;
      float v = 0.f;
      for (int m = j / 16 * 16; m < b0; m += 16)
#pragma unroll
        for (int i = 0; i < 16; ++i) v = fmaf(Am[(b0 + t) * LDA + m + i], Ti[(m + i) * LDA + j], v);
      Xs[t * 48 + j] = v;
    }
    __syncthreads();
    for (int o = tid; o < 16 * b0; o += CP_THREADS) {
      const int t = o / b0, j = o % b0;
      float v = 0.f;
#pragma unroll
      for (int i = 0; i < 16; ++i) v = fmaf(Ti[(b0 + t) * LDA + b0 + i], Xs[i * 48 + j], v);
      Ti[(b0 + t) * LDA + j] = -v;
    }
    __syncthreads();
  }
  // T' = T diag(beta) and P T', eight columns of a row per thread
  {
    const int t = tid / 8, j0 = tid % 8 * 8;
    float* gT = rec + 3 * CC * DKP + t * CC + j0;
    float m[8] = {};
    if (j0 <= t) {
#pragma unroll 4
      for (int i = j0; i <= t; ++i) {
        const float p = Pm[t * LDA + i];
        const float4 x = *reinterpret_cast<const float4*>(Ti + i * LDA + j0), y = *reinterpret_cast<const float4*>(Ti + i * LDA + j0 + 4);
        m[0] = fmaf(p, x.x, m[0]); m[1] = fmaf(p, x.y, m[1]); m[2] = fmaf(p, x.z, m[2]); m[3] = fmaf(p, x.w, m[3]);
        m[4] = fmaf(p, y.x, m[4]); m[5] = fmaf(p, y.y, m[5]); m[6] = fmaf(p, y.z, m[6]); m[7] = fmaf(p, y.w, m[7]);
      }
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      gT[e] = Ti[t * LDA + j0 + e] * bs[j0 + e];
      gT[CC * CC + e] = m[e] * bs[j0 + e];
    }
  }
}

// ---- scan --------------------------------------------------------------------------------------------------------------------
// grid (ceil(vdim / W), heads, segments), 8 W threads. A thread's tile: two rows of the chunk x 4 columns (shared-memory reads per FMA
// set the pace). Kt and Qt of the next chunk
// are fetched while the current one is past them, Kh, T', P T', eC likewise, and so are the raw inputs of v.
template <int DKP, int W>
struct ScanSmem {
  static constexpr int LDK = DKP + 4, LDT = CC + 4;
  static constexpr size_t BYTES = ((size_t)3 * CC * LDK + 2 * CC * LDT + DKP + DKP * W + 3 * CC * W) * 4;
};

template <typename T, int DKP, int W, int NT>
__global__ void __launch_bounds__(8 * W)
cd_chunk_scan_kernel(float* __restrict__ y, float* __restrict__ rec_state, const float* __restrict__ scratch, const T* __restrict__ proj,
                     long ldp, const float* __restrict__ conv_w, const T* __restrict__ conv_state, const int* __restrict__ seg_slot,
                     const int* __restrict__ seg_row0, const int* __restrict__ seg_nrows, CdLayer L) {
  using M = ScanSmem<DKP, W>;
  constexpr int NTH = 8 * W, LDK = M::LDK, LDT = M::LDT, CG = W / 4, RG = NTH / CG, R = CC / RG;       // rows rg, rg + RG of the chunk
  constexpr int R3 = DKP / RG;                                                              // state rows per thread
  static_assert(R == 2 && R3 >= 2, "tiles");
  extern __shared__ __align__(16) float cs_smem[];
  float* KQ = cs_smem;                                      // [2 C][LDK]: K~ rows, then Q~ rows
  float* Kh = KQ + 2 * CC * LDK;                            // [C][LDK]
  float* Ts = Kh + CC * LDK;                                // [C][LDT]
  float* Ps = Ts + CC * LDT;                                // [C][LDT]
  float* eC = Ps + CC * LDT;                                // [DKP]
  float* Ss = eC + DKP;                                     // [DKP][W] state slice
  float* Bs = Ss + DKP * W;                                 // [C][W] V - K~ S
  float* Ds = Bs + CC * W;                                  // [C][W]
  float* Vs = Ds + CC * W;                                  // [C][W]
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.y, seg = blockIdx.z, tid = threadIdx.x, col0 = blockIdx.x * W;
  const int n = seg_nrows[seg];
  if (n <= 0) return;
  const int seg0 = seg_row0[seg], slot = seg_slot[seg], C = L.channels();
  float* Sg = rec_state + ((size_t)slot * L.heads + h) * L.dim * L.vdim + col0;
  for (int i = tid; i < DKP * W; i += NTH) {
    const int k = i / W, c = i % W;
    Ss[i] = k < L.dim && col0 + c < L.vdim ? Sg[(size_t)k * L.vdim + c] : 0.f;
  }
  const size_t rec_stride = (size_t)L.heads * cc_rec_floats(DKP);
  const float* rec = scratch + ((size_t)(seg0 / CC + seg) * L.heads + h) * cc_rec_floats(DKP);
  auto load_kq = [&](const float* r) {
    for (int i = tid; i < 2 * CC * DKP / 4; i += NTH) cc_cp16(KQ + i / (DKP / 4) * LDK + i % (DKP / 4) * 4, r + i * 4);
    cc_commit();
  };
  auto load_rest = [&](const float* r) {
    r += 2 * CC * DKP;
    for (int i = tid; i < CC * DKP / 4; i += NTH) cc_cp16(Kh + i / (DKP / 4) * LDK + i % (DKP / 4) * 4, r + i * 4);
    r += CC * DKP;
    for (int i = tid; i < 2 * CC * CC / 4; i += NTH) cc_cp16(Ts + i / (CC / 4) * LDT + i % (CC / 4) * 4, r + i * 4);
    r += 2 * CC * CC;
    for (int i = tid; i < DKP / 4; i += NTH) cc_cp16(eC + i * 4, r + i * 4);
    cc_commit();
  };
  load_kq(rec);
  load_rest(rec);

  // this thread's share of v: one column, eight rows of every chunk and the NT - 1 inputs ahead of them
  constexpr int VR = CC * W / NTH;
  const int vc = tid % W, vt = tid / W * VR, vcol = min(col0 + vc, L.vdim - 1), vch = 2 * L.kv_heads * L.dim + h * L.vdim + vcol;
  const T* tail = conv_state + (size_t)slot * (L.taps - 1) * C;
  const T* vsrc = proj + (size_t)seg0 * ldp + L.q_off + vch;
  float w[NT];
  cd_load_taps(w, conv_w, vch, L.taps);
  T raw[VR + NT - 1];
  auto fetch = [&](int r) {                                 // rows r - (NT - 1) .. r + VR - 1 of the segment, held inside it
#pragma unroll
    for (int j = 0; j < VR + NT - 1; ++j) raw[j] = vsrc[(size_t)max(0, min(r + j - (NT - 1), n - 1)) * ldp];
  };
  fetch(vt);
  const int cg = tid % CG * 4, rg = tid / CG;
  const int nchunks = (n + CC - 1) / CC;
  for (int chn = 0; chn < nchunks; ++chn) {
    const int r0 = chn * CC, valid = min(CC, n - r0);
    {
      float win[NT - 1];
#pragma unroll
      for (int j = 0; j < NT - 1; ++j) {
        const int r = r0 + vt + j - (NT - 1);
        win[j] = r >= 0 ? Elem<T>::to(raw[j]) : cd_input(proj, ldp, L.q_off, tail, C, L.taps, seg0, r, vch);
      }
#pragma unroll
      for (int t = 0; t < VR; ++t) {
        const float v = cd_conv_step<T, NT>(w, win, Elem<T>::to(raw[NT - 1 + t]));
        Vs[(vt + t) * W + vc] = vt + t < valid && col0 + vc < L.vdim ? v : 0.f;
      }
      if (chn + 1 < nchunks) fetch(r0 + CC + vt);
    }
    cc_wait<1>();                                           // K~, Q~ have landed (Kh and the rest may still be on their way)
    __syncthreads();                                        // ... for everyone, V too, and the state slice is complete
    float u[R][4] = {}, o[R][4] = {};                       // this thread's rows of K~ S and of Q~ S
#pragma unroll 2
    for (int k = 0; k < DKP; k += 4) {
      float4 sv[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) sv[e] = *reinterpret_cast<const float4*>(Ss + (k + e) * W + cg);
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const float4 a = *reinterpret_cast<const float4*>(KQ + (rg + i * RG) * LDK + k);
        const float4 b = *reinterpret_cast<const float4*>(KQ + (CC + rg + i * RG) * LDK + k);
        const float ax[4] = {a.x, a.y, a.z, a.w}, bx[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float4 v = sv[e];
          u[i][0] = fmaf(ax[e], v.x, u[i][0]); u[i][1] = fmaf(ax[e], v.y, u[i][1]);
          u[i][2] = fmaf(ax[e], v.z, u[i][2]); u[i][3] = fmaf(ax[e], v.w, u[i][3]);
          o[i][0] = fmaf(bx[e], v.x, o[i][0]); o[i][1] = fmaf(bx[e], v.y, o[i][1]);
          o[i][2] = fmaf(bx[e], v.z, o[i][2]); o[i][3] = fmaf(bx[e], v.w, o[i][3]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const float4 v = *reinterpret_cast<const float4*>(Vs + (rg + i * RG) * W + cg);
      *reinterpret_cast<float4*>(Bs + (rg + i * RG) * W + cg) = make_float4(v.x - u[i][0], v.y - u[i][1], v.z - u[i][2], v.w - u[i][3]);
    }
    cc_wait<0>();                                           // Kh, T', P T', eC
    __syncthreads();                                        // ... and B; K~ and Q~ are free
    if (chn + 1 < nchunks) load_kq(rec + (size_t)(chn + 1) * rec_stride);
    // D = T' B, O = Q~ S + P T' B (both lower triangular, zeros above); past its own diagonal the first row is done
    float d[R][4] = {};
    auto triangle = [&](int k, auto first) {
      constexpr int I0 = decltype(first)::value;
      float4 sv[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) sv[e] = *reinterpret_cast<const float4*>(Bs + (k + e) * W + cg);
#pragma unroll
      for (int i = I0; i < R; ++i) {
        const float4 a = *reinterpret_cast<const float4*>(Ts + (rg + i * RG) * LDT + k);
        const float4 b = *reinterpret_cast<const float4*>(Ps + (rg + i * RG) * LDT + k);
        const float ax[4] = {a.x, a.y, a.z, a.w}, bx[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float4 v = sv[e];
          d[i][0] = fmaf(ax[e], v.x, d[i][0]); d[i][1] = fmaf(ax[e], v.y, d[i][1]);
          d[i][2] = fmaf(ax[e], v.z, d[i][2]); d[i][3] = fmaf(ax[e], v.w, d[i][3]);
          o[i][0] = fmaf(bx[e], v.x, o[i][0]); o[i][1] = fmaf(bx[e], v.y, o[i][1]);
          o[i][2] = fmaf(bx[e], v.z, o[i][2]); o[i][3] = fmaf(bx[e], v.w, o[i][3]);
        }
      }
    };
#pragma unroll 2
    for (int k = 0; k < RG; k += 4) triangle(k, std::integral_constant<int, 0>());
    const int last = RG + (rg | 7) + 1;                     // the same bound for all rows of a warp
#pragma unroll 2
    for (int k = RG; k < last; k += 4) triangle(k, std::integral_constant<int, 1>());
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int t = rg + i * RG;
      *reinterpret_cast<float4*>(Ds + t * W + cg) = make_float4(d[i][0], d[i][1], d[i][2], d[i][3]);
      if (t < valid) {
        float* dst = y + ((size_t)(seg0 + r0 + t) * L.heads + h) * L.vdim + col0 + cg;
        if (L.vdim % 4 == 0 && col0 + cg < L.vdim) {
          *reinterpret_cast<float4*>(dst) = make_float4(o[i][0], o[i][1], o[i][2], o[i][3]);
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (col0 + cg + e < L.vdim) dst[e] = o[i][e];
        }
      }
    }
    __syncthreads();
    // S = diag(eC) S + Kh^T D: this thread's R3 consecutive state rows
    {
      float s[R3][4];
#pragma unroll
      for (int i = 0; i < R3; ++i) {
        const int k = rg * R3 + i;
        const float4 a = *reinterpret_cast<const float4*>(Ss + k * W + cg);
        const float f = eC[k];
        s[i][0] = a.x * f; s[i][1] = a.y * f; s[i][2] = a.z * f; s[i][3] = a.w * f;
      }
#pragma unroll 8
      for (int t = 0; t < CC; ++t) {
        const float4 dd = *reinterpret_cast<const float4*>(Ds + t * W + cg);
        float kx[R3];
#pragma unroll
        for (int i = 0; i < R3; i += 2) {
          const float2 a = *reinterpret_cast<const float2*>(Kh + t * LDK + rg * R3 + i);
          kx[i] = a.x; kx[i + 1] = a.y;
        }
#pragma unroll
        for (int i = 0; i < R3; ++i) {
          s[i][0] = fmaf(kx[i], dd.x, s[i][0]); s[i][1] = fmaf(kx[i], dd.y, s[i][1]);
          s[i][2] = fmaf(kx[i], dd.z, s[i][2]); s[i][3] = fmaf(kx[i], dd.w, s[i][3]);
        }
      }
#pragma unroll
      for (int i = 0; i < R3; ++i)
        *reinterpret_cast<float4*>(Ss + (rg * R3 + i) * W + cg) = make_float4(s[i][0], s[i][1], s[i][2], s[i][3]);
    }
    __syncthreads();                                        // Kh, T', P T', eC and the work arrays are free
    if (chn + 1 < nchunks) load_rest(rec + (size_t)(chn + 1) * rec_stride);
  }
  for (int i = tid; i < DKP * W; i += NTH) {
    const int k = i / W, c = i % W;
    if (k < L.dim && col0 + c < L.vdim) Sg[(size_t)k * L.vdim + c] = Ss[i];
  }
}

template <typename T, int DKP, int W, int NT>
static int cd_chunk(float* y, float* rec, float* scratch, const void* tail, const void* proj, long ldp, const float* decay, long ldd,
                    const float* conv_w, const float* A_log, const float* dt_bias, const int* seg_slot, const int* seg_row0,
                    const int* seg_nrows, int nseg, int max_rows, CdLayer L, cudaStream_t s) {
  auto prep = cd_chunk_prep_kernel<T, DKP, NT>;
  auto scan = cd_chunk_scan_kernel<T, DKP, W, NT>;
  constexpr size_t psm = PrepSmem<T, DKP>::BYTES, ssm = ScanSmem<DKP, W>::BYTES;
  cudaError_t e = cudaFuncSetAttribute(prep, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)psm);
  if (e == cudaSuccess) e = cudaFuncSetAttribute(scan, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ssm);
  if (e == cudaSuccess)
    e = launch_pdl(prep, dim3((max_rows + CC - 1) / CC, L.heads, nseg), dim3(CP_THREADS), psm, s, scratch, (const T*)proj, ldp, decay, ldd,
                   conv_w, A_log, dt_bias, (const T*)tail, seg_slot, seg_row0, seg_nrows, L);
  if (e == cudaSuccess)
    e = launch_pdl(scan, dim3((L.vdim + W - 1) / W, L.heads, nseg), dim3(8 * W), ssm, s, y, rec, (const float*)scratch, (const T*)proj,
                   ldp, conv_w, (const T*)tail, seg_slot, seg_row0, seg_nrows, L);
  return (int)e;
}

template <typename T, int NT>
static int cd_chunk_any(float* y, float* rec, float* scratch, const void* tail, const void* proj, long ldp, const float* decay, long ldd,
                        const float* conv_w, const float* A_log, const float* dt_bias, const int* seg_slot, const int* seg_row0,
                        const int* seg_nrows, int nseg, int max_rows, int wide, CdLayer L, cudaStream_t s) {
#define FB_CC(DKP, W)                                                                                                                  \
  return cd_chunk<T, DKP, W, NT>(y, rec, scratch, tail, proj, ldp, decay, ldd, conv_w, A_log, dt_bias, seg_slot, seg_row0, seg_nrows, nseg, \
                             max_rows, L, s)
  if (L.dim <= 64) {
    if (wide) FB_CC(64, 32);
    FB_CC(64, 16);
  }
  if (wide) FB_CC(128, 32);
  FB_CC(128, 16);
#undef FB_CC
}

}  // namespace fb

using namespace fb;

extern "C" long fb_cd_chunk_scratch_bytes(int rows, int nseg, int heads, int dim) {
  return ((long)rows / CC + nseg + 1) * heads * cc_rec_floats(dim <= 64 ? 64 : 128) * 4l;
}

// Prompt segments; y [rows][heads][vdim] fp32 before the gated norm, the new state in place, the tail left as it is. -20: dim > 128.
extern "C" int fb_cd_chunk(float* y, float* rec, float* scratch, const void* tail, const void* proj, long ldp, const float* decay, long ldd,
                           const float* conv_w, const float* A_log, const float* dt_bias, const int* seg_slot, const int* seg_row0,
                           const int* seg_nrows, int nseg, int max_rows, int heads, int kv_heads, int dim, int vdim, int taps, int q_off,
                           int sm_count, int f32, cudaStream_t s) {
  if (nseg <= 0 || max_rows <= 0) return 0;
  if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || taps < 1 || taps > CD_TAPS || heads > 65535 || nseg > 65535 || !scratch) return -1;
  if (dim > 128) return -20;
  const CdLayer L{heads, kv_heads, dim, vdim, taps, q_off};
  const int wide = (long)((vdim + 31) / 32) * heads * nseg * 4 >= 3l * sm_count;       // 32-column slices when they fill the GPU
  auto go = [&](auto fn) {
    return fn(y, rec, scratch, tail, proj, ldp, decay, ldd, conv_w, A_log, dt_bias, seg_slot, seg_row0, seg_nrows, nseg, max_rows, wide, L, s);
  };
  if (f32) return taps <= 4 ? go(cd_chunk_any<float, 4>) : go(cd_chunk_any<float, CD_TAPS>);
  return taps <= 4 ? go(cd_chunk_any<__nv_bfloat16, 4>) : go(cd_chunk_any<__nv_bfloat16, CD_TAPS>);
}
