// Channel-delta layers, prompt segments: the recurrence of cdelta.cuh over chunks of C = 64 rows. With G_t = sum_{i <= t} log g_i (a
// vector over the key channels, inside the chunk) and S_0 the state the chunk starts from:
//   (I + A) D = diag(beta) (V - K~ S_0),   K~_t = k_t e^{G_t},   A[t][i] = beta_t sum_c k_t[c] k_i[c] e^{G_t[c] - G_i[c]}   (i < t)
//   O = Q~ S_0 + P D,                      Q~_t = q_t e^{G_t},   P[t][i] = sum_c q_t[c] k_i[c] e^{G_t[c] - G_i[c]}          (i <= t)
//   S_C = diag(e^{G_C}) S_0 + sum_i k_i e^{G_C - G_i} d_i^T
// prep (parallel over chunks x heads) forms K~, Q~, k e^{G_C - G}, T' = (I + A)^{-1} diag(beta), P; scan (serial over the chunks of a
// segment, parallel over heads x slices of state columns) runs the products with S.
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

namespace fb {

constexpr int CC = 64;                  // rows per chunk
constexpr int CP_THREADS = 512, CS_THREADS = 256;

__device__ __forceinline__ void cc_cp16(void* smem, const void* gmem) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem)), "l"(gmem) : "memory");
}
__device__ __forceinline__ void cc_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cc_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// One (chunk, head) of the scratch: floats Kt [C][DKP] | Qt [C][DKP] | Kh [C][DKP] | T' [C][C] | P [C][C] | eC [DKP]
__host__ __device__ constexpr long cc_rec_floats(int dkp) { return 3l * CC * dkp + 2l * CC * CC + dkp; }

// ---- prep --------------------------------------------------------------------------------------------------------------------
template <typename T, int DKP>
struct PrepSmem {
  static constexpr int LDR = DKP + 16 / sizeof(T);          // raw rows
  static constexpr int LDK = DKP + 4, LDA = CC + 1;
  static constexpr size_t BYTES = (size_t)2 * CC * LDR * sizeof(T) + ((size_t)3 * CC * LDK + 2 * CC * LDA + 3 * CC) * 4;
};

template <typename T, int DKP>
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

  // convolved q and k of the head: a thread walks down its share of one channel's rows
  {
    constexpr int SHARES = CP_THREADS / (2 * DKP), ROWS = CC / SHARES;
    const int c2 = tid % (2 * DKP), share = tid / (2 * DKP), c = c2 % DKP;
    const bool is_k = c2 >= DKP;
    T* dst = (is_k ? Kr : Qr) + c;
    if (c < L.dim) {
      const int ch = (is_k ? L.kv_heads + kh : kh) * L.dim + c;
      float w[CD_TAPS], win[CD_TAPS - 1];
      cd_load_taps(w, conv_w, ch, L.taps);
      const int t0 = share * ROWS;
#pragma unroll
      for (int j = 0; j < CD_TAPS - 1; ++j) {
        const int r = r0 + t0 + j - (CD_TAPS - 1);
        win[j] = r < n ? cd_input(proj, ldp, L.q_off, tail, C, L.taps, seg0, r, ch) : 0.f;
      }
#pragma unroll 8
      for (int t = t0; t < t0 + ROWS; ++t)
        dst[t * LDR] = Elem<T>::from(t < valid ? cd_conv_step<T>(w, win, Elem<T>::to(proj[(size_t)(seg0 + r0 + t) * ldp + L.q_off + ch])) : 0.f);
    } else {
      for (int t = share * ROWS; t < (share + 1) * ROWS; ++t) dst[t * LDR] = Elem<T>::from(0.f);
    }
  }
  {
    const float expA = expf(A_log[h]);
    const int c = tid % DKP;
    const float dtb = c < L.dim ? dt_bias[h * L.dim + c] : 0.f;
#pragma unroll 4
    for (int t = tid / DKP; t < CC; t += GROUPS)            // rows past the segment's end leave the state as it is
      lg[t * LDK + c] = t < valid && c < L.dim ? cd_log_decay(expA, decay[(size_t)(seg0 + r0 + t) * ldd + h * L.dim + c] + dtb) : 0.f;
  }
  if (tid < CC) bs[tid] = tid < valid ? cd_sigmoid(Elem<T>::to(proj[(size_t)(seg0 + r0 + tid) * ldp + L.b_off() + h])) : 0.f;
  for (int i = tid; i < CC * LDA; i += CP_THREADS) Pm[i] = 0.f;
  __syncthreads();
  for (int t = warp; t < CC; t += CP_THREADS / 32) {
    float sq = 0.f, sk = 0.f, qk = 0.f;
    for (int c = lane; c < DKP; c += 32) {
      const float q = Elem<T>::to(Qr[t * LDR + c]), k = Elem<T>::to(Kr[t * LDR + c]);
      sq = fmaf(q, q, sq); sk = fmaf(k, k, sk); qk = fmaf(q, k, qk);
    }
    sq = warp_sum(sq); sk = warp_sum(sk); qk = warp_sum(qk);
    if (lane == 0) {
      const float fq = 1.f / (sqrtf(sq + CD_UNIT_EPS) * sqrtf((float)L.dim)), fk = 1.f / sqrtf(sk + CD_UNIT_EPS);
      rq[t] = fq; rk[t] = fk;
      Pm[t * LDA + t] = qk * fq * fk;
    }
  }
  __syncthreads();

  // what the scan multiplies with the state
  {
    const int c = tid % DKP, g = tid / DKP;                 // group 0: K~, Q~ down the rows; group 1: k e^{G_C - G} up the rows
    float* gKt = rec;
    float* gQt = gKt + CC * DKP;
    float* gKh = gQt + CC * DKP;
    if (g == 0) {
      float acc = 0.f;
#pragma unroll 4
      for (int t = 0; t < CC; ++t) {
        acc += lg[t * LDK + c];
        const float f = __expf(acc);
        gKt[t * DKP + c] = Elem<T>::to(Kr[t * LDR + c]) * rk[t] * f;
        gQt[t * DKP + c] = Elem<T>::to(Qr[t * LDR + c]) * rq[t] * f;
      }
      rec[3 * CC * DKP + 2 * CC * CC + c] = __expf(acc);
    } else if (g == 1) {
      float acc = 0.f;
#pragma unroll 4
      for (int t = CC - 1; t >= 0; --t) {
        gKh[t * DKP + c] = Elem<T>::to(Kr[t * LDR + c]) * rk[t] * __expf(acc);
        acc += lg[t * LDK + c];
      }
    }
  }
  // A and P, level by level
#pragma unroll 1
  for (int lv = CC / 2; lv >= 1; lv >>= 1) {
    {
      const int c = tid % DKP;
      for (int run = tid / DKP; run < CC / lv; run += GROUPS) {        // runs of lv rows: even = lower half, odd = upper half
        float acc = 0.f;
        if (run & 1) {
          for (int t = run * lv; t < (run + 1) * lv; ++t) {
            acc += lg[t * LDK + c];
            const float f = __expf(acc);
            Ks[t * LDK + c] = Elem<T>::to(Kr[t * LDR + c]) * f;
            Qs[t * LDK + c] = Elem<T>::to(Qr[t * LDR + c]) * f;
          }
        } else {
          for (int t = (run + 1) * lv - 1; t >= run * lv; --t) {
            Ks[t * LDK + c] = Elem<T>::to(Kr[t * LDR + c]) * __expf(acc);
            acc += lg[t * LDK + c];
          }
        }
      }
    }
    __syncthreads();
    const int pairs = CC / 2 * lv;
    const int lanes = pairs >= CP_THREADS ? 1 : CP_THREADS / pairs;    // threads that share a pair's channels
    const int sub = tid % lanes;
    for (int p = tid / lanes; p < pairs; p += CP_THREADS / lanes) {
      const int blk = p / (lv * lv), in = p % (lv * lv);
      const int t = blk * 2 * lv + lv + in / lv, i = blk * 2 * lv + in % lv;
      const float4* kt = reinterpret_cast<const float4*>(Ks + t * LDK);
      const float4* qt = reinterpret_cast<const float4*>(Qs + t * LDK);
      const float4* ki = reinterpret_cast<const float4*>(Ks + i * LDK);
      float a = 0.f, b = 0.f;
#pragma unroll 4
      for (int c = sub; c < DKP / 4; c += lanes) {
        const float4 x = kt[c], y = qt[c], z = ki[c];
        a = fmaf(x.x, z.x, fmaf(x.y, z.y, fmaf(x.z, z.z, fmaf(x.w, z.w, a))));
        b = fmaf(y.x, z.x, fmaf(y.y, z.y, fmaf(y.z, z.z, fmaf(y.w, z.w, b))));
      }
      for (int o = lanes / 2; o > 0; o >>= 1) {
        a += __shfl_xor_sync(0xffffffffu, a, o);
        b += __shfl_xor_sync(0xffffffffu, b, o);
      }
      if (sub == 0) {
        Am[t * LDA + i] = bs[t] * rk[t] * rk[i] * a;
        Pm[t * LDA + i] = rq[t] * rk[i] * b;
      }
    }
    __syncthreads();
  }
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
      for (int i = j / 16 * 16; i < b0; ++i) v = fmaf(Am[(b0 + t) * LDA + i], Ti[i * LDA + j], v);
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
  float* gT = rec + 3 * CC * DKP;
  float* gP = gT + CC * CC;
  for (int i = tid; i < CC * CC; i += CP_THREADS) {
    const int t = i / CC, j = i % CC;
    gT[i] = Ti[t * LDA + j] * bs[j];
    gP[i] = Pm[t * LDA + j];
  }
}

// ---- scan --------------------------------------------------------------------------------------------------------------------
// grid (ceil(vdim / W), heads, segments). A thread's tile: rows of one row group x 4 columns. Kt and Qt of the next chunk are fetched
// while the current one is past them, Kh, T', P, eC likewise.
template <int DKP, int W>
struct ScanSmem {
  static constexpr int LDK = DKP + 4, LDT = CC + 4;
  static constexpr size_t BYTES = ((size_t)3 * CC * LDK + 2 * CC * LDT + DKP + DKP * W + 3 * CC * W) * 4;
};

template <typename T, int DKP, int W>
__global__ void __launch_bounds__(CS_THREADS)
cd_chunk_scan_kernel(float* __restrict__ y, float* __restrict__ rec_state, const float* __restrict__ scratch, const T* __restrict__ proj,
                     long ldp, const float* __restrict__ conv_w, const T* __restrict__ conv_state, const int* __restrict__ seg_slot,
                     const int* __restrict__ seg_row0, const int* __restrict__ seg_nrows, CdLayer L) {
  using M = ScanSmem<DKP, W>;
  constexpr int LDK = M::LDK, LDT = M::LDT, CG = W / 4, RG = CS_THREADS / CG;
  constexpr int R1 = 2 * CC / RG, R2 = CC / RG, R3 = DKP / RG;        // rows per thread: [K~; Q~] S, T' B and P D, the new state
  static_assert(R2 >= 1 && R3 >= 1, "tiles");
  extern __shared__ __align__(16) float cs_smem[];
  float* KQ = cs_smem;                                      // [2 C][LDK]: K~ rows, then Q~ rows
  float* Kh = KQ + 2 * CC * LDK;                            // [C][LDK]
  float* Ts = Kh + CC * LDK;                                // [C][LDT]
  float* Ps = Ts + CC * LDT;                                // [C][LDT]
  float* eC = Ps + CC * LDT;                                // [DKP]
  float* Ss = eC + DKP;                                     // [DKP][W] state slice
  float* Bs = Ss + DKP * W;                                 // [C][W] V - K~ S
  float* Rs = Bs + CC * W;                                  // [C][W] Q~ S
  float* Ds = Rs + CC * W;                                  // [C][W]
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.y, seg = blockIdx.z, tid = threadIdx.x, col0 = blockIdx.x * W;
  const int n = seg_nrows[seg];
  if (n <= 0) return;
  const int seg0 = seg_row0[seg], slot = seg_slot[seg], C = L.channels();
  float* Sg = rec_state + ((size_t)slot * L.heads + h) * L.dim * L.vdim + col0;
  for (int i = tid; i < DKP * W; i += CS_THREADS) {
    const int k = i / W, c = i % W;
    Ss[i] = k < L.dim && col0 + c < L.vdim ? Sg[(size_t)k * L.vdim + c] : 0.f;
  }
  const size_t rec_stride = (size_t)L.heads * cc_rec_floats(DKP);
  const float* rec = scratch + ((size_t)(seg0 / CC + seg) * L.heads + h) * cc_rec_floats(DKP);
  auto load_kq = [&](const float* r) {
    for (int i = tid; i < 2 * CC * DKP / 4; i += CS_THREADS) cc_cp16(KQ + i / (DKP / 4) * LDK + i % (DKP / 4) * 4, r + i * 4);
    cc_commit();
  };
  auto load_rest = [&](const float* r) {
    r += 2 * CC * DKP;
    for (int i = tid; i < CC * DKP / 4; i += CS_THREADS) cc_cp16(Kh + i / (DKP / 4) * LDK + i % (DKP / 4) * 4, r + i * 4);
    r += CC * DKP;
    for (int i = tid; i < 2 * CC * CC / 4; i += CS_THREADS) cc_cp16(Ts + i / (CC / 4) * LDT + i % (CC / 4) * 4, r + i * 4);
    r += 2 * CC * CC;
    for (int i = tid; i < DKP / 4; i += CS_THREADS) cc_cp16(eC + i * 4, r + i * 4);
    cc_commit();
  };
  load_kq(rec);
  load_rest(rec);

  // this thread's share of v: one column, VR rows of every chunk
  constexpr int VR = CC * W / CS_THREADS;
  const int vc = tid % W, vt = tid / W * VR, vch = 2 * L.kv_heads * L.dim + h * L.vdim + col0 + vc;
  const bool v_on = col0 + vc < L.vdim;
  const T* tail = conv_state + (size_t)slot * (L.taps - 1) * C;
  float w[CD_TAPS];
  if (v_on) cd_load_taps(w, conv_w, vch, L.taps);
  const int cg = tid % CG * 4, rg = tid / CG;
  const int nchunks = (n + CC - 1) / CC;
  for (int chn = 0; chn < nchunks; ++chn) {
    const int r0 = chn * CC, valid = min(CC, n - r0);
    float vv[VR];
    {
      float win[CD_TAPS - 1];
      if (v_on)
#pragma unroll
        for (int j = 0; j < CD_TAPS - 1; ++j) {
          const int r = r0 + vt + j - (CD_TAPS - 1);
          win[j] = r < n ? cd_input(proj, ldp, L.q_off, tail, C, L.taps, seg0, r, vch) : 0.f;
        }
#pragma unroll
      for (int t = 0; t < VR; ++t)
        vv[t] = v_on && vt + t < valid ? cd_conv_step<T>(w, win, Elem<T>::to(proj[(size_t)(seg0 + r0 + vt + t) * ldp + L.q_off + vch])) : 0.f;
    }
    cc_wait<1>();                                           // K~, Q~ have landed (Kh and the rest may still be on their way)
    __syncthreads();                                        // ... for everyone, and the state slice is complete
#pragma unroll
    for (int t = 0; t < VR; ++t) Bs[(vt + t) * W + vc] = vv[t];
    float acc[R1][4] = {};
#pragma unroll 2
    for (int k = 0; k < DKP; k += 4) {
      float4 s4[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) s4[e] = *reinterpret_cast<const float4*>(Ss + (k + e) * W + cg);
#pragma unroll
      for (int i = 0; i < R1; ++i) {
        const float4 a = *reinterpret_cast<const float4*>(KQ + (rg + i * RG) * LDK + k);
        const float ax[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          acc[i][0] = fmaf(ax[e], s4[e].x, acc[i][0]); acc[i][1] = fmaf(ax[e], s4[e].y, acc[i][1]);
          acc[i][2] = fmaf(ax[e], s4[e].z, acc[i][2]); acc[i][3] = fmaf(ax[e], s4[e].w, acc[i][3]);
        }
      }
    }
    __syncthreads();                                        // V is in place, K~ and Q~ are free
    if (chn + 1 < nchunks) load_kq(rec + (size_t)(chn + 1) * rec_stride);
    else cc_commit();
#pragma unroll
    for (int i = 0; i < R1; ++i) {
      const int row = rg + i * RG;
      if (row < CC) {
        float4* b = reinterpret_cast<float4*>(Bs + row * W + cg);
        const float4 v = *b;
        *b = make_float4(v.x - acc[i][0], v.y - acc[i][1], v.z - acc[i][2], v.w - acc[i][3]);
      } else {
        *reinterpret_cast<float4*>(Rs + (row - CC) * W + cg) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
      }
    }
    cc_wait<1>();                                           // Kh, T', P, eC
    __syncthreads();
    // D = T' B (lower triangular)
#pragma unroll
    for (int i = 0; i < R2; ++i) {
      const int t = rg + i * RG;
      float d[4] = {};
      for (int k = 0; k <= t; k += 4) {
        const float4 a = *reinterpret_cast<const float4*>(Ts + t * LDT + k);
        const float ax[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float4 b = *reinterpret_cast<const float4*>(Bs + (k + e) * W + cg);
          d[0] = fmaf(ax[e], b.x, d[0]); d[1] = fmaf(ax[e], b.y, d[1]); d[2] = fmaf(ax[e], b.z, d[2]); d[3] = fmaf(ax[e], b.w, d[3]);
        }
      }
      *reinterpret_cast<float4*>(Ds + t * W + cg) = make_float4(d[0], d[1], d[2], d[3]);
    }
    __syncthreads();
    // O = Q~ S + P D
#pragma unroll
    for (int i = 0; i < R2; ++i) {
      const int t = rg + i * RG;
      const float4 r = *reinterpret_cast<const float4*>(Rs + t * W + cg);
      float o[4] = {r.x, r.y, r.z, r.w};
      for (int k = 0; k <= t; k += 4) {
        const float4 a = *reinterpret_cast<const float4*>(Ps + t * LDT + k);
        const float ax[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float4 b = *reinterpret_cast<const float4*>(Ds + (k + e) * W + cg);
          o[0] = fmaf(ax[e], b.x, o[0]); o[1] = fmaf(ax[e], b.y, o[1]); o[2] = fmaf(ax[e], b.z, o[2]); o[3] = fmaf(ax[e], b.w, o[3]);
        }
      }
      if (t < valid) {
        float* dst = y + ((size_t)(seg0 + r0 + t) * L.heads + h) * L.vdim + col0 + cg;
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (col0 + cg + e < L.vdim) dst[e] = o[e];
      }
    }
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
#pragma unroll 4
      for (int t = 0; t < CC; ++t) {
        const float4 d = *reinterpret_cast<const float4*>(Ds + t * W + cg);
        float kx[R3];
        if constexpr (R3 % 4 == 0) {
#pragma unroll
          for (int i = 0; i < R3; i += 4) {
            const float4 a = *reinterpret_cast<const float4*>(Kh + t * LDK + rg * R3 + i);
            kx[i] = a.x; kx[i + 1] = a.y; kx[i + 2] = a.z; kx[i + 3] = a.w;
          }
        } else {
#pragma unroll
          for (int i = 0; i < R3; ++i) kx[i] = Kh[t * LDK + rg * R3 + i];
        }
#pragma unroll
        for (int i = 0; i < R3; ++i) {
          s[i][0] = fmaf(kx[i], d.x, s[i][0]); s[i][1] = fmaf(kx[i], d.y, s[i][1]);
          s[i][2] = fmaf(kx[i], d.z, s[i][2]); s[i][3] = fmaf(kx[i], d.w, s[i][3]);
        }
      }
#pragma unroll
      for (int i = 0; i < R3; ++i)
        *reinterpret_cast<float4*>(Ss + (rg * R3 + i) * W + cg) = make_float4(s[i][0], s[i][1], s[i][2], s[i][3]);
    }
    __syncthreads();                                        // Kh, T', P, eC and the work arrays are free
    if (chn + 1 < nchunks) load_rest(rec + (size_t)(chn + 1) * rec_stride);
    else cc_commit();
  }
  cc_wait<0>();
  for (int i = tid; i < DKP * W; i += CS_THREADS) {
    const int k = i / W, c = i % W;
    if (k < L.dim && col0 + c < L.vdim) Sg[(size_t)k * L.vdim + c] = Ss[i];
  }
}

template <typename T, int DKP, int W>
static int cd_chunk(float* y, float* rec, float* scratch, const void* tail, const void* proj, long ldp, const float* decay, long ldd,
                    const float* conv_w, const float* A_log, const float* dt_bias, const int* seg_slot, const int* seg_row0,
                    const int* seg_nrows, int nseg, int max_rows, CdLayer L, cudaStream_t s) {
  auto prep = cd_chunk_prep_kernel<T, DKP>;
  auto scan = cd_chunk_scan_kernel<T, DKP, W>;
  constexpr size_t psm = PrepSmem<T, DKP>::BYTES, ssm = ScanSmem<DKP, W>::BYTES;
  cudaError_t e = cudaFuncSetAttribute(prep, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)psm);
  if (e == cudaSuccess) e = cudaFuncSetAttribute(scan, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ssm);
  if (e == cudaSuccess)
    e = launch_pdl(prep, dim3((max_rows + CC - 1) / CC, L.heads, nseg), dim3(CP_THREADS), psm, s, scratch, (const T*)proj, ldp, decay, ldd,
                   conv_w, A_log, dt_bias, (const T*)tail, seg_slot, seg_row0, seg_nrows, L);
  if (e == cudaSuccess)
    e = launch_pdl(scan, dim3((L.vdim + W - 1) / W, L.heads, nseg), dim3(CS_THREADS), ssm, s, y, rec, (const float*)scratch, (const T*)proj,
                   ldp, conv_w, (const T*)tail, seg_slot, seg_row0, seg_nrows, L);
  return (int)e;
}

template <typename T>
static int cd_chunk_any(float* y, float* rec, float* scratch, const void* tail, const void* proj, long ldp, const float* decay, long ldd,
                        const float* conv_w, const float* A_log, const float* dt_bias, const int* seg_slot, const int* seg_row0,
                        const int* seg_nrows, int nseg, int max_rows, int wide, CdLayer L, cudaStream_t s) {
#define FB_CC(DKP, W)                                                                                                                  \
  return cd_chunk<T, DKP, W>(y, rec, scratch, tail, proj, ldp, decay, ldd, conv_w, A_log, dt_bias, seg_slot, seg_row0, seg_nrows, nseg, \
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
  return f32 ? cd_chunk_any<float>(y, rec, scratch, tail, proj, ldp, decay, ldd, conv_w, A_log, dt_bias, seg_slot, seg_row0, seg_nrows, nseg,
                                   max_rows, wide, L, s)
             : cd_chunk_any<__nv_bfloat16>(y, rec, scratch, tail, proj, ldp, decay, ldd, conv_w, A_log, dt_bias, seg_slot, seg_row0,
                                           seg_nrows, nseg, max_rows, wide, L, s);
}
