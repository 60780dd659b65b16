// Channel-delta layers, few rows (see cdelta.cuh for the recurrence):
//   cd_lowrank   both low-rank up-projections of a few rows in one launch, straight from the fused projection
//   cd_step      convolutions, unit norms, decays, recurrence and gated head norm of a segment in one launch (dim, vdim <= 128)
//   cd_conv, cd_rec   the same split up, for any sizes: convolutions into a buffer, then the recurrence by slices of 32 state columns
//   cd_tail      the last taps - 1 inputs of every channel of a segment into its slot
// State: fp32 [slot][head][dim][vdim]; tail: [slot][taps - 1][channels] in the projection's type. Prompt segments: cdelta_chunk.cu.
#include "api_ext.h"
#include "cdelta.cuh"

namespace fb {

// ---- low-rank up-projections -------------------------------------------------------------------------------------------------
// out[row] = [W_a a1 | W_g g1], fp32. Eight lanes per output, four outputs per warp, rows in tiles of 8.
template <typename T>
__global__ void __launch_bounds__(256) cd_lowrank_kernel(float* __restrict__ out, const T* __restrict__ proj, long ldp,
                                                         const T* __restrict__ wa, int na, int ra, const T* __restrict__ wg, int ng,
                                                         int rg, int rows) {
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, sub = lane & 7;
  const int n = (blockIdx.x * 8 + warp) * 4 + (lane >> 3);
  const bool live = n < na + ng, is_a = n < na;
  const int R = is_a ? ra : rg;
  const T* w = is_a ? wa + (size_t)n * ra : wg + (size_t)(live ? n - na : 0) * rg;
  pdl_wait();
  const T* x = proj + (is_a ? 0 : ra);
  for (int m0 = 0; m0 < rows; m0 += 8) {
    float acc[8] = {};
    if (live)
      for (int k = sub * 4; k < R; k += 32) {
        const float4 a = Elem<T>::load4(w + k);
#pragma unroll
        for (int m = 0; m < 8; ++m) {
          if (m0 + m >= rows) break;
          const float4 b = Elem<T>::load4(x + (size_t)(m0 + m) * ldp + k);
          acc[m] = fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, fmaf(a.w, b.w, acc[m]))));
        }
      }
#pragma unroll
    for (int m = 0; m < 8; ++m) {
      if (m0 + m >= rows) break;
#pragma unroll
      for (int o = 4; o > 0; o >>= 1) acc[m] += __shfl_xor_sync(0xffffffffu, acc[m], o);
      if (live && sub == 0) out[(size_t)(m0 + m) * (na + ng) + n] = acc[m];
    }
  }
}

// ---- fused step ----------------------------------------------------------------------------------------------------------------
// grid (heads, segments), 512 threads. Roles of a row's inputs: DKP threads convolve q channels, DKP k channels, DVP v channels, DKP
// form the decays. State: thread (col = tid % DVP, part = tid / DVP) holds DKP / PARTS rows of column col across the segment.
constexpr int CD_THREADS = 512;

template <typename T, int DKP, int DVP, int NT>
__global__ void __launch_bounds__(CD_THREADS)
cd_step_kernel(T* __restrict__ out, int ko, float* __restrict__ rec_state, T* __restrict__ conv_state, const T* __restrict__ proj, long ldp,
               const float* __restrict__ decay, long ldd, const float* __restrict__ gate, long ldg, const float* __restrict__ conv_w,
               const float* __restrict__ A_log, const float* __restrict__ dt_bias, const float* __restrict__ norm_w,
               const int* __restrict__ seg_slot, const int* __restrict__ seg_row0, const int* __restrict__ seg_nrows, CdLayer L, float eps,
               int commit) {
  constexpr int PARTS = CD_THREADS / DVP, RP = DKP / PARTS;
  static_assert(3 * DKP + DVP <= CD_THREADS, "roles");
  __shared__ __align__(16) float qs[DKP], ks[DKP], gs[DKP], vs[DVP];
  __shared__ float red1[PARTS][DVP], red2[PARTS][DVP];
  __shared__ float ssq[2][DKP / 32], ssn[DVP / 32];
  pdl_launch_dependents();
  const int h = blockIdx.x, seg = blockIdx.y, tid = threadIdx.x, col = tid % DVP, part = tid / DVP;
  const int kh = h / (L.heads / L.kv_heads), C = L.channels();
  // role of this thread: 0 q, 1 k, 2 v, 3 decay; idx: its channel inside the head
  const int role = tid < DKP ? 0 : tid < 2 * DKP ? 1 : tid < 2 * DKP + DVP ? 2 : tid < 3 * DKP + DVP ? 3 : 4;
  const int idx = role == 0 ? tid : role == 1 ? tid - DKP : role == 2 ? tid - 2 * DKP : tid - 2 * DKP - DVP;
  const bool live = role < 4 && idx < (role == 2 ? L.vdim : L.dim);
  const int ch = role == 0 ? kh * L.dim + idx : role == 1 ? (L.kv_heads + kh) * L.dim + idx : 2 * L.kv_heads * L.dim + h * L.vdim + idx;
  float w[NT], win[NT - 1], dtb = 0.f, expA = 0.f;
  if (live && role < 3) cd_load_taps(w, conv_w, ch, L.taps);
  if (live && role == 3) { dtb = dt_bias[h * L.dim + idx]; expA = expf(A_log[h]); }
  const float nw = col < L.vdim ? norm_w[col] : 0.f;
  pdl_wait();
  const int n = seg_nrows[seg];
  if (n <= 0) return;
  const int row0 = seg_row0[seg], slot = seg_slot[seg];
  T* tail = conv_state + (size_t)slot * (L.taps - 1) * C;
  if (live && role < 3)
#pragma unroll
    for (int j = 0; j < NT - 1; ++j)
      win[j] = cd_input(proj, ldp, L.q_off, tail, C, L.taps, row0, j - (NT - 1), ch);
  float* Sg = rec_state + ((size_t)slot * L.heads + h) * L.dim * L.vdim;
  float S[RP];
#pragma unroll
  for (int i = 0; i < RP; ++i) {
    const int r = part * RP + i;
    S[i] = r < L.dim && col < L.vdim ? Sg[(size_t)r * L.vdim + col] : 0.f;
  }
  const float qscale = 1.f / sqrtf((float)L.dim);

  struct RowIn { float x, b, z; };                          // fetched one row ahead
  auto fetch = [&](int r) {
    RowIn in = {0.f, 0.f, 0.f};
    const size_t row = row0 + r;
    if (live) in.x = role == 3 ? decay[row * ldd + h * L.dim + idx] : Elem<T>::to(proj[row * ldp + L.q_off + ch]);
    in.b = Elem<T>::to(proj[row * ldp + L.b_off() + h]);
    if (part == 0 && col < L.vdim) in.z = gate[row * ldg + h * L.vdim + col];
    return in;
  };
  RowIn nxt = fetch(0);
  for (int r = 0; r < n; ++r) {
    const RowIn cur = nxt;
    if (r + 1 < n) nxt = fetch(r + 1);
    if (role < 2) {
      const float cv = live ? cd_conv_step<T, NT>(w, win, cur.x) : 0.f;
      (role == 0 ? qs : ks)[idx] = cv;
      const float sq = warp_sum(cv * cv);
      if ((tid & 31) == 0) ssq[role][idx >> 5] = sq;
    } else if (role == 2) {
      vs[idx] = live ? cd_conv_step<T, NT>(w, win, cur.x) : 0.f;
    } else if (role == 3) {
      gs[idx] = live ? expf(cd_log_decay(expA, cur.x + dtb)) : 0.f;
    }
    __syncthreads();
    float sq = 0.f, sk = 0.f;
#pragma unroll
    for (int i = 0; i < DKP / 32; ++i) { sq += ssq[0][i]; sk += ssq[1][i]; }
    const float rq = qscale / sqrtf(sq + CD_UNIT_EPS), rk = 1.f / sqrtf(sk + CD_UNIT_EPS);
    const float beta = cd_sigmoid(cur.b);
    const float4* k4 = reinterpret_cast<const float4*>(ks + part * RP);
    const float4* q4 = reinterpret_cast<const float4*>(qs + part * RP);
    const float4* g4 = reinterpret_cast<const float4*>(gs + part * RP);
    float p = 0.f;
#pragma unroll
    for (int i = 0; i < RP / 4; ++i) {
      const float4 kk = k4[i], gg = g4[i];
      S[4 * i] *= gg.x; S[4 * i + 1] *= gg.y; S[4 * i + 2] *= gg.z; S[4 * i + 3] *= gg.w;
      p = fmaf(S[4 * i], kk.x, p); p = fmaf(S[4 * i + 1], kk.y, p); p = fmaf(S[4 * i + 2], kk.z, p); p = fmaf(S[4 * i + 3], kk.w, p);
    }
    red1[part][col] = p;
    __syncthreads();
    float kv = 0.f;
#pragma unroll
    for (int i = 0; i < PARTS; ++i) kv += red1[i][col];
    const float u = (vs[col] - kv * rk) * beta * rk;
    float yp = 0.f;
#pragma unroll
    for (int i = 0; i < RP / 4; ++i) {
      const float4 kk = k4[i], qq = q4[i];
      const float kx[4] = {kk.x, kk.y, kk.z, kk.w}, qx[4] = {qq.x, qq.y, qq.z, qq.w};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        S[4 * i + e] = fmaf(kx[e], u, S[4 * i + e]);
        yp = fmaf(S[4 * i + e], qx[e], yp);
      }
    }
    red2[part][col] = yp;
    __syncthreads();
    float yy = 0.f;
    if (part == 0) {
#pragma unroll
      for (int i = 0; i < PARTS; ++i) yy += red2[i][col];
      yy *= rq;
      const float s2 = warp_sum(yy * yy);                   // columns past vdim hold zeros
      if ((tid & 31) == 0) ssn[tid >> 5] = s2;
    }
    __syncthreads();
    if (part == 0 && col < L.vdim) {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < DVP / 32; ++i) ss += ssn[i];
      out[(size_t)(row0 + r) * ko + h * L.vdim + col] = Elem<T>::from(yy / sqrtf(ss / (float)L.vdim + eps) * nw * cd_sigmoid(cur.z));
    }
    if (h == L.heads - 1 && L.heads * L.vdim + tid < ko) out[(size_t)(row0 + r) * ko + L.heads * L.vdim + tid] = Elem<T>::from(0.f);
  }
  if (!commit) return;
#pragma unroll
  for (int i = 0; i < RP; ++i) {
    const int r = part * RP + i;
    if (r < L.dim && col < L.vdim) Sg[(size_t)r * L.vdim + col] = S[i];
  }
  // every q / k channel belongs to one CTA only when heads do not share them; cd_tail writes the tail otherwise
  if (L.heads == L.kv_heads && live && role < 3)
#pragma unroll
    for (int j = 0; j < NT - 1; ++j) {
      const int i = j - (NT - L.taps);
      if (i >= 0) tail[(size_t)i * C + ch] = Elem<T>::from(win[j]);
    }
}

// ---- the same in parts ---------------------------------------------------------------------------------------------------------
// out [rows][channels] = activated convolutions; grid (ceil(channels / 256), row chunks of 32, segments)
template <typename T>
__global__ void __launch_bounds__(256) cd_conv_kernel(T* __restrict__ out, const T* __restrict__ proj, long ldp,
                                                      const float* __restrict__ conv_w, const T* __restrict__ conv_state,
                                                      const int* __restrict__ seg_slot, const int* __restrict__ seg_row0,
                                                      const int* __restrict__ seg_nrows, CdLayer L) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = blockIdx.x * 256 + threadIdx.x, seg = blockIdx.z, n = seg_nrows[seg], r0 = blockIdx.y * 32, C = L.channels();
  if (c >= C || r0 >= n) return;
  const int row0 = seg_row0[seg];
  const T* tail = conv_state + (size_t)seg_slot[seg] * (L.taps - 1) * C;
  float w[CD_TAPS], win[CD_TAPS - 1];
  cd_load_taps(w, conv_w, c, L.taps);
#pragma unroll
  for (int j = 0; j < CD_TAPS - 1; ++j) win[j] = cd_input(proj, ldp, L.q_off, tail, C, L.taps, row0, r0 + j - (CD_TAPS - 1), c);
  for (int r = r0; r < min(n, r0 + 32); ++r)
    out[(size_t)(row0 + r) * C + c] =
        Elem<T>::from(cd_conv_step<T, CD_TAPS>(w, win, Elem<T>::to(proj[(size_t)(row0 + r) * ldp + L.q_off + c])));
}

// y [rows][heads][vdim] fp32. grid (ceil(vdim / 32), heads, segments), 8 warps: warp p holds rows p, p + 8, ... of 32 state columns
template <typename T, int RP>
__global__ void __launch_bounds__(256)
cd_rec_kernel(float* __restrict__ y, float* __restrict__ rec_state, const T* __restrict__ qkv, const T* __restrict__ proj, long ldp,
              const float* __restrict__ decay, long ldd, const float* __restrict__ A_log, const float* __restrict__ dt_bias,
              const int* __restrict__ seg_slot, const int* __restrict__ seg_row0, const int* __restrict__ seg_nrows, CdLayer L, int commit) {
  constexpr int DK = RP * 8;
  __shared__ float qs[DK], ks[DK], gs[DK], red1[8][32], red2[8][32], ssq[2][8];
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.y, seg = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, col = blockIdx.x * 32 + lane;
  const int n = seg_nrows[seg];
  if (n <= 0) return;
  const int row0 = seg_row0[seg], kh = h / (L.heads / L.kv_heads), C = L.channels();
  float* Sg = rec_state + ((size_t)seg_slot[seg] * L.heads + h) * L.dim * L.vdim;
  float S[RP];
#pragma unroll
  for (int i = 0; i < RP; ++i) {
    const int r = warp + 8 * i;
    S[i] = r < L.dim && col < L.vdim ? Sg[(size_t)r * L.vdim + col] : 0.f;
  }
  const float expA = expf(A_log[h]), qscale = 1.f / sqrtf((float)L.dim);
  for (int r = 0; r < n; ++r) {
    const size_t row = row0 + r;
    const T* xr = qkv + row * C;
    float sq = 0.f, sk = 0.f;
    for (int c = tid; c < DK; c += 256) {
      const float qv = c < L.dim ? Elem<T>::to(xr[kh * L.dim + c]) : 0.f, kv = c < L.dim ? Elem<T>::to(xr[(L.kv_heads + kh) * L.dim + c]) : 0.f;
      qs[c] = qv; ks[c] = kv;
      gs[c] = c < L.dim ? expf(cd_log_decay(expA, decay[row * ldd + h * L.dim + c] + dt_bias[h * L.dim + c])) : 0.f;
      sq += qv * qv; sk += kv * kv;
    }
    sq = warp_sum(sq); sk = warp_sum(sk);
    if (lane == 0) { ssq[0][warp] = sq; ssq[1][warp] = sk; }
    const float v = col < L.vdim ? Elem<T>::to(xr[2 * L.kv_heads * L.dim + h * L.vdim + col]) : 0.f;
    const float beta = cd_sigmoid(Elem<T>::to(proj[row * ldp + L.b_off() + h]));
    __syncthreads();
    sq = sk = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) { sq += ssq[0][i]; sk += ssq[1][i]; }
    const float rq = qscale / sqrtf(sq + CD_UNIT_EPS), rk = 1.f / sqrtf(sk + CD_UNIT_EPS);
    float p = 0.f;
#pragma unroll
    for (int i = 0; i < RP; ++i) {
      S[i] *= gs[warp + 8 * i];
      p = fmaf(S[i], ks[warp + 8 * i], p);
    }
    red1[warp][lane] = p;
    __syncthreads();
    float kv = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) kv += red1[i][lane];
    const float u = (v - kv * rk) * beta * rk;
    float yp = 0.f;
#pragma unroll
    for (int i = 0; i < RP; ++i) {
      S[i] = fmaf(ks[warp + 8 * i], u, S[i]);
      yp = fmaf(S[i], qs[warp + 8 * i], yp);
    }
    red2[warp][lane] = yp;
    __syncthreads();
    if (warp == 0 && col < L.vdim) {
      float yy = 0.f;
#pragma unroll
      for (int i = 0; i < 8; ++i) yy += red2[i][lane];
      y[(row * L.heads + h) * L.vdim + col] = yy * rq;
    }
    __syncthreads();
  }
  if (commit)
#pragma unroll
    for (int i = 0; i < RP; ++i) {
      const int r = warp + 8 * i;
      if (r < L.dim && col < L.vdim) Sg[(size_t)r * L.vdim + col] = S[i];
    }
}

// grid (ceil(channels / 256), segments)
template <typename T>
__global__ void __launch_bounds__(256) cd_tail_kernel(T* __restrict__ conv_state, const T* __restrict__ proj, long ldp,
                                                      const int* __restrict__ seg_slot, const int* __restrict__ seg_row0,
                                                      const int* __restrict__ seg_nrows, CdLayer L) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = blockIdx.x * 256 + threadIdx.x, seg = blockIdx.y, n = seg_nrows[seg], C = L.channels();
  if (c >= C || n <= 0) return;
  T* tail = conv_state + (size_t)seg_slot[seg] * (L.taps - 1) * C;
  for (int j = 0; j < L.taps - 1; ++j) {                    // row j takes row j + n: later rows are still the old ones
    const int r = n - (L.taps - 1) + j;
    tail[(size_t)j * C + c] = r >= 0 ? proj[(size_t)(seg_row0[seg] + r) * ldp + L.q_off + c] : tail[(size_t)(j + n) * C + c];
  }
}

}  // namespace fb

using namespace fb;
using bf16 = __nv_bfloat16;

static bool cd_ok(const CdLayer& L) {
  return L.heads > 0 && L.kv_heads > 0 && L.heads % L.kv_heads == 0 && L.dim > 0 && L.dim <= 512 && L.vdim > 0 && L.taps >= 1 &&
         L.taps <= CD_TAPS && L.heads <= 65535;
}

extern "C" int fb_cd_lowrank(float* out, const void* proj, long ldp, const void* wa, int na, int ra, const void* wg, int ng, int rg,
                             int rows, int f32, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (ra % 4 || rg % 4 || ldp % 4) return -1;
  const dim3 grid((na + ng + 31) / 32);
  if (f32)
    return (int)launch_pdl(cd_lowrank_kernel<float>, grid, dim3(256), 0, s, out, (const float*)proj, ldp, (const float*)wa, na, ra,
                           (const float*)wg, ng, rg, rows);
  return (int)launch_pdl(cd_lowrank_kernel<bf16>, grid, dim3(256), 0, s, out, (const bf16*)proj, ldp, (const bf16*)wa, na, ra,
                         (const bf16*)wg, ng, rg, rows);
}

template <typename T>
static int cd_step(void* out, int ko, float* rec, void* tail, const void* proj, long ldp, const float* decay, long ldd, const float* gate,
                   long ldg, const float* conv_w, const float* A_log, const float* dt_bias, const float* norm_w, const int* seg_slot,
                   const int* seg_row0, const int* seg_nrows, int nseg, CdLayer L, float eps, int commit, cudaStream_t s) {
  auto go = [&](auto kern) {
    return (int)launch_pdl(kern, dim3(L.heads, nseg), dim3(CD_THREADS), 0, s, (T*)out, ko, rec, (T*)tail, (const T*)proj, ldp, decay, ldd,
                           gate, ldg, conv_w, A_log, dt_bias, norm_w, seg_slot, seg_row0, seg_nrows, L, eps, commit);
  };
  if (L.taps <= 4) {
    if (L.dim <= 64) return L.vdim <= 64 ? go(cd_step_kernel<T, 64, 64, 4>) : go(cd_step_kernel<T, 64, 128, 4>);
    return L.vdim <= 64 ? go(cd_step_kernel<T, 128, 64, 4>) : go(cd_step_kernel<T, 128, 128, 4>);
  }
  if (L.dim <= 64) return L.vdim <= 64 ? go(cd_step_kernel<T, 64, 64, CD_TAPS>) : go(cd_step_kernel<T, 64, 128, CD_TAPS>);
  return L.vdim <= 64 ? go(cd_step_kernel<T, 128, 64, CD_TAPS>) : go(cd_step_kernel<T, 128, 128, CD_TAPS>);
}

template <typename T>
static int cd_tail(void* tail, const void* proj, long ldp, const int* seg_slot, const int* seg_row0, const int* seg_nrows, int nseg, CdLayer L,
                   cudaStream_t s) {
  if (L.taps < 2) return 0;
  return (int)launch_pdl(cd_tail_kernel<T>, dim3((L.channels() + 255) / 256, nseg), dim3(256), 0, s, (T*)tail, (const T*)proj, ldp, seg_slot,
                         seg_row0, seg_nrows, L);
}

// decay: [rows][heads * dim] (stride ldd), gate: [rows][heads * vdim] (ldg), both fp32; out [rows][ko]. -20: sizes for the split form.
extern "C" int fb_cd_step(void* out, int ko, float* rec, void* tail, const void* proj, long ldp, const float* decay, long ldd,
                          const float* gate, long ldg, const float* conv_w, const float* A_log, const float* dt_bias, const float* norm_w,
                          const int* seg_slot, const int* seg_row0, const int* seg_nrows, int nseg, int heads, int kv_heads, int dim,
                          int vdim, int taps, int q_off, float eps, int commit, int f32, cudaStream_t s) {
  if (nseg <= 0) return 0;
  const CdLayer L{heads, kv_heads, dim, vdim, taps, q_off};
  if (!cd_ok(L) || ko < heads * vdim || ko - heads * vdim > CD_THREADS || nseg > 65535) return -1;
  if (dim > 128 || vdim > 128) return -20;
  return f32 ? cd_step<float>(out, ko, rec, tail, proj, ldp, decay, ldd, gate, ldg, conv_w, A_log, dt_bias, norm_w, seg_slot, seg_row0,
                              seg_nrows, nseg, L, eps, commit, s)
             : cd_step<bf16>(out, ko, rec, tail, proj, ldp, decay, ldd, gate, ldg, conv_w, A_log, dt_bias, norm_w, seg_slot, seg_row0,
                             seg_nrows, nseg, L, eps, commit, s);
}

extern "C" int fb_cd_tail(void* tail, const void* proj, long ldp, const int* seg_slot, const int* seg_row0, const int* seg_nrows, int nseg,
                          int heads, int kv_heads, int dim, int vdim, int taps, int q_off, int f32, cudaStream_t s) {
  if (nseg <= 0) return 0;
  const CdLayer L{heads, kv_heads, dim, vdim, taps, q_off};
  if (!cd_ok(L) || nseg > 65535) return -1;
  return f32 ? cd_tail<float>(tail, proj, ldp, seg_slot, seg_row0, seg_nrows, nseg, L, s)
             : cd_tail<bf16>(tail, proj, ldp, seg_slot, seg_row0, seg_nrows, nseg, L, s);
}

template <typename T>
static int cd_rec(float* y, float* rec, void* qkv, const void* tail, const void* proj, long ldp, const float* decay, long ldd,
                  const float* conv_w, const float* A_log, const float* dt_bias, const int* seg_slot, const int* seg_row0,
                  const int* seg_nrows, int nseg, int max_rows, CdLayer L, int commit, cudaStream_t s) {
  cudaError_t e = launch_pdl(cd_conv_kernel<T>, dim3((L.channels() + 255) / 256, (max_rows + 31) / 32, nseg), dim3(256), 0, s, (T*)qkv,
                             (const T*)proj, ldp, conv_w, (const T*)tail, seg_slot, seg_row0, seg_nrows, L);
  if (e != cudaSuccess) return (int)e;
  auto go = [&](auto kern) {
    return (int)launch_pdl(kern, dim3((L.vdim + 31) / 32, L.heads, nseg), dim3(256), 0, s, y, rec, (const T*)qkv, (const T*)proj, ldp, decay,
                           ldd, A_log, dt_bias, seg_slot, seg_row0, seg_nrows, L, commit);
  };
  if (L.dim <= 64) return go(cd_rec_kernel<T, 8>);
  if (L.dim <= 128) return go(cd_rec_kernel<T, 16>);
  if (L.dim <= 256) return go(cd_rec_kernel<T, 32>);
  return go(cd_rec_kernel<T, 64>);
}

// qkv: scratch [rows][channels] in the projection's type; y [rows][heads][vdim] fp32, before the gated norm. The tail is left as it is.
extern "C" int fb_cd_rec(float* y, float* rec, void* qkv, const void* tail, const void* proj, long ldp, const float* decay, long ldd,
                         const float* conv_w, const float* A_log, const float* dt_bias, const int* seg_slot, const int* seg_row0,
                         const int* seg_nrows, int nseg, int max_rows, int heads, int kv_heads, int dim, int vdim, int taps, int q_off,
                         int commit, int f32, cudaStream_t s) {
  if (nseg <= 0 || max_rows <= 0) return 0;
  const CdLayer L{heads, kv_heads, dim, vdim, taps, q_off};
  if (!cd_ok(L) || nseg > 65535 || (max_rows + 31) / 32 > 65535) return -1;
  return f32 ? cd_rec<float>(y, rec, qkv, tail, proj, ldp, decay, ldd, conv_w, A_log, dt_bias, seg_slot, seg_row0, seg_nrows, nseg, max_rows, L,
                             commit, s)
             : cd_rec<bf16>(y, rec, qkv, tail, proj, ldp, decay, ldd, conv_w, A_log, dt_bias, seg_slot, seg_row0, seg_nrows, nseg, max_rows, L,
                            commit, s);
}
