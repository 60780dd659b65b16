// State-space recurrence of prompt segments in chunks of 64 rows (state-space duality; operands bf16, state fp32):
//
//   with a_t = A dt_t and G_t = a_1 + .. + a_t inside a chunk, S the state that enters it:
//     y_t   = e^{G_t} S^T C_t  +  sum over s <= t of (C_t . B_s) e^{G_t - G_s} dt_s x_s  +  skip x_t
//     S'    = e^{G_end} S  +  sum over s of e^{G_end - G_s} dt_s B_s x_s^T
//
//   ssd_state  per (chunk, head): what the chunk adds to the state, as a product of (weighted B)^T and x on the tensor cores (mma.sync)
//   ssd_scan   per element of a state: the states that enter the chunks, one after another, and the last one into the slot
//   ssd_out    per (chunk, head): scores C B^T, weighted in registers, times x, plus C times the entering state
//
// Weights and states enter the bf16 products as a value plus its remainder, which keeps 16 bits of them; all exponents are <= 0. Sums of
// a_t are formed in double and kept as a float and its remainder, so differences of long sums keep their digits. grid.y = (head, tile of 64
// columns of V); shared memory rows are padded by 8 elements.
#include "api_listed.h"
#include "common.cuh"

namespace fb {

using bf16 = __nv_bfloat16;

constexpr int SD_Q = 64, SD_THREADS = 256, SD_V = 64, SD_LDX = SD_V + 8;

__device__ __forceinline__ void sd_cp16(void* smem, const void* gmem, bool valid) {
  const int sz = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(smem)), "l"(gmem), "r"(sz) : "memory");
}
__device__ __forceinline__ void sd_cp_wait() { asm volatile("cp.async.wait_all;" ::: "memory"); }

__device__ __forceinline__ void sd_ldsm(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void sd_ldsm_t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void sd_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

struct SdDims {
  int heads, groups, N, V, NP, VT;      // NP: N rounded up to 16; VT: tiles of 64 columns
  int inner, ch;
};

// rows x cols of a row-major source (ld elements apart) into smem rows of lds elements, zeros beyond; VEC: 8 elements at a time, without
// waiting (sd_cp_wait does)
template <bool VEC>
__device__ __forceinline__ void sd_load(bf16* dst, int lds, const bf16* src, long ld, int rows, int cols, int cols_pad) {
  if (VEC) {
    const int per = cols_pad / 8;
    for (int i = threadIdx.x; i < SD_Q * per; i += SD_THREADS) {
      const int r = i / per, c = i % per * 8;
      const bool ok = r < rows && c < cols;
      sd_cp16(dst + r * lds + c, src + (ok ? (size_t)r * ld + c : 0), ok);
    }
  } else {
    for (int i = threadIdx.x; i < SD_Q * cols_pad; i += SD_THREADS) {
      const int r = i / cols_pad, c = i % cols_pad;
      dst[r * lds + c] = r < rows && c < cols ? src[(size_t)r * ld + c] : f2bf(0.f);
    }
  }
}

// rowinfo[row][head] = (G, its remainder, dt); end[(seg, chunk)][head] = e^{G_end}; states[(seg, chunk)][head][N][V]
template <bool VEC>
__global__ void __launch_bounds__(SD_THREADS) ssd_state_kernel(float* __restrict__ states, float4* __restrict__ rowinfo, float* __restrict__ ends,
                                                               const bf16* __restrict__ xbc, const bf16* __restrict__ proj, long ldp,
                                                               const float* __restrict__ A, const float* __restrict__ dt_bias,
                                                               const int* __restrict__ seg_row0, const int* __restrict__ seg_nrows, SdDims d,
                                                               int chunks) {
  extern __shared__ __align__(16) unsigned char sd_smem[];
  const int LDN = d.NP + 8;
  bf16* sH = reinterpret_cast<bf16*>(sd_smem);               // [64][LDN] weighted B: value
  bf16* sL = sH + SD_Q * LDN;                                // ... remainder
  bf16* sX = sL + SD_Q * LDN;                                // [64][LDX]
  float* wt = reinterpret_cast<float*>(sX + SD_Q * SD_LDX);  // [64]
  pdl_launch_dependents();
  pdl_wait();
  xbc = after_wait(xbc); proj = after_wait(proj);
  const int c = blockIdx.x, h = blockIdx.y / d.VT, v0 = blockIdx.y % d.VT * SD_V, seg = blockIdx.z;
  const int n = seg_nrows[seg] - c * SD_Q;
  if (n <= 0) return;
  const int here = min(SD_Q, n), row0 = seg_row0[seg] + c * SD_Q, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bf16* rows = xbc + (size_t)row0 * d.ch;
  sd_load<VEC>(sX, SD_LDX, rows + h * d.V + v0, d.ch, here, min(SD_V, d.V - v0), SD_V);
  sd_load<VEC>(sH, LDN, rows + d.inner + h / (d.heads / d.groups) * d.N, d.ch, here, d.N, d.NP);
  if (warp == 0) {
    float dt[2];
    double a[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = 2 * lane + e;
      dt[e] = 0.f;
      if (t < here) {
        const float z = bf2f(proj[(size_t)(row0 + t) * ldp + d.inner + d.ch + h]) + dt_bias[h];
        dt[e] = z > 20.f ? z : log1pf(expf(z));
      }
      a[e] = (double)(A[h] * dt[e]);
    }
    double s = a[0] + a[1];
    for (int o = 1; o < 32; o <<= 1) {
      const double p = __shfl_up_sync(0xffffffffu, s, o);
      if (lane >= o) s += p;
    }
    const double G[2] = {s - a[1], s}, end = __shfl_sync(0xffffffffu, s, 31);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = 2 * lane + e;
      wt[t] = expf((float)(end - G[e])) * dt[e];
      if (v0 == 0 && t < here) {
        const float hi = (float)G[e];
        rowinfo[(size_t)(row0 + t) * d.heads + h] = make_float4(hi, (float)(G[e] - (double)hi), dt[e], 0.f);
      }
    }
    if (v0 == 0 && lane == 0) ends[((size_t)seg * chunks + c) * d.heads + h] = expf((float)end);
  }
  if (VEC) sd_cp_wait();
  __syncthreads();
  for (int i = threadIdx.x; i < SD_Q * d.NP / 2; i += SD_THREADS) {
    const int t = i / (d.NP / 2), at = t * LDN + i % (d.NP / 2) * 2;
    const uint32_t u = *reinterpret_cast<const uint32_t*>(sH + at);
    const float a = bf_lo(u) * wt[t], b = bf_hi(u) * wt[t];
    const uint32_t v = pack_bf2(a, b);
    *reinterpret_cast<uint32_t*>(sH + at) = v;
    *reinterpret_cast<uint32_t*>(sL + at) = pack_bf2(a - bf_lo(v), b - bf_hi(v));
  }
  __syncthreads();
  float* out = states + (((size_t)seg * chunks + c) * d.heads + h) * d.N * d.V;
  // warps 0 .. 3 take the first 32 columns of the tile, warps 4 .. 7 the others
  const int vh = warp / 4 * 32;
  for (int m0 = warp % 4 * 16; m0 < d.NP; m0 += 64) {
    float acc[4][4] = {};
#pragma unroll
    for (int k0 = 0; k0 < SD_Q; k0 += 16) {
      uint32_t ah[4], al[4];
      const int at = (k0 + (lane & 7) + (lane >> 4) * 8) * LDN + m0 + ((lane >> 3) & 1) * 8;
      sd_ldsm_t(ah, sH + at);
      sd_ldsm_t(al, sL + at);
#pragma unroll
      for (int np = 0; np < 2; ++np) {
        uint32_t b[4];
        sd_ldsm_t(b, sX + (k0 + ((lane >> 3) & 1) * 8 + (lane & 7)) * SD_LDX + vh + np * 16 + (lane >> 4) * 8);
        sd_mma(acc[2 * np], ah, b[0], b[1]);
        sd_mma(acc[2 * np + 1], ah, b[2], b[3]);
        sd_mma(acc[2 * np], al, b[0], b[1]);
        sd_mma(acc[2 * np + 1], al, b[2], b[3]);
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = m0 + lane / 4 + (e >> 1) * 8, v = v0 + vh + i * 8 + (lane & 3) * 2 + (e & 1);
        if (VEC) {
          if ((e & 1) == 0 && r < d.N && v < d.V) *reinterpret_cast<float2*>(out + (size_t)r * d.V + v) = make_float2(acc[i][e], acc[i][e + 1]);
        } else if (r < d.N && v < d.V) {
          out[(size_t)r * d.V + v] = acc[i][e];
        }
      }
  }
}

// grid (elements / 256, heads, segments): the sums of the chunks give way to the states that enter them
__global__ void __launch_bounds__(256) ssd_scan_kernel(float* __restrict__ states, const float* __restrict__ ends, float* __restrict__ rec,
                                                       const int* __restrict__ seg_slot, const int* __restrict__ seg_nrows, SdDims d, int chunks) {
  pdl_launch_dependents();
  pdl_wait();
  ends = after_wait(ends);
  const int i = blockIdx.x * 256 + threadIdx.x, h = blockIdx.y, seg = blockIdx.z, size = d.N * d.V;
  const int nc = (seg_nrows[seg] + SD_Q - 1) / SD_Q;
  if (i >= size || nc <= 0) return;
  float* slot = rec + ((size_t)seg_slot[seg] * d.heads + h) * size + i;
  float* st = states + ((size_t)seg * chunks * d.heads + h) * size + i;
  const float* en = ends + (size_t)seg * chunks * d.heads + h;
  const size_t step = (size_t)d.heads * size;
  float S = *slot;
  for (int c = 0; c < nc; c += 8) {
    float add[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) add[j] = c + j < nc ? st[(c + j) * step] : 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (c + j >= nc) break;
      st[(c + j) * step] = S;
      S = fmaf(en[(size_t)(c + j) * d.heads], S, add[j]);
    }
  }
  *slot = S;
}

template <bool VEC>
__global__ void __launch_bounds__(SD_THREADS) ssd_out_kernel(float* __restrict__ y, long ldy, const float* __restrict__ states,
                                                             const float4* __restrict__ rowinfo, const bf16* __restrict__ xbc,
                                                             const float* __restrict__ skip, const int* __restrict__ seg_row0,
                                                             const int* __restrict__ seg_nrows, SdDims d, int chunks) {
  extern __shared__ __align__(16) unsigned char sd_smem[];
  const int LDN = d.NP + 8;
  bf16* sC = reinterpret_cast<bf16*>(sd_smem);               // [64][LDN]
  bf16* sB = sC + SD_Q * LDN;                                // [64][LDN]
  bf16* sX = sB + SD_Q * LDN;                                // [64][LDX]
  bf16* sS = sX + SD_Q * SD_LDX;                             // [2][NP][LDX] entering state: value, remainder
  float4* info = reinterpret_cast<float4*>(sS + 2 * d.NP * SD_LDX);      // [64]
  pdl_launch_dependents();
  pdl_wait();
  states = after_wait(states); rowinfo = after_wait(rowinfo); xbc = after_wait(xbc);
  const int c = blockIdx.x, h = blockIdx.y / d.VT, v0 = blockIdx.y % d.VT * SD_V, seg = blockIdx.z;
  const int n = seg_nrows[seg] - c * SD_Q;
  if (n <= 0) return;
  const int here = min(SD_Q, n), row0 = seg_row0[seg] + c * SD_Q, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = h / (d.heads / d.groups);
  const bf16* rows = xbc + (size_t)row0 * d.ch;
  sd_load<VEC>(sC, LDN, rows + d.inner + (d.groups + g) * d.N, d.ch, here, d.N, d.NP);
  sd_load<VEC>(sB, LDN, rows + d.inner + g * d.N, d.ch, here, d.N, d.NP);
  sd_load<VEC>(sX, SD_LDX, rows + h * d.V + v0, d.ch, here, min(SD_V, d.V - v0), SD_V);
  const float* st = states + (((size_t)seg * chunks + c) * d.heads + h) * d.N * d.V;
  if (VEC) {
    for (int i = threadIdx.x; i < d.NP * (SD_V / 4); i += SD_THREADS) {
      const int r = i / (SD_V / 4), v = i % (SD_V / 4) * 4;
      const float4 f = r < d.N && v0 + v < d.V ? *reinterpret_cast<const float4*>(st + (size_t)r * d.V + v0 + v) : make_float4(0.f, 0.f, 0.f, 0.f);
      const uint32_t a = pack_bf2(f.x, f.y), b = pack_bf2(f.z, f.w);
      *reinterpret_cast<uint2*>(sS + r * SD_LDX + v) = make_uint2(a, b);
      *reinterpret_cast<uint2*>(sS + (d.NP + r) * SD_LDX + v) = make_uint2(pack_bf2(f.x - bf_lo(a), f.y - bf_hi(a)), pack_bf2(f.z - bf_lo(b), f.w - bf_hi(b)));
    }
  } else {
    for (int i = threadIdx.x; i < d.NP * SD_V; i += SD_THREADS) {
      const int r = i / SD_V, v = i % SD_V;
      const float f = r < d.N && v0 + v < d.V ? st[(size_t)r * d.V + v0 + v] : 0.f;
      const bf16 a = f2bf(f);
      sS[r * SD_LDX + v] = a;
      sS[(d.NP + r) * SD_LDX + v] = f2bf(f - bf2f(a));
    }
  }
  for (int t = threadIdx.x; t < SD_Q; t += SD_THREADS)
    info[t] = t < here ? rowinfo[(size_t)(row0 + t) * d.heads + h] : make_float4(0.f, 0.f, 0.f, 0.f);
  if (VEC) sd_cp_wait();
  __syncthreads();
  // warp: 16 rows against the rows up to its last one, half of the tile's columns
  const int tw = warp % 4, t0 = tw * 16, r_lo = t0 + lane / 4, vh = warp / 4 * 32;
  float sc[8][4] = {}, inter[4][4] = {}, acc[4][4] = {};
  for (int ks = 0; ks < d.NP / 16; ++ks) {
    uint32_t a[4];
    sd_ldsm(a, sC + (t0 + (lane & 7) + ((lane >> 3) & 1) * 8) * LDN + ks * 16 + (lane >> 4) * 8);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      if (j > tw) break;
      uint32_t b[4];
      sd_ldsm(b, sB + (j * 16 + (lane >> 4) * 8 + (lane & 7)) * LDN + ks * 16 + ((lane >> 3) & 1) * 8);
      sd_mma(sc[2 * j], a, b[0], b[1]);
      sd_mma(sc[2 * j + 1], a, b[2], b[3]);
    }
#pragma unroll
    for (int part = 0; part < 2; ++part)
#pragma unroll
      for (int np = 0; np < 2; ++np) {
        uint32_t b[4];
        sd_ldsm_t(b, sS + (part * d.NP + ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * SD_LDX + vh + np * 16 + (lane >> 4) * 8);
        sd_mma(inter[2 * np], a, b[0], b[1]);
        sd_mma(inter[2 * np + 1], a, b[2], b[3]);
      }
  }
  const float4 it[2] = {info[r_lo], info[r_lo + 8]};
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    if (j > tw) break;
    uint32_t ah[4], al[4];
#pragma unroll
    for (int half = 0; half < 2; ++half)
#pragma unroll
      for (int hr = 0; hr < 2; ++hr) {
        float p[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int s = (2 * j + half) * 8 + (lane & 3) * 2 + e, t = r_lo + 8 * hr;
          const float4 is = info[s];
          p[e] = s <= t ? sc[2 * j + half][2 * hr + e] * __expf((it[hr].x - is.x) + (it[hr].y - is.y)) * is.z : 0.f;
        }
        const uint32_t v = pack_bf2(p[0], p[1]);
        ah[half * 2 + hr] = v;
        al[half * 2 + hr] = pack_bf2(p[0] - bf_lo(v), p[1] - bf_hi(v));
      }
#pragma unroll
    for (int np = 0; np < 2; ++np) {
      uint32_t b[4];
      sd_ldsm_t(b, sX + (j * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * SD_LDX + vh + np * 16 + (lane >> 4) * 8);
      sd_mma(acc[2 * np], ah, b[0], b[1]);
      sd_mma(acc[2 * np + 1], ah, b[2], b[3]);
      sd_mma(acc[2 * np], al, b[0], b[1]);
      sd_mma(acc[2 * np + 1], al, b[2], b[3]);
    }
  }
  const float sk = skip[h];
#pragma unroll
  for (int hr = 0; hr < 2; ++hr) {
    const int t = r_lo + 8 * hr;
    if (t >= here) continue;
    const float dec = __expf(it[hr].x + it[hr].y);
    float* dst = y + (size_t)(row0 + t) * ldy + (size_t)h * d.V;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int v = vh + i * 8 + (lane & 3) * 2;
      float o[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) o[e] = fmaf(dec, inter[i][2 * hr + e], acc[i][2 * hr + e]) + sk * bf2f(sX[t * SD_LDX + v + e]);
      if (VEC) {
        if (v0 + v < d.V) *reinterpret_cast<float2*>(dst + v0 + v) = make_float2(o[0], o[1]);
      } else {
        if (v0 + v < d.V) dst[v0 + v] = o[0];
        if (v0 + v + 1 < d.V) dst[v0 + v + 1] = o[1];
      }
    }
  }
}

static size_t up256(size_t n) { return (n + 255) & ~(size_t)255; }

}  // namespace fb

using namespace fb;

extern "C" long fb_ssd_chunk_scratch_bytes(int rows, int nseg, int max_rows, int heads, int N, int V) {
  const size_t chunks = (size_t)nseg * ((max_rows + SD_Q - 1) / SD_Q);
  return (long)(up256(chunks * heads * N * V * 4) + up256((size_t)rows * heads * 16) + up256(chunks * heads * 4));
}

// xbc: convolved rows [T][channels] dense; proj: the projection's rows (dt behind its first inner + channels columns), of which `rows` are the
// step's; y fp32 rows ldy apart. Returns -20 for states of more than 256 rows.
extern "C" int fb_ssd_chunk(float* y, long ldy, float* rec, void* scratch, const void* xbc, const void* proj, long ldp, const float* A,
                            const float* dt_bias, const float* skip, const int* seg_slot, const int* seg_row0, const int* seg_nrows, int nseg,
                            int max_rows, int rows, int heads, int groups, int N, int V, cudaStream_t s) {
  if (nseg <= 0 || max_rows <= 0 || rows <= 0) return 0;
  if (heads < 1 || groups < 1 || heads % groups || N < 1 || V < 1 || nseg > 65535) return -1;
  if (N > 256) return -20;
  SdDims d;
  d.heads = heads; d.groups = groups; d.N = N; d.V = V; d.NP = (N + 15) / 16 * 16; d.VT = (V + SD_V - 1) / SD_V;
  d.inner = heads * V; d.ch = d.inner + 2 * groups * N;
  if ((long)heads * d.VT > 65535) return -1;
  const int chunks = (max_rows + SD_Q - 1) / SD_Q;
  char* p = (char*)scratch;
  float* states = (float*)p;
  float4* rowinfo = (float4*)(p + up256((size_t)nseg * chunks * heads * N * V * 4));
  float* ends = (float*)((char*)rowinfo + up256((size_t)rows * heads * 16));
  const bool vec = N % 8 == 0 && V % 8 == 0 && ldy % 2 == 0 && (((uintptr_t)xbc | (uintptr_t)rec) & 15) == 0 && ((uintptr_t)y & 7) == 0;
  const int LDN = d.NP + 8;
  const size_t sm1 = (size_t)(2 * SD_Q * LDN + SD_Q * SD_LDX) * 2 + SD_Q * 4;
  const size_t sm2 = (size_t)(2 * SD_Q * LDN + SD_Q * SD_LDX + 2 * d.NP * SD_LDX) * 2 + SD_Q * 16;
  const dim3 grid(chunks, heads * d.VT, nseg);
  auto go = [&](auto k1, auto k2) {
    cudaError_t e = cudaFuncSetAttribute(k1, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm1);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(k2, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm2);
    if (e != cudaSuccess) return (int)e;
    int rc = (int)launch_pdl(k1, grid, dim3(SD_THREADS), sm1, s, states, rowinfo, ends, (const bf16*)xbc, (const bf16*)proj, ldp, A, dt_bias, seg_row0,
                             seg_nrows, d, chunks);
    if (!rc) rc = (int)launch_pdl(ssd_scan_kernel, dim3((N * V + 255) / 256, heads, nseg), dim3(256), 0, s, states, (const float*)ends, rec, seg_slot,
                                  seg_nrows, d, chunks);
    if (!rc) rc = (int)launch_pdl(k2, grid, dim3(SD_THREADS), sm2, s, y, ldy, (const float*)states, (const float4*)rowinfo, (const bf16*)xbc, skip,
                                  seg_row0, seg_nrows, d, chunks);
    return rc;
  };
  return vec ? go(ssd_state_kernel<true>, ssd_out_kernel<true>) : go(ssd_state_kernel<false>, ssd_out_kernel<false>);
}
