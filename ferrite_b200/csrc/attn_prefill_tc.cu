// Causal flash attention for prompt chunks on the 5th-generation tensor cores (tcgen05 + TMEM), over the paged KV cache.
//
// One CTA = 128 query rows of one q head; keys stream in tiles of 64 (one or part of one KV page) through a two-stage
// TMA pipeline. Warp roles: warp 0 lane 0 issues the TMA loads, warp 1 lane 0 issues every tcgen05.mma, warps 2..9
// (256 threads, two per query row = TMEM lane, each taking half of a tile's keys and half of the O columns) run the
// online softmax and the epilogue: two warps per SM sub-partition, so one's TMEM / ex2 latencies hide behind the other.
//
//   S = Q K^T        SS form: Q and K tiles in shared memory (K-major, 128-byte swizzle), S in TMEM (2 buffers x 64 cols)
//   P = exp2(S - m)  softmax threads read S with tcgen05.ld, write P as packed bf16 back into TMEM with tcgen05.st
//   O += P V         TS form: A = P from TMEM, B = the V tile in shared memory read MN-major (V rows are keys, the
//                    head dim is contiguous), O in TMEM (head_dim columns) for the whole key loop
//
// The running maximum only moves when a row's new maximum exceeds it by more than 2^8 (then the O accumulator is
// rescaled in TMEM; between such events P may exceed 1, which bf16 and the fp32 row sum absorb), so the common key
// tile costs one TMEM read of S and one TMEM write of P per thread. Tensor-pipe order is S(0) S(1) PV(0) S(2) PV(1) ...:
// the softmax of tile j overlaps PV(j-1) and S(j+1). Every mbarrier wait is bounded; a wait that runs out sets the
// status word and an abort flag, all roles leave their loops, and the CTA frees its TMEM and returns.
//
// Counterpart of the reference's `fe_flash_prefill` (`kernels/k-core/src/flash.rs:50`: BQ 64 / BKV 32 on mma.sync with
// the gate epilogue); same contract as `fb_attn_prefill` (sigmoid output gate fused, paged cache with a prefix).
#include "api.h"
#include "common.cuh"
#include "gemm_core.cuh"

namespace fb {

constexpr int FT_BQ = 128, FT_BKV = 64, FT_THREADS = 64 + 256;

__device__ __forceinline__ void tmem_st32(uint32_t taddr, const uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
      "{%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,"
      "%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31,%32};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]),
        "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]),
        "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]), "r"(r[24]), "r"(r[25]), "r"(r[26]),
        "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
      : "memory");
}
__device__ __forceinline__ void tmem_st16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]),
        "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}
__device__ __forceinline__ void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }

// D[tmem] (+)= A[tmem] * B[smem desc]
__device__ __forceinline__ void tc_mma_f16_ts(uint32_t tmem_d, uint32_t tmem_a, uint64_t desc_b, uint32_t idesc,
                                              uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
      ::"r"(tmem_d), "r"(tmem_a), "l"(desc_b), "r"(idesc), "r"(accumulate) : "memory");
}

// MN-major operand tile with the 128-byte swizzle: rows are K (here: keys), each row holds 64 contiguous MN elements
// (128 bytes). Eight rows form one swizzle atom; SBO = bytes between 8-row groups along K, LBO = bytes between
// 64-element chunks along MN.
__device__ __forceinline__ uint64_t umma_desc_mn128(uint32_t smem_addr, uint32_t lbo_bytes, uint32_t sbo_bytes) {
  uint64_t d = 0;
  d |= (uint64_t)((smem_addr & 0x3ffffu) >> 4);
  d |= (uint64_t)((lbo_bytes >> 4) & 0x3fff) << 16;
  d |= (uint64_t)((sbo_bytes >> 4) & 0x3fff) << 32;
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;
  return d;
}

__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// PX: the softmax weights enter the PV product as a bf16 value plus its bf16 remainder (two TS products per k step, a second
// P buffer in TMEM), which keeps 16 bits of their mantissa instead of 8.
// BND: rows see a window or a chunk of the keys, scores are softcapped (cap_log2 = cap * log2 e, scale_log2 then leads to the argument of
// the tanh, which is a polynomial where all scores of a warp's tile are below the cap). Key tiles that no row of the CTA sees are skipped; out_f32: rows of floats.
// Two CTAs share an SM where heads have up to 128 columns (`ft_pair`), so that one's waits hide behind the other's arithmetic: fewer K / V
// buffers, and P and its remainder take the place of the scores they came from (all of them are in registers by then), so that 256 TMEM
// columns do. The scores of tile j + 2 then wait for PV(j), which read that place, instead of for the softmax threads.
constexpr bool ft_pair(int hd, bool bnd) { return bnd && hd <= 128; }
constexpr int ft_k_stages(int hd, bool bnd) { return ft_pair(hd, bnd) ? (hd == 128 ? 2 : 3) : hd == 256 ? 3 : 4; }
constexpr int ft_v_stages(int hd, bool bnd) { return ft_pair(hd, bnd) ? (hd == 128 ? 2 : 3) : hd == 256 ? 2 : 3; }

// DUAL: two softmax maps per head over shared values (a key row holds both maps' keys, a query has zeros in the other's columns). A CTA takes
// both maps of 64 query rows, map 0 in lanes 0..63 and map 1 in lanes 64..127, and ends with the difference of the two, its norm over vdim,
// the scale and the output gate: the maps' own rows never leave the SM.
//
// HD, HV: columns of a head's keys and values. POOL: the means of the blocks before a row's window are keys as well; the CTA's first tiles are
// those of the means that its last row sees, out of a buffer where a segment's means lie side by side from row pool_start[seg] on.
template <int HD, int HV, bool PX, bool BND, bool DUAL, bool POOL>
__global__ void __launch_bounds__(FT_THREADS, ft_pair(HD, BND) ? 2 : 1)
attn_prefill_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                       const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmKp,
                       const __grid_constant__ CUtensorMap tmVp, const int* __restrict__ pool_start, int pool, __nv_bfloat16* __restrict__ out,
                       const __nv_bfloat16* __restrict__ proj, long proj_stride, const int* __restrict__ seg_slot,
                       const int* __restrict__ seg_row0, const int* __restrict__ seg_nrows,
                       const int* __restrict__ seg_pos0, const int* __restrict__ block_table, int max_blocks,
                       int kv_block, int nq, int nkv, int gated, float scale_log2, const float* __restrict__ sink, int window, int chunk,
                       float cap_log2, long ldo, int out_f32, const HeadMix mix, int head_groups, int* status) {
  constexpr int NCH = HD / 64, VCH = HV / 64;      // 64-element (128-byte) chunks of the head dims
  constexpr int Q_CH = FT_BQ * 128;                // bytes of one Q chunk box (128 rows x 128 B)
  constexpr int KV_CH = FT_BKV * 128;              // bytes of one K / V chunk box (64 rows x 128 B)
  constexpr int Q_BYTES = NCH * Q_CH, K_BYTES = NCH * KV_CH, V_BYTES = VCH * KV_CH;
  constexpr bool PAIR = ft_pair(HD, BND);
  // TMEM columns: O | S0 S1 | P0 P1 | remainders; PAIR: O | S0 S1, P and remainder in the place of their S
  constexpr uint32_t COL_O = 0, COL_S = HV, COL_P = PAIR ? COL_S : HV + 2 * FT_BKV;
  constexpr uint32_t P_STEP = PAIR ? FT_BKV : FT_BKV / 2, REM = PAIR ? FT_BKV / 2 : FT_BKV;   // between P buffers; from P to its remainder
  constexpr uint32_t TMEM_COLS = PAIR ? 256 : 512;
  // K runs three tiles ahead at head_dim 256 (S(j+1) is issued a whole tile before PV(j), so with two K buffers a K
  // load had one tile period to arrive and its latency set the pace), four below; V two / three.
  constexpr int KS = ft_k_stages(HD, BND), VS = ft_v_stages(HD, BND);
  // All shared state lives in the dynamic allocation (no static shared memory), so the tile area starts at the
  // 1024-byte aligned base: [Q][K x KS][V x VS][row maxima 2 KB][barriers][flags]
  extern __shared__ __align__(1024) unsigned char smem_raw[];
  unsigned char* sQ = smem_raw;
  unsigned char* sK = sQ + Q_BYTES;                         // [KS][K_BYTES]
  unsigned char* sV = sK + KS * K_BYTES;                    // [VS][V_BYTES]
  float (*mx_s)[2][FT_BQ] = reinterpret_cast<float (*)[2][FT_BQ]>(sV + VS * V_BYTES);   // [2][2][128] by tile parity
  uint64_t* bars = reinterpret_cast<uint64_t*>(sV + VS * V_BYTES + 2 * 2 * FT_BQ * 4);
  uint64_t* q_full = bars;
  uint64_t* s_full = bars + 2;                              // [2]
  uint64_t* s_empty = bars + 4;                             // [2]
  uint64_t* p_full = bars + 6;                              // [2]
  uint64_t* p_empty = bars + 8;                             // [2]: PV(j) has completed (P buffer free, O up to date)
  uint64_t* k_full = bars + 10;                             // [KS]
  uint64_t* k_empty = k_full + KS;
  uint64_t* v_full = k_empty + KS;                          // [VS]
  uint64_t* v_empty = v_full + VS;
  uint32_t* tmem_base_p = reinterpret_cast<uint32_t*>(v_empty + VS);
  int* abort_p = reinterpret_cast<int*>(tmem_base_p + 1);
  int* fail_s = abort_p + 1;                                // [3]: a softmax wait ran out (tile parity; [2]: after the loop)

  // the long (late) query tiles of a group of heads first, so that the last CTAs to start are short ones; one group after another keeps
  // the keys and values in use few enough for L2
  const int seg = blockIdx.z / head_groups, qh = blockIdx.z % head_groups * gridDim.x + blockIdx.x;
  const int qt = (int)gridDim.y - 1 - (int)blockIdx.y;
  pdl_launch_dependents();
  pdl_wait();
  if (qh >= (DUAL ? nq / 2 : nq)) return;
  const int n = seg_nrows[seg];
  constexpr int QR = DUAL ? FT_BQ / 2 : FT_BQ;              // query rows of the CTA
  const int q0 = qt * QR;
  if (q0 >= n) return;                                      // uniform for the CTA, before any barrier or allocation
  if (smem_u32(smem_raw) & 1023u) {                         // the swizzled tiles need the 1024-byte base
    if (threadIdx.x == 0) set_status(status, ST_BOUNDS);
    return;
  }
  const int row0 = seg_row0[seg], pos0 = seg_pos0[seg], slot = seg_slot[seg];
  const int kvh = (DUAL ? 2 * qh : qh) / (nq / nkv);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int tile0 = BND ? first_key(pos0 + q0, window, chunk) / FT_BKV : 0;   // first key tile that a row of the CTA sees
  const int last_pos = pos0 + min(q0 + QR, n) - 1;
  const int np = POOL ? (first_key(last_pos, window, 0) / pool + FT_BKV - 1) / FT_BKV : 0;   // tiles of means
  const int nt = np + last_pos / FT_BKV + 1 - tile0;        // ... and key tiles up to the one the last query row ends in
  volatile int* abort_flag = abort_p;

  if (threadIdx.x == 0) {
    *abort_p = 0;
    fail_s[0] = fail_s[1] = fail_s[2] = 0;
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_full[i], 1); mbar_init(&s_empty[i], 8); mbar_init(&p_full[i], 8); mbar_init(&p_empty[i], 1);
    }
    for (int i = 0; i < KS; ++i) { mbar_init(&k_full[i], 1); mbar_init(&k_empty[i], 1); }
    for (int i = 0; i < VS; ++i) { mbar_init(&v_full[i], 1); mbar_init(&v_empty[i], 1); }
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_base_p, TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_base_p;

  if (warp == 0) {
    if (lane == 0) {
      // ---- TMA producer: K(j+1) is issued before V(j), so the K ring really runs KS - 1 tiles ahead ----------------
      tma_prefetch_desc(&tmQ); tma_prefetch_desc(&tmK); tma_prefetch_desc(&tmV);
      mbar_expect_tx(q_full, Q_BYTES);
#pragma unroll
      for (int c = 0; c < NCH; ++c) {
        if constexpr (DUAL) {
          tma_load_2d(sQ + c * Q_CH, &tmQ, q_full, 2 * qh * HD + c * 64, row0 + q0);
          tma_load_2d(sQ + c * Q_CH + Q_CH / 2, &tmQ, q_full, (2 * qh + 1) * HD + c * 64, row0 + q0);
        } else {
          tma_load_2d(sQ + c * Q_CH, &tmQ, q_full, qh * HD + c * 64, row0 + q0);
        }
      }
      const int* bt = block_table + (size_t)slot * max_blocks;
      int k_armed = 0, v_armed = 0;                           // tiles whose K / V loads were issued
      bool ok = true;
      auto tile_row = [&](int j) -> int {
        if (POOL && j < np) return pool_start[seg] + j * FT_BKV;
        const int t0 = (tile0 + j - np) * FT_BKV;
        const int blk = bt[t0 / kv_block];
        return blk < 0 ? -1 : blk * kv_block + t0 % kv_block;
      };
      auto load_k = [&](int j) -> bool {
        const int st = j % KS, krow = tile_row(j);
        if (krow < 0) { set_status(status, ST_BOUNDS); return false; }
        if (j >= KS && !mbar_wait_or_flag(&k_empty[st], ((j / KS) - 1) & 1, abort_flag)) { set_status(status, ST_MBAR_TIMEOUT); return false; }
        mbar_expect_tx(&k_full[st], K_BYTES);
        const CUtensorMap* tm = POOL && j < np ? &tmKp : &tmK;
#pragma unroll
        for (int c = 0; c < NCH; ++c) tma_load_2d(sK + st * K_BYTES + c * KV_CH, tm, &k_full[st], kvh * HD + c * 64, krow);
        k_armed = j + 1;
        return true;
      };
      auto load_v = [&](int j) -> bool {
        const int st = j % VS, krow = tile_row(j);
        if (krow < 0) { set_status(status, ST_BOUNDS); return false; }
        if (j >= VS && !mbar_wait_or_flag(&v_empty[st], ((j / VS) - 1) & 1, abort_flag)) { set_status(status, ST_MBAR_TIMEOUT); return false; }
        mbar_expect_tx(&v_full[st], V_BYTES);
        const CUtensorMap* tm = POOL && j < np ? &tmVp : &tmV;
#pragma unroll
        for (int c = 0; c < VCH; ++c) tma_load_2d(sV + st * V_BYTES + c * KV_CH, tm, &v_full[st], kvh * HV + c * 64, krow);
        v_armed = j + 1;
        return true;
      };
      ok = load_k(0);
      for (int j = 0; ok && j < nt; ++j) {
        if (j + 1 < nt) ok = load_k(j + 1);
        if (ok) ok = load_v(j);
      }
      if (!ok) *abort_p = 1;
      if (*abort_flag) {
        // loads issued by this thread may still be landing: give them a bounded time before the CTA's memory goes away
        mbar_wait(q_full, 0, 1u << 20);
        for (int j = max(0, k_armed - KS); j < k_armed; ++j) mbar_wait(&k_full[j % KS], (j / KS) & 1, 1u << 20);
        for (int j = max(0, v_armed - VS); j < v_armed; ++j) mbar_wait(&v_full[j % VS], (j / VS) & 1, 1u << 20);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      // ---- MMA issuer ---------------------------------------------------------------------------------------
      constexpr uint32_t idesc_s = umma_idesc(1, 1, FT_BQ, FT_BKV);
      constexpr uint32_t idesc_pv = umma_idesc(1, 1, FT_BQ, HV) | (1u << 16);     // B read MN-major
      const uint32_t aQ = smem_u32(sQ), aK = smem_u32(sK), aV = smem_u32(sV);
      bool ok = mbar_wait_or_flag(q_full, 0, abort_flag);
      auto issue_s = [&](int j) -> bool {
        const int s = j & 1, st = j % KS;
        if (!mbar_wait_or_flag(&k_full[st], (j / KS) & 1, abort_flag)) return false;
        if (j >= 2 && !mbar_wait_or_flag(PAIR ? &p_empty[s] : &s_empty[s], ((j >> 1) - 1) & 1, abort_flag)) return false;
        tc_fence_after();
#pragma unroll
        for (int kk = 0; kk < HD / 16; ++kk) {
          const uint32_t off = (uint32_t)(kk & 3) * 32u;
          tc_mma_f16(tmem + COL_S + s * FT_BKV, umma_desc_k128(aQ + (kk >> 2) * Q_CH + off),
                     umma_desc_k128(aK + st * K_BYTES + (kk >> 2) * KV_CH + off), idesc_s, kk > 0 ? 1u : 0u);
        }
        tc_commit(&s_full[s]);
        tc_commit(&k_empty[st]);
        return true;
      };
      if (ok) ok = issue_s(0);
      for (int j = 0; ok && j < nt; ++j) {
        const int s = j & 1, st = j % VS;
        if (j + 1 < nt && !issue_s(j + 1)) { ok = false; break; }
        if (!mbar_wait_or_flag(&p_full[s], (j >> 1) & 1, abort_flag) ||
            !mbar_wait_or_flag(&v_full[st], (j / VS) & 1, abort_flag)) { ok = false; break; }
        tc_fence_after();
#pragma unroll
        for (int kk = 0; kk < FT_BKV / 16; ++kk)
          tc_mma_f16_ts(tmem + COL_O, tmem + COL_P + s * P_STEP + kk * 8,
                        umma_desc_mn128(aV + st * V_BYTES + kk * 16 * 128, KV_CH, 1024), idesc_pv, (j > 0 || kk > 0) ? 1u : 0u);
        if (PX) {
#pragma unroll
          for (int kk = 0; kk < FT_BKV / 16; ++kk)
            tc_mma_f16_ts(tmem + COL_O, tmem + COL_P + REM + s * P_STEP + kk * 8,
                          umma_desc_mn128(aV + st * V_BYTES + kk * 16 * 128, KV_CH, 1024), idesc_pv, 1u);
        }
        tc_commit(&v_empty[st]);
        tc_commit(&p_empty[s]);
      }
      if (!ok) { set_status(status, ST_MBAR_TIMEOUT); *abort_p = 1; }
    }
  } else {
    // ---- softmax + epilogue: two threads per query row (warps 2..5 take keys 0..31 of a tile, warps 6..9 keys 32..63;
    // a row's two threads sit in the same TMEM lane quadrant) -----------------------------------------------------
    // The halves of a row exchange their tile maxima through shared memory around a named barrier of the 256 softmax
    // threads. A failed wait is published through fail_s BEFORE that barrier and acted on AFTER it, so the 256 threads
    // always leave the loop in the same iteration and nobody is left alone at the barrier.
    const int quad = warp & 3;
    const int half = (warp - 2) >> 2;
    const int row = quad * 32 + lane;
    const uint32_t lane_addr = (uint32_t)(quad * 32) << 16;
    const int qpos = pos0 + q0 + (DUAL ? row % QR : row);
    const int klo = BND ? first_key(qpos, window, chunk) : 0;
    const int klo_last = BND ? first_key(pos0 + q0 + QR - 1, window, chunk) : 0;
    constexpr int HC = FT_BKV / 2;                          // keys per thread and tile
    constexpr int OC = HV / 2;                              // O columns per thread (rescale, epilogue)
    float m_ref = -INFINITY, l = 0.f;
    bool broke = false;
    bool late_fail = false;                                 // a wait after the barrier ran out: reported at the next one
    for (int j = 0; j < nt; ++j) {
      const int s = j & 1;
      bool ok = !late_fail && mbar_wait_or_flag(&s_full[s], (j >> 1) & 1, abort_flag);
      ok = __all_sync(0xffffffffu, ok);
      uint32_t sr[HC];
      float mx = -INFINITY;
      if (ok) {
        tc_fence_after();
        tmem_ld32(tmem + lane_addr + COL_S + s * FT_BKV + half * HC, sr);
        tmem_ld_wait();
        tc_fence_before();
        if (!PAIR) {                                          // one arrival per softmax warp: its loads are done
          __syncwarp();
          if (lane == 0) mbar_arrive(&s_empty[s]);
        }
        const bool means = POOL && j < np;                    // keys of the tile are means: number t0 + c
        const int t0 = (means ? j : tile0 + j - np) * FT_BKV + half * HC;
        const bool need_mask = means || t0 + HC - 1 > pos0 + q0 || (BND && t0 < klo_last);
        const bool capped = BND && cap_log2 > 0.f;
        if (capped) {
          float am = 0.f;
          const uint64_t scale2 = f2_pack(scale_log2, scale_log2), cap2 = f2_pack(cap_log2, cap_log2);
          uint64_t x[HC / 2];
#pragma unroll
          for (int c = 0; c < HC / 2; ++c) {
            x[c] = f2_mul(f2_pack(__uint_as_float(sr[2 * c]), __uint_as_float(sr[2 * c + 1])), scale2);
            const float2 v = f2_unpack(x[c]);
            am = fmaxf(am, fmaxf(fabsf(v.x), fabsf(v.y)));
          }
          if (__any_sync(0xffffffffu, am > 1.f)) {
#pragma unroll
            for (int c = 0; c < HC / 2; ++c) {
              const float2 v = f2_unpack(x[c]);
              sr[2 * c] = __float_as_uint(cap_log2 * tanh_exp(v.x));
              sr[2 * c + 1] = __float_as_uint(cap_log2 * tanh_exp(v.y));
            }
          } else {
#pragma unroll
            for (int c = 0; c < HC / 2; ++c) {
              const float2 v = f2_unpack(f2_mul(f2_mul(x[c], cap2), f2_tanh_ratio(x[c])));
              sr[2 * c] = __float_as_uint(v.x);
              sr[2 * c + 1] = __float_as_uint(v.y);
            }
          }
        }
        if constexpr (BND) {
          if (!capped) {
#pragma unroll
            for (int c = 0; c < HC; ++c) sr[c] = __float_as_uint(__uint_as_float(sr[c]) * scale_log2);
          }
          if (means) {
#pragma unroll
            for (int c = 0; c < HC; ++c)
              if ((t0 + c + 1) * pool > klo) sr[c] = __float_as_uint(-INFINITY);
          } else if (need_mask) {
#pragma unroll
            for (int c = 0; c < HC; ++c)
              if (t0 + c > qpos || t0 + c < klo) sr[c] = __float_as_uint(-INFINITY);
          }
#pragma unroll
          for (int c = 0; c < HC; ++c) mx = fmaxf(mx, __uint_as_float(sr[c]));
        } else {
#pragma unroll
          for (int c = 0; c < HC; ++c) {
            float v = __uint_as_float(sr[c]) * scale_log2;
            if (need_mask && t0 + c > qpos) v = -INFINITY;
            sr[c] = __float_as_uint(v);
            mx = fmaxf(mx, v);
          }
        }
      } else {
        fail_s[s] = 1;
      }
      mx_s[s][half][row] = mx;
      asm volatile("bar.sync 1, 256;" ::: "memory");
      if (fail_s[s]) { broke = true; break; }
      mx = fmaxf(mx, mx_s[s][half ^ 1][row]);               // the row's maximum over the whole tile
      const bool any = __any_sync(0xffffffffu, mx > m_ref + 8.f);
      // The P buffer of this parity was last read by PV(j-2); O may only be rescaled once PV(j-1) has completed. Both
      // are phases of p_empty; neither wait sits on the common path's critical chain (PV(j-1) runs while this tile's
      // softmax does, and P(j) is handed over without waiting for it).
      ok = true;
      if (j >= 2) ok = mbar_wait_or_flag(&p_empty[s], ((j >> 1) - 1) & 1, abort_flag);
      if (ok && any && j > 0) ok = mbar_wait_or_flag(&p_empty[s ^ 1], ((j - 1) >> 1) & 1, abort_flag);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) { late_fail = true; continue; }
      tc_fence_after();
      if (any) {
        const float m_new = fmaxf(m_ref, mx);
        const float f = (m_ref == -INFINITY) ? 0.f : fast_exp2(m_ref - m_new);
        l *= f;
        if (j > 0) {
#pragma unroll 1
          for (int c0 = 0; c0 < OC; c0 += 32) {
            uint32_t o[32];
            tmem_ld32(tmem + lane_addr + COL_O + half * OC + c0, o);
            tmem_ld_wait();
#pragma unroll
            for (int c = 0; c < 32; ++c) o[c] = __float_as_uint(__uint_as_float(o[c]) * f);
            tmem_st32(tmem + lane_addr + COL_O + half * OC + c0, o);
          }
          tmem_st_wait();
        }
        m_ref = m_new;
      }
      const float mr = (m_ref == -INFINITY) ? 0.f : m_ref;
      uint32_t pr[HC / 2], px[PX ? HC / 2 : 1];
      float sum = 0.f;
      uint64_t sum2 = f2_pack(0.f, 0.f);
#pragma unroll
      for (int c = 0; c < HC / 2; ++c) {
        if constexpr (BND) {                                  // the same two keys at a time
          const float2 d = f2_unpack(f2_add(f2_pack(__uint_as_float(sr[2 * c]), __uint_as_float(sr[2 * c + 1])), f2_pack(-mr, -mr)));
          const float p0 = fast_exp2(d.x), p1 = fast_exp2(d.y);
          const uint64_t pp = f2_pack(p0, p1);
          sum2 = f2_add(sum2, pp);
          pr[c] = pack_bf2(p0, p1);
          const float2 rest = f2_unpack(f2_add(pp, f2_pack(-bf_lo(pr[c]), -bf_hi(pr[c]))));
          px[c] = pack_bf2(rest.x, rest.y);
          continue;
        }
        const float p0 = fast_exp2(__uint_as_float(sr[2 * c]) - mr);
        const float p1 = fast_exp2(__uint_as_float(sr[2 * c + 1]) - mr);
        sum += p0 + p1;
        __nv_bfloat162 h = __floats2bfloat162_rn(p0, p1);     // .x (low half) = even key
        pr[c] = *reinterpret_cast<uint32_t*>(&h);
        if constexpr (PX) px[c] = pack_bf2(p0 - bf_lo(pr[c]), p1 - bf_hi(pr[c]));
      }
      if constexpr (BND) {
        const float2 v = f2_unpack(sum2);
        sum = v.x + v.y;
      }
      l += sum;
      tmem_st16(tmem + lane_addr + COL_P + s * P_STEP + half * (HC / 2), pr);
      if constexpr (PX) tmem_st16(tmem + lane_addr + COL_P + REM + s * P_STEP + half * (HC / 2), px);
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[s]);
    }
    // final hand-over: the row sum of the other half, and agreement on whether the output is complete
    bool ok = !broke && !late_fail;
    if (ok) ok = mbar_wait_or_flag(&p_empty[(nt - 1) & 1], ((nt - 1) >> 1) & 1, abort_flag);
    ok = __all_sync(0xffffffffu, ok);
    if (!ok) fail_s[2] = 1;
    // row sums go through the maxima buffer of the parity the last tile did NOT use: nobody reads that one any more
    float (*l_s)[FT_BQ] = mx_s[nt & 1];
    l_s[half][row] = l;
    asm volatile("bar.sync 1, 256;" ::: "memory");
    if (!fail_s[2]) {
      tc_fence_after();
      float lt = l + l_s[half ^ 1][row];
      if (sink) lt += exp2f(sink[qh] * 1.4426950408889634f - m_ref);
      const float inv = lt > 0.f ? 1.f / lt : 0.f;
      if constexpr (DUAL) {
        // map 1 hands its rows over through the (now idle) key tiles; map 0 finishes them
        constexpr int LDX = HD + 4;
        const int qr = row % QR;
        float* xs = reinterpret_cast<float*>(sK) + (size_t)qr * LDX + half * OC;
        float (*ss_s)[FT_BQ] = mx_s[(nt & 1) ^ 1];            // everyone is past the last tile's maxima
        if (row >= QR) {
#pragma unroll 1
          for (int c0 = 0; c0 < OC; c0 += 32) {
            uint32_t o[32];
            tmem_ld32(tmem + lane_addr + COL_O + half * OC + c0, o);
            tmem_ld_wait();
#pragma unroll
            for (int c = 0; c < 32; c += 4)
              *reinterpret_cast<float4*>(xs + c0 + c) = make_float4(__uint_as_float(o[c]) * inv, __uint_as_float(o[c + 1]) * inv,
                                                                    __uint_as_float(o[c + 2]) * inv, __uint_as_float(o[c + 3]) * inv);
          }
        }
        asm volatile("bar.sync 1, 256;" ::: "memory");
        if (row < QR) {
          const float lam = mix.lam[0];
          float ss = 0.f;
#pragma unroll 1
          for (int c0 = 0; c0 < OC; c0 += 32) {
            uint32_t o[32];
            tmem_ld32(tmem + lane_addr + COL_O + half * OC + c0, o);
            tmem_ld_wait();
#pragma unroll
            for (int c = 0; c < 32; c += 4) {
              float4 v = *reinterpret_cast<const float4*>(xs + c0 + c);
              v.x = __uint_as_float(o[c]) * inv - lam * v.x; v.y = __uint_as_float(o[c + 1]) * inv - lam * v.y;
              v.z = __uint_as_float(o[c + 2]) * inv - lam * v.z; v.w = __uint_as_float(o[c + 3]) * inv - lam * v.w;
              ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
              *reinterpret_cast<float4*>(xs + c0 + c) = v;
            }
          }
          ss_s[half][qr] = ss;
        }
        asm volatile("bar.sync 1, 256;" ::: "memory");
        // all threads together, columns of a row side by side
        const float* xall = reinterpret_cast<const float*>(sK);
        const int rows_here = min(QR, n - q0);
        for (int i = threadIdx.x - 64; i < rows_here * (HD / 4); i += 256) {
          const int xr = i / (HD / 4), d = i % (HD / 4) * 4;
          const float r = mix.scale / sqrtf((ss_s[0][xr] + ss_s[1][xr]) / (float)mix.vdim + mix.eps);
          const size_t grow = (size_t)(row0 + q0 + xr);
          const float4 x = *reinterpret_cast<const float4*>(xall + (size_t)xr * LDX + d);
          float v[4] = {x.x * r, x.y * r, x.z * r, x.w * r};
          if (mix.gate) {
            const float* gate = mix.gate + grow * mix.ldg + (size_t)qh * mix.vdim + d;
#pragma unroll
            for (int e = 0; e < 4; ++e)
              if (d + e < mix.vdim) v[e] *= sigmoidf_(gate[e]);
          }
          *reinterpret_cast<uint2*>(out + grow * (size_t)ldo + (size_t)qh * HD + d) = make_uint2(pack_bf2(v[0], v[1]), pack_bf2(v[2], v[3]));
        }
      } else {
        const bool valid = q0 + row < n;
        const size_t grow = (size_t)(row0 + q0 + row);
        __nv_bfloat16* dst = out + grow * (size_t)ldo + (size_t)qh * HV + half * OC;
        float* dst32 = reinterpret_cast<float*>(out) + grow * (size_t)ldo + (size_t)qh * HV + half * OC;
        const __nv_bfloat16* gate = proj + grow * proj_stride + (size_t)qh * 2 * HD + HD + half * OC;
#pragma unroll 1
        for (int c0 = 0; c0 < OC; c0 += 32) {
          uint32_t o[32];
          tmem_ld32(tmem + lane_addr + COL_O + half * OC + c0, o);
          tmem_ld_wait();
          if (BND && valid && out_f32) {
#pragma unroll
            for (int v4 = 0; v4 < 8; ++v4)
              *reinterpret_cast<float4*>(dst32 + c0 + v4 * 4) =
                  make_float4(__uint_as_float(o[v4 * 4]) * inv, __uint_as_float(o[v4 * 4 + 1]) * inv, __uint_as_float(o[v4 * 4 + 2]) * inv,
                              __uint_as_float(o[v4 * 4 + 3]) * inv);
          } else if (valid) {
#pragma unroll
            for (int v4 = 0; v4 < 4; ++v4) {
              uint32_t w[4];
              uint4 g4 = make_uint4(0, 0, 0, 0);
              if (gated) g4 = *reinterpret_cast<const uint4*>(gate + c0 + v4 * 8);
              const uint32_t gu[4] = {g4.x, g4.y, g4.z, g4.w};
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                float a = __uint_as_float(o[v4 * 8 + 2 * e]) * inv, b = __uint_as_float(o[v4 * 8 + 2 * e + 1]) * inv;
                if (gated) { a *= sigmoidf_(bf_lo(gu[e])); b *= sigmoidf_(bf_hi(gu[e])); }
                __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
                w[e] = *reinterpret_cast<uint32_t*>(&h);
              }
              *reinterpret_cast<uint4*>(dst + c0 + v4 * 8) = make_uint4(w[0], w[1], w[2], w[3]);
            }
          }
        }
      }
    } else if (threadIdx.x == 64) {
      set_status(status, ST_MBAR_TIMEOUT);
      *abort_p = 1;
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem, TMEM_COLS);
}

}  // namespace fb

using namespace fb;

// q: [q_rows][nq*hd] bf16 (post norm / RoPE); caches: [cache_rows = blocks*kv_block] rows of nkv*hd bf16, kv_stride elements
// apart (0: dense); scale: of the scores (0: 1 / sqrt(hd)); exact_p: softmax weights as value + remainder; sink: a number per q head
// that joins the softmax denominator, or null; hdv: columns of a head's values (0: hd; 128 beside 192 of the keys); pool: gathered means of the
// blocks before the window, or null; kb: window, chunk and softcap, or null (only with exact_p and a bounded call: fp32 rows,
// out_f32); mix: what follows two maps per head (nq counts both maps' queries, out has nq / 2 heads), or null; ldo: elements between rows of out (0: dense); same outputs as fb_attn_prefill. Returns -20 when the shape is outside what this kernel takes (the caller uses fb_attn_prefill).
extern "C" int fb_attn_prefill_tc(void* out, const void* q, const void* k_cache, const void* v_cache, const void* proj,
                                  long proj_stride, const int* seg_slot, const int* seg_row0, const int* seg_nrows,
                                  const int* seg_pos0, const int* block_table, int max_blocks, int kv_block, int nseg,
                                  int max_rows, long q_rows, long cache_rows, int nq, int nkv, int hd, int hdv, int gated,
                                  float scale, int exact_p, long kv_stride, const float* sink, const KeyBounds* kb, const PoolKeys* pool,
                                  long ldo, int out_f32, const HeadMix* mix, int* status, cudaStream_t s) {
  if (nseg <= 0 || max_rows <= 0) return 0;
  if (nq % nkv) return -1;
  if (hdv == 0) hdv = hd;
  const bool wide = hd == 192 && hdv == 128;
  if ((!wide && ((hd != 64 && hd != 128 && hd != 256) || hdv != hd)) || kv_block % FT_BKV) return -20;
  if (kv_stride == 0) kv_stride = wide ? -1 : (long)nkv * hd;          // keys and values of different widths lie in one buffer
  if (kv_stride < 0 || (wide && (mix || pool || gated || out_f32 || sink || !exact_p))) return -20;
  if (pool && (pool->size < 1 || !pool->start || pool->rows < 0 || !kb || !kb->window || mix || out_f32)) return -1;
  if (kv_stride % 8) return -20;
  const int heads = mix ? nq / 2 : nq, q_rows_cta = mix ? FT_BQ / 2 : FT_BQ;
  CUtensorMap tmQ, tmK, tmV, tmKp, tmVp;
  int rc;
  if ((rc = make_tmap_bf16_2d(&tmQ, q, (uint64_t)q_rows, (uint64_t)nq * hd, (uint64_t)nq * hd, q_rows_cta))) return rc;
  if ((rc = make_tmap_bf16_2d(&tmK, k_cache, (uint64_t)cache_rows, (uint64_t)nkv * hd, (uint64_t)kv_stride, FT_BKV))) return rc;
  if ((rc = make_tmap_bf16_2d(&tmV, v_cache, (uint64_t)cache_rows, (uint64_t)nkv * hdv, (uint64_t)kv_stride, FT_BKV))) return rc;
  tmKp = tmK; tmVp = tmV;
  if (pool && pool->rows > 0) {
    if ((rc = make_tmap_bf16_2d(&tmKp, pool->k, (uint64_t)pool->rows, (uint64_t)nkv * hd, (uint64_t)nkv * hd, FT_BKV))) return rc;
    if ((rc = make_tmap_bf16_2d(&tmVp, pool->v, (uint64_t)pool->rows, (uint64_t)nkv * hd, (uint64_t)nkv * hd, FT_BKV))) return rc;
  }
  // up to four waves of CTAs are one group; more go in groups of about two waves, whole sets of query heads that share keys
  const int q_tiles = (max_rows + q_rows_cta - 1) / q_rows_cta, share = heads / nkv > 0 ? heads / nkv : 1;
  const int slots = 148 * (ft_pair(hd, kb || out_f32 || mix) ? 2 : 1);
  const int few = (2 * slots / q_tiles + share) / share * share;
  const int group = (long)heads * q_tiles <= 4 * slots || few > heads ? heads : few, head_groups = (heads + group - 1) / group;
  dim3 grid(group, q_tiles, nseg * head_groups);
  const HeadMix no_mix{};
  if ((kb || out_f32 || mix) && (!exact_p || gated)) return -20;
  if (mix && (nq % 2 || (nq / nkv) % 2 || !mix->lam || mix->vdim < 1 || mix->vdim > hd || sink || out_f32)) return -1;
  if (kb && (kb->window < 0 || kb->chunk < 0 || (kb->window && kb->chunk) || kb->cap < 0.f)) return -1;
  if (ldo == 0) ldo = (long)heads * hdv;
  if (ldo % 8) return -20;
  constexpr float LOG2E = 1.4426950408889634f;
  const float cap = kb ? kb->cap : 0.f, raw_scale = scale != 0.f ? scale : 1.f / sqrtf((float)hd);
  const float scale_log2 = cap > 0.f ? raw_scale / cap : raw_scale * LOG2E;
#define FB_FT(HDK, HVV, PXV, BNDV, DUALV, POOLV)                                                                   \
  {                                                                                                                \
    const size_t smem = (size_t)(FT_BQ + ft_k_stages(HDK, BNDV) * FT_BKV) * HDK * 2 +                              \
                        (size_t)ft_v_stages(HDK, BNDV) * FT_BKV * HVV * 2 + 2048 + 512;                            \
    auto kern = attn_prefill_tc_kernel<HDK, HVV, PXV, BNDV, DUALV, POOLV>;                                         \
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);            \
    if (e != cudaSuccess) return (int)e;                                                                           \
    launch_pdl(kern, grid, dim3(FT_THREADS), smem, s, tmQ, tmK, tmV, tmKp, tmVp, pool ? pool->start : nullptr, pool ? pool->size : 1, (__nv_bfloat16*)out, (const __nv_bfloat16*)proj, \
               proj_stride, seg_slot, seg_row0, seg_nrows, seg_pos0, block_table, max_blocks, kv_block, nq, nkv,   \
               gated, scale_log2, sink, kb ? kb->window : 0, kb ? kb->chunk : 0, cap * LOG2E, ldo, out_f32, mix ? *mix : no_mix, head_groups, status);                                                                   \
  }
  if (wide) {
    FB_FT(192, 128, true, true, false, false)
  } else if (pool) {
    if (hd == 256) FB_FT(256, 256, true, true, false, true) else if (hd == 128) FB_FT(128, 128, true, true, false, true)
    else FB_FT(64, 64, true, true, false, true)
  } else if (mix) {
    if (hd == 256) FB_FT(256, 256, true, true, true, false) else if (hd == 128) FB_FT(128, 128, true, true, true, false)
    else FB_FT(64, 64, true, true, true, false)
  } else if (kb || out_f32) {
    if (hd == 256) FB_FT(256, 256, true, true, false, false) else if (hd == 128) FB_FT(128, 128, true, true, false, false)
    else FB_FT(64, 64, true, true, false, false)
  } else if (exact_p) {
    if (hd == 256) FB_FT(256, 256, true, false, false, false) else if (hd == 128) FB_FT(128, 128, true, false, false, false)
    else FB_FT(64, 64, true, false, false, false)
  } else {
    if (hd == 256) FB_FT(256, 256, false, false, false, false) else if (hd == 128) FB_FT(128, 128, false, false, false, false)
    else FB_FT(64, 64, false, false, false, false)
  }
#undef FB_FT
  return (int)cudaGetLastError();
}
