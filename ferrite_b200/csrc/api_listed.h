// C launch API, third part: convolved operands, pooled blocks, rotated latents and state-space layers of the models of listed layers.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#include "api.h"

#ifdef __cplusplus
extern "C" {
#endif

// ---- conv_rows.cu ----
int fb_add_conv_normed(const float* x_in, float* x, const float* y, long ldy, const float* yp, const float* wts, int top, const float* w, float* xs,
                       long xs_step, int place, const float* dwa, const float* next_w, void* h_out, void* xb, const float* cw, int taps, void* tails,
                       long tail_step, const int* row_slot, int commit, int rows, int width, int ld, float eps, int f32, cudaStream_t s);
int fb_conv_rows(void* out, long ldo, const void* x, long ldx, const float* w, int taps, int C, const void* tails, long tail_step,
                 const int* row_slot, const int* row_pos, const float* bias, int silu, int residual, int rows, int f32, cudaStream_t s);
int fb_conv_tail(void* tails, long tail_step, int taps, const void* x, long ldx, int C, const int* seg_slot, const int* seg_row0,
                 const int* seg_nrows, int nseg, int f32, cudaStream_t s);

// ---- ssm.cu, ssm_chunk.cu ----
int fb_ssm_step(float* y, long ldy, float* rec, const void* tails, long tail_step, const void* proj, long ldp, const float* conv_w,
                const float* conv_b, const float* A, const float* dt_bias, const float* skip, const int* seg_slot, const int* seg_row0,
                const int* seg_nrows, int nseg, int heads, int groups, int N, int V, int taps, int commit, int f32, cudaStream_t s);
int fb_group_norm_gated(void* out, long ldo, const float* y, long ldy, const void* proj, long ldp, const float* w, int rows, int inner, int parts,
                        int ko, float eps, void* tails, long tail_step, int taps, int ch, const int* row_slot, int f32, cudaStream_t s);
long fb_ssd_chunk_scratch_bytes(int rows, int nseg, int max_rows, int heads, int N, int V);
int fb_ssd_chunk(float* y, long ldy, float* rec, void* scratch, const void* xbc, const void* proj, long ldp, const float* A, const float* dt_bias,
                 const float* skip, const int* seg_slot, const int* seg_row0, const int* seg_nrows, int nseg, int max_rows, int rows, int heads,
                 int groups, int N, int V, cudaStream_t s);

// ---- gqa.cu ----
int fb_pool_keys(void* k_mean, void* v_mean, const void* k_cache, const void* v_cache, const int* seg_slot, const int* seg_pos0,
                 const int* seg_nrows, int nseg, int max_rows, const int* block_table, int max_blocks, int kv_block, int kv_heads, int hp, int pool,
                 int f32, int* status, cudaStream_t s);
int fb_pool_gather(void* k_out, void* v_out, const void* k_mean, const void* v_mean, const int* seg_slot, const int* start, const int* count,
                   int nseg, int rows, const int* block_table, int max_blocks, int kv_block, int width, int pool, int* status, cudaStream_t s);

// ---- latent.cu ----
int fb_latent_rot_prep(void* q_out, void* cache, const float* proj, long ldp, const float* kv_norm, const double* inv_freq, const int* row_slot,
                       const int* row_pos, const int* block_table, int max_blocks, int kv_block, int rows, int heads, int dim, int rot, int hp,
                       int kv_rank, int lat, float eps, int f32, int* status, cudaStream_t s);

#ifdef __cplusplus
}
#endif
