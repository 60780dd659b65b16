// Python bindings, third part: convolved operands, pooled blocks, rotated latents and state-space layers of the models of listed layers. The
// element type of activations, caches and tails (bf16 / fp32) is read off the tensors.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAStream.h>
#include <torch/extension.h>

#include <vector>

#include "api_listed.h"

namespace {

using torch::Tensor;
using OptTensor = c10::optional<Tensor>;

inline cudaStream_t cur_stream() { return c10::cuda::getCurrentCUDAStream().stream(); }
inline void check(int rc, const char* what) {
  if (rc == 0) return;
  if (rc > 0) TORCH_CHECK(false, what, ": CUDA error ", rc, " (", cudaGetErrorString((cudaError_t)rc), ")");
  TORCH_CHECK(false, what, ": unsupported arguments (code ", rc, ")");
}
inline bool f32(const Tensor& t) { return t.scalar_type() == torch::kFloat32; }
inline bool f32v(const OptTensor& t, int64_t n) { return !t || (f32(*t) && t->is_contiguous() && t->numel() == n); }
template <typename T>
inline T* ptr(const OptTensor& t) { return t ? reinterpret_cast<T*>(t->data_ptr()) : nullptr; }
inline bool same_type(const Tensor& a, const OptTensor& b) { return !b || a.scalar_type() == b->scalar_type(); }

// tails [slots, taps - 1, C]: rows of C side by side, slots any distance apart
void check_tails(const Tensor& t, int64_t taps, int64_t C, const char* what) {
  TORCH_CHECK(t.dim() == 3 && t.size(1) == taps - 1 && (taps == 1 || (t.size(2) == C && t.stride(2) == 1 && t.stride(1) == C)), what, ": tails");
}

// xs: results of the layers [layers + 1, rows, W]; conv: weights [taps, W]; xb is written when conv is given
void add_conv_normed(Tensor x_in, Tensor x, OptTensor y, OptTensor yp, OptTensor wts, OptTensor w, OptTensor xs, int64_t place, OptTensor dwa,
                     OptTensor next_w, OptTensor h_out, OptTensor xb, OptTensor conv, OptTensor tails, OptTensor row_slot, bool commit, int64_t width,
                     double eps, bool is_f32) {
  const int64_t rows = x.size(0), W = x.size(1);
  TORCH_CHECK(x.is_contiguous() && f32(x) && x_in.is_contiguous() && f32(x_in) && x_in.sizes() == x.sizes() && width <= W &&
              (!y || (f32(*y) && y->stride(1) == 1 && y->sizes() == x.sizes())) && f32v(w, W) && f32v(next_w, W), "add_conv_normed: rows");
  const int top = wts ? (int)wts->size(1) : 0;
  TORCH_CHECK(yp.has_value() == wts.has_value() && (!yp || (yp->is_contiguous() && wts->is_contiguous() && f32(*yp) && f32(*wts) &&
              wts->size(0) == rows && yp->size(0) == rows * top && yp->size(1) == W)), "add_conv_normed: expert rows");
  TORCH_CHECK(!xs || (f32(*xs) && xs->is_contiguous() && xs->dim() == 3 && xs->size(0) > place && xs->size(1) == rows && xs->size(2) == W && dwa &&
              f32(*dwa) && dwa->is_contiguous() && dwa->numel() == place + 1), "add_conv_normed: results");
  auto operand = [&](const OptTensor& t) { return !t || (t->is_contiguous() && t->sizes() == x.sizes() && f32(*t) == is_f32); };
  TORCH_CHECK(operand(h_out) && operand(xb) && (!xb || (conv && tails && row_slot)), "add_conv_normed: operands");
  int taps = 1;
  if (xb) {
    taps = (int)conv->size(0);
    TORCH_CHECK(f32(*conv) && conv->is_contiguous() && conv->size(1) == W && f32(*tails) == is_f32 && row_slot->numel() == rows, "add_conv_normed: convolution");
    check_tails(*tails, taps, W, "add_conv_normed");
  }
  check(fb_add_conv_normed(x_in.data_ptr<float>(), x.data_ptr<float>(), ptr<float>(y), y ? (long)y->stride(0) : 0, ptr<float>(yp), ptr<float>(wts),
                           top, ptr<float>(w), ptr<float>(xs), xs ? (long)xs->stride(0) : 0, (int)place, ptr<float>(dwa), ptr<float>(next_w),
                           ptr<void>(h_out), ptr<void>(xb), ptr<float>(conv), taps, xb ? ptr<void>(tails) : nullptr, xb ? (long)tails->stride(0) : 0,
                           xb ? ptr<int>(row_slot) : nullptr, commit ? 1 : 0, (int)rows, (int)width, (int)W, (float)eps, is_f32 ? 1 : 0,
                           cur_stream()), "add_conv_normed");
}

void conv_rows(Tensor out, Tensor x, Tensor w, Tensor tails, Tensor row_slot, Tensor row_pos, OptTensor bias, bool silu, bool residual) {
  const int64_t C = x.size(1), taps = w.size(0);
  TORCH_CHECK(out.sizes() == x.sizes() && out.stride(1) == 1 && x.stride(1) == 1 && out.scalar_type() == x.scalar_type() &&
              tails.scalar_type() == x.scalar_type() && f32(w) && w.is_contiguous() && w.size(1) == C && f32v(bias, C) &&
              row_slot.numel() == x.size(0) && row_pos.numel() == x.size(0), "conv_rows: layouts");
  check_tails(tails, taps, C, "conv_rows");
  check(fb_conv_rows(out.data_ptr(), (long)out.stride(0), x.data_ptr(), (long)x.stride(0), w.data_ptr<float>(), (int)taps, (int)C, tails.data_ptr(),
                     (long)tails.stride(0), row_slot.data_ptr<int>(), row_pos.data_ptr<int>(), ptr<float>(bias), silu, residual, (int)x.size(0),
                     f32(x), cur_stream()), "conv_rows");
}

void conv_tail(Tensor tails, Tensor x, Tensor seg_slot, Tensor seg_row0, Tensor seg_nrows) {
  const int64_t C = x.size(1), taps = tails.size(1) + 1;
  TORCH_CHECK(x.stride(1) == 1 && tails.scalar_type() == x.scalar_type(), "conv_tail: layouts");
  check_tails(tails, taps, C, "conv_tail");
  check(fb_conv_tail(tails.data_ptr(), (long)tails.stride(0), (int)taps, x.data_ptr(), (long)x.stride(0), (int)C, seg_slot.data_ptr<int>(),
                     seg_row0.data_ptr<int>(), seg_nrows.data_ptr<int>(), (int)seg_slot.numel(), f32(x), cur_stream()), "conv_tail");
}

// sizes: heads, groups, state, vdim, taps
struct SsmArgs { int heads, groups, N, V, taps, inner, ch; };
SsmArgs ssm_args(const std::vector<int64_t>& v, const Tensor& proj, const Tensor& rec, const Tensor& A, const Tensor& dt_bias, const Tensor& skip) {
  TORCH_CHECK(v.size() == 5, "ssm: five sizes");
  SsmArgs a{(int)v[0], (int)v[1], (int)v[2], (int)v[3], (int)v[4], 0, 0};
  a.inner = a.heads * a.V;
  a.ch = a.inner + 2 * a.groups * a.N;
  TORCH_CHECK(proj.stride(1) == 1 && proj.size(1) >= a.inner + a.ch + a.heads && rec.is_contiguous() && f32(rec) && rec.size(1) == a.heads &&
              rec.size(2) == a.N && rec.size(3) == a.V && f32v(A, a.heads) && f32v(dt_bias, a.heads) && f32v(skip, a.heads), "ssm: layouts");
  return a;
}

int64_t ssm_step(Tensor y, Tensor rec, Tensor tails, Tensor proj, Tensor conv_w, Tensor conv_b, Tensor A, Tensor dt_bias, Tensor skip,
                 Tensor seg_slot, Tensor seg_row0, Tensor seg_nrows, std::vector<int64_t> sizes, bool commit) {
  const SsmArgs a = ssm_args(sizes, proj, rec, A, dt_bias, skip);
  TORCH_CHECK(f32(y) && y.stride(1) == 1 && y.size(1) == a.inner && y.size(0) == proj.size(0) && f32v(conv_w, (int64_t)a.taps * a.ch) &&
              f32v(conv_b, a.ch) && tails.scalar_type() == proj.scalar_type(), "ssm_step: layouts");
  check_tails(tails, a.taps, a.ch, "ssm_step");
  const int rc = fb_ssm_step(y.data_ptr<float>(), (long)y.stride(0), rec.data_ptr<float>(), tails.data_ptr(), (long)tails.stride(0), proj.data_ptr(),
                             (long)proj.stride(0), conv_w.data_ptr<float>(), conv_b.data_ptr<float>(), A.data_ptr<float>(), dt_bias.data_ptr<float>(),
                             skip.data_ptr<float>(), seg_slot.data_ptr<int>(), seg_row0.data_ptr<int>(), seg_nrows.data_ptr<int>(),
                             (int)seg_slot.numel(), a.heads, a.groups, a.N, a.V, a.taps, commit ? 1 : 0, f32(proj), cur_stream());
  check(rc, "ssm_step");
  return 0;
}

int64_t ssd_chunk_scratch_bytes(int64_t rows, int64_t nseg, int64_t max_rows, int64_t heads, int64_t N, int64_t V) {
  return fb_ssd_chunk_scratch_bytes((int)rows, (int)nseg, (int)max_rows, (int)heads, (int)N, (int)V);
}

// xbc: convolved rows of the step. Returns -20 for states the kernel does not take (the caller runs ssm_step).
int64_t ssd_chunk(Tensor y, Tensor rec, Tensor scratch, Tensor xbc, Tensor proj, Tensor A, Tensor dt_bias, Tensor skip, Tensor seg_slot,
                  Tensor seg_row0, Tensor seg_nrows, int64_t max_rows, std::vector<int64_t> sizes) {
  const SsmArgs a = ssm_args(sizes, proj, rec, A, dt_bias, skip);
  const int rows = (int)proj.size(0);
  TORCH_CHECK(f32(y) && y.stride(1) == 1 && y.size(1) == a.inner && y.size(0) == rows && !f32(proj) && xbc.is_contiguous() &&
              xbc.scalar_type() == proj.scalar_type() && xbc.size(0) == rows && xbc.size(1) == a.ch && scratch.is_contiguous() &&
              scratch.numel() * scratch.element_size() >= fb_ssd_chunk_scratch_bytes(rows, (int)seg_slot.numel(), (int)max_rows, a.heads, a.N, a.V),
              "ssd_chunk: layouts");
  const int rc = fb_ssd_chunk(y.data_ptr<float>(), (long)y.stride(0), rec.data_ptr<float>(), scratch.data_ptr(), xbc.data_ptr(), proj.data_ptr(),
                              (long)proj.stride(0), A.data_ptr<float>(), dt_bias.data_ptr<float>(), skip.data_ptr<float>(), seg_slot.data_ptr<int>(),
                              seg_row0.data_ptr<int>(), seg_nrows.data_ptr<int>(), (int)seg_slot.numel(), (int)max_rows, rows, a.heads, a.groups, a.N,
                              a.V, cur_stream());
  if (rc == -20) return rc;
  check(rc, "ssd_chunk");
  return 0;
}

// proj [rows, >= inner + ch]; tails: every row joins its slot's tail (one row per segment)
void group_norm_gated(Tensor out, Tensor y, Tensor proj, Tensor w, int64_t parts, double eps, OptTensor tails, OptTensor row_slot) {
  const int64_t inner = y.size(1), rows = y.size(0);
  TORCH_CHECK(out.stride(1) == 1 && f32(y) && y.stride(1) == 1 && proj.stride(1) == 1 && out.scalar_type() == proj.scalar_type() &&
              out.size(0) == rows && proj.size(0) == rows && out.size(1) >= inner && f32v(w, inner) && tails.has_value() == row_slot.has_value(),
              "group_norm_gated: layouts");
  int taps = 0, ch = 0;
  if (tails) {
    taps = (int)tails->size(1) + 1; ch = (int)tails->size(2);
    check_tails(*tails, taps, ch, "group_norm_gated");
    TORCH_CHECK(tails->scalar_type() == proj.scalar_type() && proj.size(1) >= inner + ch && row_slot->numel() == rows, "group_norm_gated: tails");
  }
  check(fb_group_norm_gated(out.data_ptr(), (long)out.stride(0), y.data_ptr<float>(), (long)y.stride(0), proj.data_ptr(), (long)proj.stride(0),
                            w.data_ptr<float>(), (int)rows, (int)inner, (int)parts, (int)out.size(1), (float)eps, ptr<void>(tails),
                            tails ? (long)tails->stride(0) : 0, taps, ch, ptr<int>(row_slot), f32(out), cur_stream()), "group_norm_gated");
}

void check_means(const Tensor& m, const Tensor& cache, int64_t kv_block, int64_t pool, const char* what) {
  TORCH_CHECK(m.is_contiguous() && cache.is_contiguous() && m.scalar_type() == cache.scalar_type() && m.dim() == 4 && m.size(0) == cache.size(0) &&
              m.size(1) == (kv_block + pool - 1) / pool && m.size(2) == cache.size(2) && m.size(3) == cache.size(3), what, ": means");
}

void pool_keys(Tensor k_mean, Tensor v_mean, Tensor k_cache, Tensor v_cache, Tensor seg_slot, Tensor seg_pos0, Tensor seg_nrows, int64_t max_rows,
               Tensor block_table, int64_t kv_block, int64_t pool, Tensor status) {
  check_means(k_mean, k_cache, kv_block, pool, "pool_keys");
  check_means(v_mean, v_cache, kv_block, pool, "pool_keys");
  check(fb_pool_keys(k_mean.data_ptr(), v_mean.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), seg_slot.data_ptr<int>(),
                     seg_pos0.data_ptr<int>(), seg_nrows.data_ptr<int>(), (int)seg_slot.numel(), (int)max_rows, block_table.data_ptr<int>(),
                     (int)block_table.size(1), (int)kv_block, (int)k_cache.size(2), (int)k_cache.size(3), (int)pool, f32(k_cache),
                     status.data_ptr<int>(), cur_stream()), "pool_keys");
}

void pool_gather(Tensor k_out, Tensor v_out, Tensor k_mean, Tensor v_mean, Tensor seg_slot, Tensor start, Tensor count, Tensor block_table,
                 int64_t kv_block, int64_t pool, Tensor status) {
  const int64_t width = k_mean.size(2) * k_mean.size(3);
  TORCH_CHECK(k_out.is_contiguous() && v_out.is_contiguous() && k_mean.is_contiguous() && v_mean.is_contiguous() && !f32(k_mean) &&
              k_out.scalar_type() == k_mean.scalar_type() && v_out.scalar_type() == k_mean.scalar_type() && k_out.sizes() == v_out.sizes() &&
              k_out.numel() == k_out.size(0) * width && start.numel() >= seg_slot.numel() && count.numel() >= seg_slot.numel(), "pool_gather: layouts");
  check(fb_pool_gather(k_out.data_ptr(), v_out.data_ptr(), k_mean.data_ptr(), v_mean.data_ptr(), seg_slot.data_ptr<int>(), start.data_ptr<int>(),
                       count.data_ptr<int>(), (int)seg_slot.numel(), (int)k_out.size(0), block_table.data_ptr<int>(), (int)block_table.size(1),
                       (int)kv_block, (int)width, (int)pool, status.data_ptr<int>(), cur_stream()), "pool_gather");
}

void latent_rot_prep(Tensor q, Tensor cache, Tensor proj, Tensor kv_norm, Tensor inv_freq, Tensor row_slot, Tensor row_pos, Tensor block_table,
                     int64_t kv_block, int64_t dim, int64_t rot, int64_t kv_rank, double eps, Tensor status) {
  const int64_t heads = q.size(1), hp = q.size(2), lat = cache.size(-1);
  TORCH_CHECK(q.is_contiguous() && cache.is_contiguous() && q.scalar_type() == cache.scalar_type() && cache.size(1) == kv_block && f32(proj) &&
              proj.stride(1) == 1 && proj.size(0) == q.size(0) && proj.size(1) >= heads * (dim + rot) + kv_rank + rot && f32(kv_norm) &&
              kv_norm.numel() >= kv_rank && inv_freq.scalar_type() == torch::kFloat64 && inv_freq.numel() * 2 >= rot, "latent_rot_prep: layouts");
  check(fb_latent_rot_prep(q.data_ptr(), cache.data_ptr(), proj.data_ptr<float>(), (long)proj.stride(0), kv_norm.data_ptr<float>(),
                           inv_freq.data_ptr<double>(), row_slot.data_ptr<int>(), row_pos.data_ptr<int>(), block_table.data_ptr<int>(),
                           (int)block_table.size(1), (int)kv_block, (int)q.size(0), (int)heads, (int)dim, (int)rot, (int)hp, (int)kv_rank, (int)lat,
                           (float)eps, f32(q), status.data_ptr<int>(), cur_stream()), "latent_rot_prep");
}

// y [M, N] = clamped gated units of x w^T, w [2 N, K] = gate rows, up rows (bf16)
void gemm_glu(Tensor Y, Tensor X, Tensor W, double limit, int64_t split_k, OptTensor workspace, OptTensor counters, Tensor status) {
  const int M = (int)X.size(0), K = (int)X.size(1), N = (int)W.size(0) / 2;
  TORCH_CHECK(!f32(X) && X.stride(1) == 1 && W.is_contiguous() && Y.size(0) == M && Y.size(1) == N && Y.stride(1) == 1 && W.size(1) == K, "gemm_glu: layouts");
  check(fb_gemm_bf16_glu(Y.data_ptr(), X.data_ptr(), W.data_ptr(), nullptr, M, N, K, (long)X.stride(0), (long)Y.stride(0), 1, (float)limit,
                         (int)split_k, ptr<float>(workspace), ptr<int>(counters), status.data_ptr<int>(),
                         at::cuda::getCurrentDeviceProperties()->multiProcessorCount, cur_stream()), "gemm_glu");
}

}  // namespace

void register_listed(pybind11::module_& m) {
  m.def("add_conv_normed", &add_conv_normed);
  m.def("conv_rows", &conv_rows);
  m.def("conv_tail", &conv_tail);
  m.def("ssm_step", &ssm_step);
  m.def("ssd_chunk", &ssd_chunk);
  m.def("ssd_chunk_scratch_bytes", &ssd_chunk_scratch_bytes);
  m.def("group_norm_gated", &group_norm_gated);
  m.def("pool_keys", &pool_keys);
  m.def("pool_gather", &pool_gather);
  m.def("latent_rot_prep", &latent_rot_prep);
  m.def("gemm_glu", &gemm_glu);
}
