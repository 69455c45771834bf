// extern "C" entry points: host-side argument validation, then dispatch to the launchers.
// Nothing here allocates device memory.  The launches are asynchronous; the one call that waits for the device
// is based_read_status (a blocking copy of the status words).
#include "common.cuh"

using namespace based;

namespace {

bool dtype_ok(int dt) { return dt == BASED_F32 || dt == BASED_BF16; }
size_t dtype_size(int dt) { return dt == BASED_F32 ? 4 : 2; }
Strides3 s3(const int64_t* s) { return Strides3{s[0], s[1], s[2]}; }       // given as (batch, head, seq)
Strides3 s3_blh(const int64_t* s) { return Strides3{s[0], s[2], s[1]}; }   // given as (batch, seq, head)
Strides2 s2(const int64_t* s) { return Strides2{s[0], s[1]}; }

}  // namespace

extern "C" {

int based_b200_version(void) { return 1; }

const char* based_error_string(int code) {
  switch (code) {
    case BASED_OK: return "ok";
    case BASED_ERR_NULL: return "a required pointer is NULL";
    case BASED_ERR_SHAPE: return "unsupported shape";
    case BASED_ERR_DTYPE: return "unsupported dtype";
    case BASED_ERR_ALIGN: return "pointer or stride not aligned as required";
    case BASED_ERR_IMPL: return "requested implementation cannot run these arguments";
    case BASED_ERR_TOO_LARGE: return "size exceeds a fixed capacity";
    case BASED_ERR_SCRATCH: return "workspace is NULL, misaligned or too small";
    default: break;
  }
  if (code > 0) return cudaGetErrorString(static_cast<cudaError_t>(code));
  return "unknown error";
}

int based_read_status(unsigned int* out, int reset) {
  unsigned int a = 0, b = 0, c = 0, d = 0, e = 0, f = 0, g = 0, h = 0, i = 0;
  int rc = read_tc_status ? read_tc_status(&a, reset) : 0;
  if (rc == 0 && read_tc_status_swa) rc = read_tc_status_swa(&b, reset);
  if (rc == 0 && read_tp_status) rc = read_tp_status(&c, reset);
  if (rc == 0 && read_tc_status_latent) rc = read_tc_status_latent(&d, reset);
  if (rc == 0 && read_tc_status_delta) rc = read_tc_status_delta(&e, reset);
  if (rc == 0 && read_tc_status_rglru) rc = read_tc_status_rglru(&f, reset);
  if (rc == 0 && read_tc_status_tied) rc = read_tc_status_tied(&g, reset);
  if (rc == 0 && read_tc_status_lightning) rc = read_tc_status_lightning(&h, reset);
  if (rc == 0 && read_tc_status_tied_decode) rc = read_tc_status_tied_decode(&i, reset);
  if (out) *out = a | b | c | d | e | f | g | h | i;
  return rc;
}

}  // extern "C"

namespace {

// Checks shared by the whole-sequence entry points.  Returns kDone when the call is already complete
// (nothing to compute), 0 to go on, a negative code to reject.
constexpr int kDone = 0x40000000;  // not a cudaError_t value
int prefill_preamble(const void* q, const void* k, const void* v, void* y, void* kv_state, void* k_state, int B,
                     int H, int L, int d, int dv, const int64_t* q_strides, const int64_t* k_strides,
                     const int64_t* v_strides, const int64_t* y_strides, int io_dtype, int state_dtype,
                     cudaStream_t st) {
  if (!q || !k || !v || !y || !q_strides || !k_strides || !v_strides || !y_strides) return BASED_ERR_NULL;
  if ((kv_state == nullptr) != (k_state == nullptr)) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype) || !dtype_ok(state_dtype)) return BASED_ERR_DTYPE;
  if (B < 0 || H < 0 || L < 0 || d != kFeatureDim || dv < 16 || dv > 128 || dv % 16 != 0) return BASED_ERR_SHAPE;
  if ((int64_t)B * H > 2147483647LL) return BASED_ERR_TOO_LARGE;
  if (B == 0 || H == 0) return kDone;
  if (L == 0) {
    // empty sequence: the states are the empty sums
    if (kv_state) {
      const size_t es = dtype_size(state_dtype);
      cudaError_t e = cudaMemsetAsync(kv_state, 0, (size_t)B * H * dv * kExpandedDim * es, st);
      if (e == cudaSuccess) e = cudaMemsetAsync(k_state, 0, (size_t)B * H * kExpandedDim * es, st);
      return e == cudaSuccess ? kDone : (int)e;
    }
    return kDone;
  }
  return 0;
}

}  // namespace

extern "C" {

int based_linattn_prefill(const void* q, const void* k, const void* v, void* y, void* kv_state, void* k_state,
                          int B, int H, int L, int d, int dv, const int64_t q_strides[3],
                          const int64_t k_strides[3], const int64_t v_strides[3], const int64_t y_strides[3],
                          int io_dtype, int state_dtype, float eps, int impl, void* stream) {
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int pre = prefill_preamble(q, k, v, y, kv_state, k_state, B, H, L, d, dv, q_strides, k_strides, v_strides,
                                   y_strides, io_dtype, state_dtype, st);
  if (pre != 0) return pre == kDone ? BASED_OK : pre;
  // AUTO: the tensor-core kernel when it accepts the arguments (bf16 I/O, its alignment
  // rules), else the CUDA-core kernel.  Both are GPU kernels; there is no host path.
  const bool autosel = impl == BASED_IMPL_AUTO;
  if (autosel) impl = (io_dtype == BASED_BF16) ? BASED_IMPL_TCGEN05 : BASED_IMPL_SIMT;
  if (impl == BASED_IMPL_TCGEN05) {
    if (io_dtype != BASED_BF16) return BASED_ERR_IMPL;
    if (!launch_linattn_prefill_tc) return BASED_ERR_IMPL;
    const int rc = launch_linattn_prefill_tc(q, k, v, y, kv_state, k_state, B, H, L, dv, s3(q_strides),
                                             s3(k_strides), s3(v_strides), s3(y_strides), state_dtype, eps, 1,
                                             nullptr, 0, st);
    if (!(autosel && rc == BASED_ERR_IMPL)) return rc;
    impl = BASED_IMPL_SIMT;
  }
  if (impl != BASED_IMPL_SIMT) return BASED_ERR_IMPL;
  if (!launch_linattn_prefill_simt) return BASED_ERR_IMPL;
  return launch_linattn_prefill_simt(q, k, v, y, kv_state, k_state, B, H, L, dv, s3(q_strides), s3(k_strides),
                                     s3(v_strides), s3(y_strides), io_dtype, state_dtype, eps, st);
}

int based_linattn_prefill_segments(int B, int H, int L) {
  if (B <= 0 || H <= 0 || L <= 0) return 1;
  if (!linattn_prefill_tc_auto_segments) return 1;
  return linattn_prefill_tc_auto_segments(B, H, L);
}

size_t based_linattn_prefill_scratch_bytes(int B, int H, int L, int dv, int nseg) {
  if (B <= 0 || H <= 0 || L <= 0 || dv <= 0 || nseg <= 1) return 0;
  if (!linattn_prefill_tc_scratch_bytes) return 0;
  return linattn_prefill_tc_scratch_bytes(B, H, L, dv, nseg);
}

int based_linattn_prefill_split(const void* q, const void* k, const void* v, void* y, void* kv_state,
                                void* k_state, int B, int H, int L, int d, int dv, const int64_t q_strides[3],
                                const int64_t k_strides[3], const int64_t v_strides[3],
                                const int64_t y_strides[3], int state_dtype, float eps, int nseg, void* scratch,
                                size_t scratch_bytes, void* stream) {
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (nseg < 1) return BASED_ERR_SHAPE;
  const int pre = prefill_preamble(q, k, v, y, kv_state, k_state, B, H, L, d, dv, q_strides, k_strides, v_strides,
                                   y_strides, BASED_BF16, state_dtype, st);
  if (pre != 0) return pre == kDone ? BASED_OK : pre;
  if (!launch_linattn_prefill_tc) return BASED_ERR_IMPL;
  return launch_linattn_prefill_tc(q, k, v, y, kv_state, k_state, B, H, L, dv, s3(q_strides), s3(k_strides),
                                   s3(v_strides), s3(y_strides), state_dtype, eps, nseg, scratch, scratch_bytes, st);
}

int based_linattn_prefill_split_static(const void* q, const void* k, const void* v, void* y, void* kv_state,
                                       void* k_state, int B, int H, int L, int d, int dv,
                                       const int64_t q_strides[3], const int64_t k_strides[3],
                                       const int64_t v_strides[3], const int64_t y_strides[3], int state_dtype,
                                       float eps, int nseg, void* stream) {
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (nseg < 1) return BASED_ERR_SHAPE;
  const int pre = prefill_preamble(q, k, v, y, kv_state, k_state, B, H, L, d, dv, q_strides, k_strides, v_strides,
                                   y_strides, BASED_BF16, state_dtype, st);
  if (pre != 0) return pre == kDone ? BASED_OK : pre;
  if (!launch_linattn_prefill_tc_static) return BASED_ERR_IMPL;
  return launch_linattn_prefill_tc_static(q, k, v, y, kv_state, k_state, B, H, L, dv, s3(q_strides), s3(k_strides),
                                          s3(v_strides), s3(y_strides), state_dtype, eps, nseg, st);
}

int based_linattn_decode(const void* q, const void* k, const void* v, void* y, void* kv_state, void* k_state,
                         int B, int H, int d, int dv, const int64_t q_strides[2], const int64_t k_strides[2],
                         const int64_t v_strides[2], const int64_t y_strides[2], int io_dtype, int state_dtype,
                         float eps, void* stream) {
  if (!q || !k || !v || !y || !kv_state || !k_state || !q_strides || !k_strides || !v_strides || !y_strides)
    return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype) || !dtype_ok(state_dtype)) return BASED_ERR_DTYPE;
  const int rows_per_group = state_dtype == BASED_F32 ? 4 : 8;
  if (B < 0 || H < 0 || d != kFeatureDim || dv < rows_per_group || dv > 128 || dv % rows_per_group != 0)
    return BASED_ERR_SHAPE;
  if ((int64_t)B * H > 2147483647LL) return BASED_ERR_TOO_LARGE;
  if (!aligned16(kv_state)) return BASED_ERR_ALIGN;
  if (B == 0 || H == 0) return BASED_OK;
  if (!launch_linattn_decode) return BASED_ERR_IMPL;
  return launch_linattn_decode(q, k, v, y, kv_state, k_state, B, H, dv, s2(q_strides), s2(k_strides),
                               s2(v_strides), s2(y_strides), io_dtype, state_dtype, eps,
                               static_cast<cudaStream_t>(stream));
}

int based_swa_prefill(const void* q, const void* k, const void* v, void* o, int B, int L, int H, int hd,
                      const int64_t q_strides[3], const int64_t k_strides[3], const int64_t v_strides[3],
                      const int64_t o_strides[3], int window_left, float softmax_scale, int io_dtype, int impl,
                      void* stream) {
  if (!q || !k || !v || !o || !q_strides || !k_strides || !v_strides || !o_strides) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (B < 0 || H < 0 || L < 0 || hd < 16 || hd > 128 || hd % 16 != 0 || window_left < 0) return BASED_ERR_SHAPE;
  if (H > 65535 || B > 65535) return BASED_ERR_TOO_LARGE;
  if (B == 0 || H == 0 || L == 0) return BASED_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool autosel = impl == BASED_IMPL_AUTO;
  if (autosel) impl = (io_dtype == BASED_BF16) ? BASED_IMPL_TCGEN05 : BASED_IMPL_SIMT;
  if (impl == BASED_IMPL_TCGEN05) {
    if (io_dtype != BASED_BF16) return BASED_ERR_IMPL;
    if (!launch_swa_prefill_tc) return BASED_ERR_IMPL;
    const int rc = launch_swa_prefill_tc(q, k, v, o, B, L, H, hd, s3_blh(q_strides), s3_blh(k_strides), s3_blh(v_strides),
                                         s3_blh(o_strides), window_left, softmax_scale, st);
    if (!(autosel && rc == BASED_ERR_IMPL)) return rc;
    impl = BASED_IMPL_SIMT;
  }
  if (impl != BASED_IMPL_SIMT) return BASED_ERR_IMPL;
  if (!launch_swa_prefill_simt) return BASED_ERR_IMPL;
  return launch_swa_prefill_simt(q, k, v, o, B, L, H, hd, s3_blh(q_strides), s3_blh(k_strides), s3_blh(v_strides),
                                 s3_blh(o_strides), window_left, softmax_scale, io_dtype, st);
}

int based_rotary_apply(void* x, int B, int L, int H, int hd, const int64_t x_strides[3], const void* rotary_cos,
                       const void* rotary_sin, int rotary_dim, const int32_t* seqlen_offsets, int seqlen_offset_scalar,
                       int io_dtype, void* stream) {
  if (!x || !x_strides || !rotary_cos || !rotary_sin) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (B < 0 || L < 0 || H < 0 || hd <= 0 || rotary_dim <= 0 || rotary_dim > hd || rotary_dim % 2 != 0 ||
      seqlen_offset_scalar < 0)
    return BASED_ERR_SHAPE;
  if (!launch_rotary) return BASED_ERR_IMPL;
  return launch_rotary(x, B, L, H, s3_blh(x_strides), rotary_cos, rotary_sin, rotary_dim, seqlen_offsets,
                       seqlen_offset_scalar, io_dtype, static_cast<cudaStream_t>(stream));
}

int based_swa_decode(const void* q, const void* k_new, const void* v_new, void* o, void* kv_cache,
                     const int32_t* cache_seqlens, int cache_seqlen_scalar, const void* rotary_cos,
                     const void* rotary_sin, int rotary_dim, int B, int H, int hd, int max_seqlen,
                     const int64_t q_strides[2], const int64_t k_strides[2], const int64_t v_strides[2],
                     const int64_t o_strides[2], int window_left, float softmax_scale, int io_dtype, void* stream) {
  if (!q || !k_new || !v_new || !o || !kv_cache || !q_strides || !k_strides || !v_strides || !o_strides)
    return BASED_ERR_NULL;
  if ((rotary_cos == nullptr) != (rotary_sin == nullptr)) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (B < 0 || H < 0 || hd < 16 || hd > 128 || hd % 16 != 0 || window_left < 0 || max_seqlen <= 0)
    return BASED_ERR_SHAPE;
  if (rotary_cos && (rotary_dim <= 0 || rotary_dim > hd || rotary_dim % 2 != 0)) return BASED_ERR_SHAPE;
  if (!cache_seqlens && (cache_seqlen_scalar < 0 || cache_seqlen_scalar >= max_seqlen)) return BASED_ERR_SHAPE;
  if (B == 0 || H == 0) return BASED_OK;
  if (!launch_swa_decode) return BASED_ERR_IMPL;
  return launch_swa_decode(q, k_new, v_new, o, kv_cache, cache_seqlens, cache_seqlen_scalar, rotary_cos, rotary_sin,
                           rotary_dim, B, H, hd, max_seqlen, s2(q_strides), s2(k_strides), s2(v_strides),
                           s2(o_strides), window_left, softmax_scale, io_dtype,
                           static_cast<cudaStream_t>(stream));
}

int based_gated_conv_prefill(const void* u1, const void* u2, void* v, void* state, const void* weight,
                             const void* bias, int B, int L, int di, int k, const int64_t u1_strides[2],
                             const int64_t u2_strides[2], const int64_t v_strides[2], int io_dtype, int w_dtype,
                             void* stream) {
  if (!u1 || !u2 || !v || !weight || !u1_strides || !u2_strides || !v_strides) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype) || !dtype_ok(w_dtype)) return BASED_ERR_DTYPE;
  if (B < 0 || L < 0 || di <= 0 || k < 1 || k > 4) return BASED_ERR_SHAPE;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (B == 0) return BASED_OK;
  if (L == 0) {  // nothing to compute; the state of an empty prompt is all zeros
    if (state) return (int)cudaMemsetAsync(state, 0, (size_t)B * di * k * dtype_size(io_dtype), st);
    return BASED_OK;
  }
  if (!launch_gated_conv_prefill) return BASED_ERR_IMPL;
  return launch_gated_conv_prefill(u1, u2, v, state, weight, bias, B, L, di, k, s2(u1_strides), s2(u2_strides),
                                   s2(v_strides), io_dtype, w_dtype, st);
}

int based_gated_conv_step(const void* u1, const void* u2, void* y, void* state, const void* weight, const void* bias,
                          int B, int di, int k, int64_t u1_batch_stride, int64_t u2_batch_stride,
                          int64_t y_batch_stride, int io_dtype, int w_dtype, void* stream) {
  if (!u1 || !u2 || !y || !state || !weight) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype) || !dtype_ok(w_dtype)) return BASED_ERR_DTYPE;
  if (B < 0 || di <= 0 || k < 1 || k > 4) return BASED_ERR_SHAPE;
  if ((int64_t)B * di > 2147483647LL) return BASED_ERR_TOO_LARGE;
  if (B == 0) return BASED_OK;
  if (!launch_gated_conv_step) return BASED_ERR_IMPL;
  return launch_gated_conv_step(u1, u2, y, state, weight, bias, B, di, k, u1_batch_stride, u2_batch_stride,
                                y_batch_stride, io_dtype, w_dtype, static_cast<cudaStream_t>(stream));
}

int based_add_rmsnorm(const void* x, const void* residual, const void* weight, const void* bias, void* out,
                      void* residual_out, int64_t M, int D, int64_t x_row_stride, int64_t residual_row_stride,
                      int64_t out_row_stride, int64_t residual_out_row_stride, float eps, int io_dtype, int res_dtype,
                      int w_dtype, int round_input, void* stream) {
  if (!x || !weight || !out) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype) || !dtype_ok(res_dtype) || !dtype_ok(w_dtype)) return BASED_ERR_DTYPE;
  if (M < 0 || D <= 0) return BASED_ERR_SHAPE;
  if (M == 0) return BASED_OK;
  return launch_add_rmsnorm(x, residual, weight, bias, out, residual_out, M, D, x_row_stride, residual_row_stride,
                            out_row_stride, residual_out_row_stride, eps, io_dtype, res_dtype, w_dtype, round_input,
                            static_cast<cudaStream_t>(stream));
}

int based_gated_act(const void* y, const void* gate, void* out, int64_t M, int F, int64_t y_row_stride,
                    int64_t gate_row_stride, int64_t out_row_stride, int act, int io_dtype, void* stream) {
  if (!y || !gate || !out) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (M < 0 || F <= 0 || (act != BASED_ACT_SILU && act != BASED_ACT_SIGMOID)) return BASED_ERR_SHAPE;
  if (M == 0) return BASED_OK;
  return launch_gated_act(y, gate, out, M, F, y_row_stride, gate_row_stride, out_row_stride, act, io_dtype,
                          static_cast<cudaStream_t>(stream));
}

int based_decode_linear(const void* x, const void* w, const void* bias, void* out, int M, int N, int K,
                        int64_t x_row_stride, int64_t out_row_stride, int epilogue, int act, void* conv_state,
                        const void* conv_weight, const void* conv_bias, int conv_k, int conv_w_dtype, void* stream) {
  if (!x || !w || !out) return BASED_ERR_NULL;
  if (M < 0 || N <= 0 || K <= 0 || M > 65535 * 16) return BASED_ERR_SHAPE;
  if (epilogue == BASED_EPI_GATED && act != BASED_ACT_SILU && act != BASED_ACT_SIGMOID) return BASED_ERR_SHAPE;
  if (epilogue == BASED_EPI_CONV) {
    if (!conv_state || !conv_weight) return BASED_ERR_NULL;
    if (conv_k < 1 || conv_k > 8) return BASED_ERR_SHAPE;
    if (!dtype_ok(conv_w_dtype)) return BASED_ERR_DTYPE;
  }
  if (M == 0) return BASED_OK;
  return launch_decode_linear(x, w, bias, out, M, N, K, x_row_stride, out_row_stride, epilogue, act, conv_state,
                              conv_weight, conv_bias, conv_k, conv_w_dtype, static_cast<cudaStream_t>(stream));
}

int based_rotary_qkv_cache(void* qkv, int B, int L, int H, int hd, const int64_t qkv_strides[4],
                           const void* rotary_cos, const void* rotary_sin, void* kv_cache,
                           const int64_t cache_strides[2], void* stream) {
  if (!qkv || !qkv_strides || !rotary_cos || !rotary_sin || !kv_cache || !cache_strides) return BASED_ERR_NULL;
  if (B < 0 || L < 0 || H < 0 || hd < 16 || hd > 256) return BASED_ERR_SHAPE;
  if (!launch_rotary_qkv_cache) return BASED_ERR_IMPL;
  return launch_rotary_qkv_cache(qkv, B, L, H, hd, qkv_strides[0], qkv_strides[1], qkv_strides[2], qkv_strides[3],
                                 rotary_cos, rotary_sin, kv_cache, cache_strides[0], cache_strides[1],
                                 static_cast<cudaStream_t>(stream));
}

size_t based_tp_outproj_workspace_bytes(int world, int max_rows, int N) {
  if (!tp_outproj_workspace_bytes) return 0;
  return tp_outproj_workspace_bytes(world, max_rows, N);
}

int based_tp_outproj_workspace_init(void* workspace, size_t bytes, void* stream) {
  if (!workspace) return BASED_ERR_NULL;
  if (bytes < 256 || (reinterpret_cast<uintptr_t>(workspace) & 255u)) return BASED_ERR_SCRATCH;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  cudaError_t e = cudaMemsetAsync(workspace, 0, bytes, st);
  if (e != cudaSuccess) return (int)e;
  // epoch of the first call = 1: the zero-filled flags then read as "nothing has arrived"
  e = cudaMemsetAsync(workspace, 1, 1, st);   // little-endian word 0 becomes 0x00000001
  return (int)e;
}

int based_tp_outproj_allreduce(const void* x, const void* w, const void* bias, void* out, int M, int N, int K,
                               int64_t x_row_stride, int64_t out_row_stride, void* const* workspaces, int max_rows,
                               int rank, int world, void* stream) {
  if (!x || !w || !out || !workspaces) return BASED_ERR_NULL;
  const void* xs[1] = {x};
  const void* ws[1] = {w};
  void* os[1] = {out};
  if (!launch_tp_outproj_allreduce) return BASED_ERR_IMPL;
  return launch_tp_outproj_allreduce(xs, ws, bias, os, workspaces, M, N, K, x_row_stride, out_row_stride, max_rows, rank,
                                     world, 0, static_cast<cudaStream_t>(stream));
}

int based_tp_outproj_allreduce_emulated(const void* const* x, const void* const* w, const void* bias, void* const* out,
                                        int M, int N, int K, int64_t x_row_stride, int64_t out_row_stride,
                                        void* const* workspaces, int max_rows, int world, void* stream) {
  if (!x || !w || !out || !workspaces) return BASED_ERR_NULL;
  if (!launch_tp_outproj_allreduce) return BASED_ERR_IMPL;
  return launch_tp_outproj_allreduce(x, w, bias, out, workspaces, M, N, K, x_row_stride, out_row_stride, max_rows, 0,
                                     world, 1, static_cast<cudaStream_t>(stream));
}

// ------------------------------------------------------------------ stateful mixers of the hybrid stacks

int based_stream_norm(const void* tokens, const void* table, const void* table_norm, int64_t V, const void* branch,
                      int64_t branch_row_stride, float mult, void* residual, const void* w1, const void* w2, void* out1,
                      void* out2, int64_t M, int D, float eps, int io_dtype, void* stream) {
  if (!residual || !w1 || !out1 || (w2 == nullptr) != (out2 == nullptr)) return BASED_ERR_NULL;
  if (tokens && (!table || !table_norm || V <= 0 || branch)) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (M < 0 || D <= 0) return BASED_ERR_SHAPE;
  if (M == 0) return BASED_OK;
  return launch_stream_norm(static_cast<const int64_t*>(tokens), table, table_norm, V, branch, branch_row_stride, mult,
                            static_cast<float*>(residual), w1, w2, out1, out2, M, D, eps, io_dtype,
                            static_cast<cudaStream_t>(stream));
}

int based_rmsnorm(const void* x, const void* weight, void* out, int64_t M, int D, int64_t x_row_stride,
                  int64_t out_row_stride, float eps, int io_dtype, void* stream) {
  if (!x || !weight || !out) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (M < 0 || D <= 0) return BASED_ERR_SHAPE;
  if (M == 0) return BASED_OK;
  if (M > 2147483647LL) return BASED_ERR_TOO_LARGE;
  return launch_rmsnorm(x, weight, out, M, D, x_row_stride, out_row_stride, eps, io_dtype, static_cast<cudaStream_t>(stream));
}

int based_short_conv(const void* x, void* y, void* ring, const void* weight, const void* bias, int B, int L, int C,
                     int taps, const int64_t x_strides[2], const int64_t y_strides[2], const int32_t* offsets, int offset,
                     int silu, int io_dtype, void* stream) {
  if (!x || !y || !weight || !x_strides || !y_strides) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (B < 0 || L < 0 || C <= 0 || taps < 1 || offset < 0) return BASED_ERR_SHAPE;
  if (!ring && (offsets || offset > 0)) return BASED_ERR_NULL;
  if (B == 0 || L == 0) return BASED_OK;
  if (!launch_short_conv) return BASED_ERR_IMPL;
  return launch_short_conv(x, y, ring, weight, bias, B, L, C, taps, s2(x_strides), s2(y_strides), offsets, offset, silu,
                           io_dtype, static_cast<cudaStream_t>(stream));
}

int based_latent_prepare(const void* z, const void* norm_weight, void* cache, void* q, const void* cos_table,
                         const void* sin_table, int table_len, int B, int L, int H, int kv_rank, int rot_dim, int dim,
                         int max_len, const int64_t z_strides[2], const int64_t cache_strides[2],
                         const int64_t q_strides[2], const int32_t* offsets, int offset, float eps, int io_dtype,
                         void* stream) {
  if (!cos_table || !sin_table || (z && (!norm_weight || !cache || !z_strides || !cache_strides)) || (q && !q_strides))
    return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (B < 0 || L < 0 || H <= 0 || kv_rank <= 0 || rot_dim <= 0 || rot_dim % 2 || dim < 0 || offset < 0) return BASED_ERR_SHAPE;
  if (!offsets && ((int64_t)offset + L > max_len || (int64_t)offset + L > table_len)) return BASED_ERR_SHAPE;
  if (B == 0 || L == 0) return BASED_OK;
  const int64_t zero[2] = {0, 0};
  const int64_t *zs = z ? z_strides : zero, *cs = z ? cache_strides : zero, *qs = q ? q_strides : zero;
  if (!launch_latent_prepare) return BASED_ERR_IMPL;
  return launch_latent_prepare(z, norm_weight, cache, q, static_cast<const float*>(cos_table),
                               static_cast<const float*>(sin_table), table_len, B, L, H, kv_rank, rot_dim, dim, max_len,
                               zs[0], zs[1], cs[0], cs[1], qs[0], qs[1], offsets, offset, eps, io_dtype,
                               static_cast<cudaStream_t>(stream));
}

int based_split_key_attention(const void* q1, const void* q2, const void* k1, const void* k2, const void* v,
                              const void* gate, void* out, int B, int L, int H, int d1, int d2, int dv,
                              const int64_t q1_strides[3], const int64_t q2_strides[3], const int64_t k1_strides[3],
                              const int64_t k2_strides[3], const int64_t v_strides[3], const int64_t out_strides[3],
                              const int64_t gate_strides[2], const int32_t* offsets, int offset, float scale,
                              int io_dtype, void* stream) {
  if (!q1 || !q2 || !k1 || !k2 || !v || !out || (gate && !gate_strides)) return BASED_ERR_NULL;
  if (!q1_strides || !q2_strides || !k1_strides || !k2_strides || !v_strides || !out_strides) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (B < 0 || L < 0 || H <= 0 || d1 <= 0 || d2 < 0 || dv <= 0 || offset < 0) return BASED_ERR_SHAPE;
  if (B == 0 || L == 0) return BASED_OK;
  if (!launch_split_key_attention) return BASED_ERR_IMPL;
  return launch_split_key_attention(q1, q2, k1, k2, v, gate, out, B, L, H, d1, d2, dv, s3_blh(q1_strides),
                                    s3_blh(q2_strides), s3_blh(k1_strides), s3_blh(k2_strides), s3_blh(v_strides),
                                    s3_blh(out_strides), gate ? gate_strides[0] : 0, gate ? gate_strides[1] : 0, offsets,
                                    offset, scale, AttentionOptions{}, io_dtype, static_cast<cudaStream_t>(stream));
}

int based_latent_prefill(const void* q1, const void* q2, const void* k1, const void* k2, const void* v, const void* gate,
                         void* out, int B, int L, int T, int H, int d1, int d2, int dv, const int64_t q1_strides[3],
                         const int64_t q2_strides[3], const int64_t k1_strides[3], const int64_t k2_strides[2],
                         const int64_t v_strides[3], const int64_t out_strides[3], const int64_t gate_strides[2],
                         int offset, float scale, int io_dtype, int impl, void* stream) {
  if (!q1 || !q2 || !k1 || !k2 || !v || !out || (gate && !gate_strides)) return BASED_ERR_NULL;
  if (!q1_strides || !q2_strides || !k1_strides || !k2_strides || !v_strides || !out_strides) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (B < 0 || L < 0 || H <= 0 || d1 <= 0 || d2 <= 0 || dv <= 0 || offset < 0 || (int64_t)offset + L > T) return BASED_ERR_SHAPE;
  if (B == 0 || L == 0) return BASED_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const Strides3 sk2{k2_strides[0], 0, k2_strides[1]};
  const int64_t gb = gate ? gate_strides[0] : 0, gl = gate ? gate_strides[1] : 0;
  if (impl == BASED_IMPL_TCGEN05 || (impl == BASED_IMPL_AUTO && io_dtype == BASED_BF16)) {
    if (io_dtype != BASED_BF16) return BASED_ERR_IMPL;
    if (!launch_latent_prefill_tc) return BASED_ERR_IMPL;
    const int rc = launch_latent_prefill_tc(q1, q2, k1, k2, v, gate, out, B, L, T, H, d1, d2, dv, s3_blh(q1_strides),
                                            s3_blh(q2_strides), s3_blh(k1_strides), sk2, s3_blh(v_strides),
                                            s3_blh(out_strides), gb, gl, nullptr, offset, scale, st);
    if (!(impl == BASED_IMPL_AUTO && rc == BASED_ERR_IMPL)) return rc;
  }
  if (!launch_split_key_attention) return BASED_ERR_IMPL;
  return launch_split_key_attention(q1, q2, k1, k2, v, gate, out, B, L, H, d1, d2, dv, s3_blh(q1_strides),
                                    s3_blh(q2_strides), s3_blh(k1_strides), sk2, s3_blh(v_strides), s3_blh(out_strides),
                                    gb, gl, nullptr, offset, scale, AttentionOptions{}, io_dtype, st);
}

size_t based_latent_decode_scratch_bytes(int B, int L, int H, int kv_rank, int max_len) {
  if (B <= 0 || L <= 0 || H <= 0 || kv_rank <= 0 || max_len <= 0) return 0;
  if (!latent_decode_scratch_bytes) return 0;
  return latent_decode_scratch_bytes(B, L * H, kv_rank, max_len);
}

int based_latent_decode(const void* qa, const void* qr, const void* cache, const void* gate, void* out, void* scratch,
                        size_t scratch_bytes, int B, int L, int H, int kv_rank, int rot_dim, int max_len,
                        const int64_t qa_strides[3], const int64_t qr_strides[3], const int64_t cache_strides[2],
                        const int64_t out_strides[3], const int64_t gate_strides[2], const int32_t* offsets, int offset,
                        float scale, int io_dtype, void* stream) {
  if (!qa || !qr || !cache || !out || (gate && !gate_strides)) return BASED_ERR_NULL;
  if (!qa_strides || !qr_strides || !cache_strides || !out_strides) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (B < 0 || L < 0 || H <= 0 || kv_rank <= 0 || rot_dim <= 0 || max_len <= 0 || offset < 0) return BASED_ERR_SHAPE;
  if (!offsets && (int64_t)offset + L > max_len) return BASED_ERR_SHAPE;
  if (B == 0 || L == 0) return BASED_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int64_t gb = gate ? gate_strides[0] : 0, gl = gate ? gate_strides[1] : 0;
  if (io_dtype == BASED_BF16) {
    if (!launch_latent_decode) return BASED_ERR_IMPL;
    const int rc = launch_latent_decode(qa, qr, cache, gate, out, scratch, scratch_bytes, B, L, H, kv_rank, rot_dim, max_len,
                                        s3_blh(qa_strides), s3_blh(qr_strides), cache_strides[0], cache_strides[1],
                                        s3_blh(out_strides), gb, gl, offsets, offset, scale, st);
    if (rc != BASED_ERR_IMPL) return rc;
  }
  // fp32 models and other sizes: the cached rows as keys and values of every head
  const Strides3 sc{cache_strides[0], 0, cache_strides[1]};
  const char* rot = static_cast<const char*>(cache) + kv_rank * dtype_size(io_dtype);
  if (!launch_split_key_attention) return BASED_ERR_IMPL;
  return launch_split_key_attention(qa, qr, cache, rot, cache, gate, out, B, L, H, kv_rank, rot_dim, kv_rank,
                                    s3_blh(qa_strides), s3_blh(qr_strides), sc, sc, sc, s3_blh(out_strides), gb, gl, offsets,
                                    offset, scale, AttentionOptions{}, io_dtype, st);
}

int based_delta_prefill(const void* q, const void* k, const void* v, const void* z, const void* a, const void* b,
                        const void* A_log, const void* dt_bias, const void* norm_weight, void* state, void* out, int B,
                        int L, int H, int Hk, int d, int dv, const int64_t q_strides[2], const int64_t k_strides[2],
                        const int64_t v_strides[2], const int64_t z_strides[2], const int64_t gate_strides[2],
                        const int64_t out_strides[2], const int32_t* offsets, int offset, float eps, int io_dtype,
                        int impl, void* scratch, size_t scratch_bytes, void* stream) {
  if (!q || !k || !v || !z || !a || !b || !A_log || !dt_bias || !norm_weight || !state || !out) return BASED_ERR_NULL;
  if (!q_strides || !k_strides || !v_strides || !z_strides || !gate_strides || !out_strides) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (B < 0 || L < 0 || H <= 0 || Hk <= 0 || H % Hk || d <= 0 || dv <= 0 || offset < 0) return BASED_ERR_SHAPE;
  if (B == 0 || L == 0) return BASED_OK;
  // AUTO: chunks for bf16 from a handful of tokens on, else token by token
  if (impl == BASED_IMPL_TCGEN05 || (impl == BASED_IMPL_AUTO && io_dtype == BASED_BF16 && L >= 8)) {
    if (io_dtype != BASED_BF16) return BASED_ERR_IMPL;
    if (!launch_delta_chunk) return BASED_ERR_IMPL;
    const int rc = launch_delta_chunk(q, k, v, z, static_cast<const float*>(a), static_cast<const float*>(b),
                                      static_cast<const float*>(A_log), static_cast<const float*>(dt_bias), norm_weight,
                                      static_cast<float*>(state), out, scratch, scratch_bytes, B, L, H, Hk, d, dv,
                                      s2(q_strides), s2(k_strides), s2(v_strides), s2(z_strides), s2(gate_strides),
                                      s2(out_strides), offsets, offset, eps, static_cast<cudaStream_t>(stream));
    if (!(impl == BASED_IMPL_AUTO && rc == BASED_ERR_IMPL)) return rc;
  }
  if (!launch_delta_recurrent) return BASED_ERR_IMPL;
  return launch_delta_recurrent(q, k, v, z, static_cast<const float*>(a), static_cast<const float*>(b),
                                static_cast<const float*>(A_log), static_cast<const float*>(dt_bias), norm_weight,
                                static_cast<float*>(state), out, B, L, H, Hk, d, dv, s2(q_strides), s2(k_strides),
                                s2(v_strides), s2(z_strides), s2(gate_strides), s2(out_strides), offsets, offset, eps,
                                io_dtype, static_cast<cudaStream_t>(stream));
}

size_t based_delta_prefill_scratch_bytes(int B, int L, int H, int d, int dv) {
  if (B <= 0 || L <= 0 || H <= 0 || d <= 0 || dv <= 0) return 0;
  if (!delta_chunk_scratch_bytes) return 0;
  return delta_chunk_scratch_bytes(B, L, H, d, dv);
}

int based_delta_step(const void* x, const void* conv_weight, void* ring, const void* a, const void* b, const void* A_log,
                     const void* dt_bias, const void* norm_weight, void* state, void* out, int B, int H, int Hk, int d,
                     int dv, int taps, int64_t x_stride, int64_t gate_stride, int64_t out_stride, const int32_t* offsets,
                     int offset, float eps, int io_dtype, void* stream) {
  if (!x || !conv_weight || !ring || !a || !b || !A_log || !dt_bias || !norm_weight || !state || !out) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (B < 0 || H <= 0 || Hk <= 0 || H % Hk || d <= 0 || dv <= 0 || taps < 1 || offset < 0) return BASED_ERR_SHAPE;
  if (B == 0) return BASED_OK;
  if (!launch_delta_step) return BASED_ERR_IMPL;
  return launch_delta_step(x, conv_weight, ring, static_cast<const float*>(a), static_cast<const float*>(b),
                           static_cast<const float*>(A_log), static_cast<const float*>(dt_bias), norm_weight,
                           static_cast<float*>(state), out, B, H, Hk, d, dv, taps, x_stride, gate_stride, out_stride,
                           offsets, offset, eps, io_dtype, static_cast<cudaStream_t>(stream));
}

int based_rglru(const void* u, const void* y, const void* gates, const void* r_bias, const void* i_bias, const void* lam,
                void* state, void* out, int B, int L, int W, int block_width, const int64_t u_strides[2],
                const int64_t y_strides[2], const int64_t out_strides[2], const int64_t gate_strides[2],
                const int32_t* offsets, int offset, int io_dtype, void* stream) {
  if (!u || !y || !gates || !r_bias || !i_bias || !lam || !state || !out) return BASED_ERR_NULL;
  if (!u_strides || !y_strides || !out_strides || !gate_strides) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (B < 0 || L < 0 || W <= 0 || block_width <= 0 || W % block_width || offset < 0) return BASED_ERR_SHAPE;
  if (B == 0 || L == 0) return BASED_OK;
  if (!launch_rglru) return BASED_ERR_IMPL;
  return launch_rglru(u, y, static_cast<const float*>(gates), r_bias, i_bias, static_cast<const float*>(lam),
                      static_cast<float*>(state), out, B, L, W, block_width, s2(u_strides), s2(y_strides),
                      s2(out_strides), gate_strides[0], gate_strides[1], offsets, offset, io_dtype,
                      static_cast<cudaStream_t>(stream));
}

int based_rglru_gated(const void* u, const void* y, const void* gate_weight, const void* r_bias, const void* i_bias,
                      const void* lam, void* state, void* out, int B, int L, int W, int block_width,
                      const int64_t u_strides[2], const int64_t y_strides[2], const int64_t out_strides[2],
                      const int32_t* offsets, int offset, int io_dtype, void* stream) {
  if (!u || !y || !gate_weight || !r_bias || !i_bias || !lam || !state || !out) return BASED_ERR_NULL;
  if (!u_strides || !y_strides || !out_strides) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (B < 0 || L < 0 || W <= 0 || block_width <= 0 || W % block_width || offset < 0) return BASED_ERR_SHAPE;
  if (B == 0 || L == 0) return BASED_OK;
  if (io_dtype != BASED_BF16) return BASED_ERR_IMPL;
  if (!launch_rglru_tc) return BASED_ERR_IMPL;
  return launch_rglru_tc(u, y, gate_weight, r_bias, i_bias, static_cast<const float*>(lam), static_cast<float*>(state), out,
                         B, L, W, block_width, s2(u_strides), s2(y_strides), s2(out_strides), offsets, offset,
                         static_cast<cudaStream_t>(stream));
}

// ------------------------------------------------------------------ post-norm stacks

int based_stream_embed(const void* tokens, const void* table, int64_t V, float scale, const void* pos_table, int64_t P,
                       void* residual, void* out, int B, int L, int D, const int32_t* offsets, int offset, int io_dtype,
                       void* stream) {
  if (!tokens || !table || !pos_table || !residual) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (B < 0 || L < 0 || D <= 0 || V <= 0 || P <= 0 || offset < 0) return BASED_ERR_SHAPE;
  if (!offsets && (int64_t)offset + L > P) return BASED_ERR_SHAPE;
  if (B == 0 || L == 0) return BASED_OK;
  return launch_stream_embed(static_cast<const int64_t*>(tokens), table, V, scale, pos_table, P, static_cast<float*>(residual),
                             out, B, L, D, offsets, offset, io_dtype, static_cast<cudaStream_t>(stream));
}

int based_stream_post_norm(const void* branch, int64_t branch_row_stride, const void* weight, void* residual,
                           const void* out_weight, void* out, int64_t M, int D, float eps, int io_dtype, void* stream) {
  if (!branch || !weight || !residual || (out_weight && !out)) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (M < 0 || D <= 0) return BASED_ERR_SHAPE;
  if (M == 0) return BASED_OK;
  return launch_stream_post_norm(branch, branch_row_stride, weight, static_cast<float*>(residual), out_weight, out, M, D, eps,
                                 io_dtype, static_cast<cudaStream_t>(stream));
}

int based_norm_gate(const void* x, int64_t x_row_stride, const void* weight, const void* gate, int64_t gate_row_stride,
                    void* out, int64_t out_row_stride, int64_t M, int D, float eps, int io_dtype, void* stream) {
  if (!x || !weight || !gate || !out) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (M < 0 || D <= 0) return BASED_ERR_SHAPE;
  if (M == 0) return BASED_OK;
  return launch_norm_gate(x, x_row_stride, weight, gate, gate_row_stride, out, out_row_stride, M, D, eps, io_dtype,
                          static_cast<cudaStream_t>(stream));
}

int based_token_gate(const void* z, int64_t z_row_stride, const void* tokens, const void* table, int64_t V,
                     int64_t table_row_stride, int64_t column, void* out, int64_t M, int n, int io_dtype, void* stream) {
  if (!z || !tokens || !table || !out) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (M < 0 || n <= 0 || V <= 0 || column < 0 || column + n > table_row_stride) return BASED_ERR_SHAPE;
  if (M == 0) return BASED_OK;
  return launch_token_gate(z, z_row_stride, static_cast<const int64_t*>(tokens), table, V, table_row_stride, column, out, M, n,
                           io_dtype, static_cast<cudaStream_t>(stream));
}

int based_token_side(const void* x, int64_t x_row_stride, const void* tokens, const void* gate_weight, const void* proj_weight,
                     const void* table, int64_t V, int64_t table_row_stride, int64_t column, const void* norm_weight, void* residual,
                     const void* out_weight, void* out, int M, int W, int n, float eps, int io_dtype, void* stream) {
  if (!x || !tokens || !gate_weight || !proj_weight || !table || !norm_weight || !residual || !out) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (M < 0 || W <= 0 || n <= 0 || V <= 0 || column < 0 || column + n > table_row_stride) return BASED_ERR_SHAPE;
  if (M == 0) return BASED_OK;
  if (io_dtype != BASED_BF16 || !launch_token_side) return BASED_ERR_IMPL;
  return launch_token_side(x, x_row_stride, static_cast<const int64_t*>(tokens), gate_weight, proj_weight, table, V, table_row_stride,
                           column, norm_weight, static_cast<float*>(residual), out_weight, out, M, W, n, eps,
                           static_cast<cudaStream_t>(stream));
}

int based_tied_prepare(void* q, const void* k, const void* q_weight, const void* k_weight, void* cache, void* factor, int B,
                       int L, int H, int G, int d, int max_len, const int64_t q_strides[2], const int64_t k_strides[2],
                       const int64_t cache_strides[2], const int64_t factor_strides[2], const int32_t* offsets, int offset,
                       float eps, float temp_coef, float temp_every, int io_dtype, void* stream) {
  if (!q || !k || !q_weight || !k_weight || !cache || !factor) return BASED_ERR_NULL;
  if (!q_strides || !k_strides || !cache_strides || !factor_strides) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (B < 0 || L < 0 || H <= 0 || G <= 0 || H % G || d <= 0 || d > 512 || offset < 0) return BASED_ERR_SHAPE;
  if (temp_coef != 0.f && !(temp_every > 0.f)) return BASED_ERR_SHAPE;
  if (!offsets && (int64_t)offset + L > max_len) return BASED_ERR_SHAPE;
  if (B == 0 || L == 0) return BASED_OK;
  if (!launch_tied_prepare) return BASED_ERR_IMPL;
  return launch_tied_prepare(q, k, q_weight, k_weight, cache, static_cast<float*>(factor), B, L, H, G, d, max_len, q_strides[0],
                             q_strides[1], k_strides[0], k_strides[1], cache_strides[0], cache_strides[1], factor_strides[0],
                             factor_strides[1], offsets, offset, eps, temp_coef, temp_every, io_dtype,
                             static_cast<cudaStream_t>(stream));
}

int based_tied_attention(const void* q, const void* cache, const void* factor, const void* gate, void* out, int B, int L, int H,
                         int G, int d, int max_len, const int64_t q_strides[2], const int64_t cache_strides[2],
                         const int64_t factor_strides[2], const int64_t gate_strides[2], const int64_t out_strides[2],
                         const int32_t* offsets, int offset, float scale, float sink, int io_dtype, int impl, void* scratch,
                         size_t scratch_bytes, void* count, int count_len, void* stream) {
  if (!q || !cache || !factor || !out || (gate && !gate_strides)) return BASED_ERR_NULL;
  if (!q_strides || !cache_strides || !factor_strides || !out_strides) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (B < 0 || L < 0 || H <= 0 || G <= 0 || H % G || d <= 0 || d > 512 || max_len <= 0 || offset < 0 || sink < 0.f) return BASED_ERR_SHAPE;
  if (!offsets && (int64_t)offset + L > max_len) return BASED_ERR_SHAPE;
  if (B == 0 || L == 0) return BASED_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  AttentionOptions x;
  x.key_factor = static_cast<const float*>(factor);
  x.fb = factor_strides[0]; x.fh = factor_strides[1];
  x.group = H / G;
  x.sink = sink;
  x.gate_per_element = 1;
  const int64_t gb = gate ? gate_strides[0] : 0, gl = gate ? gate_strides[1] : 0;
  const bool autosel = impl == BASED_IMPL_AUTO;
  if (io_dtype != BASED_BF16 && !autosel && impl != BASED_IMPL_SIMT) return BASED_ERR_IMPL;
  if (io_dtype == BASED_BF16 && (impl == BASED_IMPL_DECODE || (autosel && (offsets || L * (H / G) <= BASED_TIED_DECODE_ROWS)))) {
    if (!launch_tied_decode) return BASED_ERR_IMPL;
    const int rc = launch_tied_decode(q, cache, x.key_factor, gate, out, scratch, scratch_bytes, static_cast<int*>(count), count_len, B,
                                      L, H, G, d, max_len, q_strides[0], q_strides[1], cache_strides[0], cache_strides[1], x.fb,
                                      x.fh, gb, gl, out_strides[0], out_strides[1], offsets, offset, scale, sink, st);
    if (!(autosel && rc == BASED_ERR_IMPL)) return rc;
  }
  if (io_dtype == BASED_BF16 && !offsets && (impl == BASED_IMPL_TCGEN05 || autosel)) {
    if (!launch_tied_prefill_tc) return BASED_ERR_IMPL;
    const int rc = launch_tied_prefill_tc(q, cache, x.key_factor, gate, out, B, L, H, G, d, q_strides[0], q_strides[1],
                                          cache_strides[0], cache_strides[1], x.fb, x.fh, gb, gl, out_strides[0],
                                          out_strides[1], offset, scale, sink, st);
    if (!(autosel && rc == BASED_ERR_IMPL)) return rc;
  }
  if (!autosel && impl != BASED_IMPL_SIMT) return BASED_ERR_IMPL;
  const Strides3 sq{q_strides[0], d, q_strides[1]}, sc{cache_strides[0], d, cache_strides[1]}, so{out_strides[0], d, out_strides[1]};
  if (!launch_split_key_attention) return BASED_ERR_IMPL;
  return launch_split_key_attention(q, q, cache, cache, cache, gate, out, B, L, H, d, 0, d, sq, sq, sc, sc, sc, so, gb, gl,
                                    offsets, offset, scale, x, io_dtype, st);
}

size_t based_tied_attention_scratch_bytes(int B, int L, int H, int G, int d, int max_len) {
  if (B <= 0 || L <= 0 || H <= 0 || G <= 0 || H % G || d <= 0 || max_len <= 0 || !tied_decode_scratch_bytes) return 0;
  return tied_decode_scratch_bytes(B, L * (H / G), G, d, max_len);
}

int based_lightning(const void* q, const void* k, const void* v, const void* decay, void* state, void* out, int B, int L, int H,
                    int d, int dv, const int64_t q_strides[2], const int64_t k_strides[2], const int64_t v_strides[2],
                    const int64_t out_strides[2], const int32_t* offsets, int offset, int io_dtype, int impl, void* stream) {
  if (!q || !k || !v || !decay || !state || !out || !q_strides || !k_strides || !v_strides || !out_strides) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (B < 0 || L < 0 || H <= 0 || d <= 0 || d > 512 || dv <= 0 || offset < 0) return BASED_ERR_SHAPE;
  if (B == 0 || L == 0) return BASED_OK;
  // AUTO: chunks for bf16 from a handful of tokens on, else token by token
  const bool autosel = impl == BASED_IMPL_AUTO;
  if (impl == BASED_IMPL_TCGEN05 || (autosel && io_dtype == BASED_BF16 && L >= 16)) {
    if (io_dtype != BASED_BF16 || !launch_lightning_tc) return BASED_ERR_IMPL;
    const int rc = launch_lightning_tc(q, k, v, static_cast<const float*>(decay), static_cast<float*>(state), out, B, L, H, d, dv,
                                       s2(q_strides), s2(k_strides), s2(v_strides), s2(out_strides), offsets, offset,
                                       static_cast<cudaStream_t>(stream));
    if (!(autosel && rc == BASED_ERR_IMPL)) return rc;
  }
  if (!launch_lightning_recurrent) return BASED_ERR_IMPL;
  return launch_lightning_recurrent(q, k, v, static_cast<const float*>(decay), static_cast<float*>(state), out, B, L, H, d, dv,
                                    s2(q_strides), s2(k_strides), s2(v_strides), s2(out_strides), offsets, offset, io_dtype,
                                    static_cast<cudaStream_t>(stream));
}

int based_lightning_step(const void* q, const void* k, const void* v, const void* gate, int64_t x_row_stride, const void* decay,
                         const void* norm_weight, void* state, void* read, void* count, void* out, int64_t out_row_stride, int B,
                         int H, int d, int dv, const int32_t* offsets, int offset, float eps, int io_dtype, void* stream) {
  if (!q || !k || !v || !gate || !decay || !norm_weight || !state || !read || !count || !out) return BASED_ERR_NULL;
  if (!dtype_ok(io_dtype)) return BASED_ERR_DTYPE;
  if (B < 0 || H <= 0 || d <= 0 || dv <= 0 || offset < 0) return BASED_ERR_SHAPE;
  if (B == 0) return BASED_OK;
  if (!launch_lightning_step) return BASED_ERR_IMPL;
  return launch_lightning_step(q, k, v, gate, x_row_stride, static_cast<const float*>(decay), norm_weight,
                               static_cast<float*>(state), static_cast<float*>(read), static_cast<int*>(count), out,
                               out_row_stride, B, H, d, dv, offsets, offset, eps, io_dtype, static_cast<cudaStream_t>(stream));
}

}  // extern "C"
