// Shared helpers for the based_b200 kernels (sm_100a).
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "based_b200.h"

namespace based {

constexpr int kFeatureDim = 16;                 // d
constexpr int kExpandedDim = BASED_EXPANDED_DIM;  // D = 1 + d + d*d

// Constants of the Taylor map for d = 16 (linear_attention.py:62-64):
//   first order  x / d^(1/4)            = x * 0.5
//   second order x_i x_j / (sqrt2 * sqrt d) = x_i x_j * 0.17677669...
constexpr float kC1 = 0.5f;
constexpr float kC2 = 0.17677669529663687f;

struct Strides3 { int64_t b, h, l; };
struct Strides2 { int64_t b, h; };

template <typename T> __device__ __forceinline__ float to_float(T x);
template <> __device__ __forceinline__ float to_float<float>(float x) { return x; }
template <> __device__ __forceinline__ float to_float<__nv_bfloat16>(__nv_bfloat16 x) { return __bfloat162float(x); }

template <typename T> __device__ __forceinline__ T from_float(float x);
template <> __device__ __forceinline__ float from_float<float>(float x) { return x; }
template <> __device__ __forceinline__ __nv_bfloat16 from_float<__nv_bfloat16>(float x) { return __float2bfloat16_rn(x); }

// phi(x)[f] for f in [0, 273) from the 16 raw values in x[] (any indexable of float).
template <typename X>
__device__ __forceinline__ float taylor_feature(const X& x, int f) {
  if (f == 0) return 1.0f;
  if (f <= kFeatureDim) return x[f - 1] * kC1;
  const int g = f - 1 - kFeatureDim;
  return x[g >> 4] * x[g & 15] * kC2;
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}

inline bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; }

// Launchers implemented one per .cu file; all return a cudaError_t-compatible int (0 = ok).
// BASED_WEAK: not in every build of the library (a part without a kernel leaves its launcher null; capi.cu checks).
#define BASED_WEAK __attribute__((weak))
BASED_WEAK int launch_linattn_decode(const void* q, const void* k, const void* v, void* y, void* kv_state, void* k_state,
                          int B, int H, int dv, Strides2 sq, Strides2 sk, Strides2 sv, Strides2 sy,
                          int io_dtype, int state_dtype, float eps, cudaStream_t stream);

BASED_WEAK int launch_linattn_prefill_simt(const void* q, const void* k, const void* v, void* y, void* kv_state, void* k_state,
                                int B, int H, int L, int dv, Strides3 sq, Strides3 sk, Strides3 sv, Strides3 sy,
                                int io_dtype, int state_dtype, float eps, cudaStream_t stream);

BASED_WEAK int launch_linattn_prefill_tc(const void* q, const void* k, const void* v, void* y, void* kv_state, void* k_state,
                              int B, int H, int L, int dv, Strides3 sq, Strides3 sk, Strides3 sv, Strides3 sy,
                              int state_dtype, float eps, int nseg, void* scratch, size_t scratch_bytes,
                              cudaStream_t stream);
BASED_WEAK int launch_linattn_prefill_tc_static(const void* q, const void* k, const void* v, void* y, void* kv_state,
                                     void* k_state, int B, int H, int L, int dv, Strides3 sq, Strides3 sk,
                                     Strides3 sv, Strides3 sy, int state_dtype, float eps, int nseg,
                                     cudaStream_t stream);
BASED_WEAK int linattn_prefill_tc_auto_segments(int B, int H, int L);
BASED_WEAK size_t linattn_prefill_tc_scratch_bytes(int B, int H, int L, int dv, int nseg);

BASED_WEAK int launch_gated_conv_prefill(const void* u1, const void* u2, void* v, void* state, const void* weight,
                              const void* bias, int B, int L, int di, int k, Strides2 s1, Strides2 s2, Strides2 sv,
                              int io_dtype, int w_dtype, cudaStream_t stream);
BASED_WEAK int launch_gated_conv_step(const void* u1, const void* u2, void* y, void* state, const void* weight, const void* bias,
                           int B, int di, int k, int64_t s1, int64_t s2, int64_t sy, int io_dtype, int w_dtype,
                           cudaStream_t stream);

int launch_add_rmsnorm(const void* x, const void* residual, const void* weight, const void* bias, void* out,
                       void* residual_out, int64_t M, int D, int64_t sx, int64_t sr, int64_t so, int64_t sro, float eps,
                       int io_dtype, int res_dtype, int w_dtype, int round_input, cudaStream_t stream);
int launch_gated_act(const void* y, const void* gate, void* out, int64_t M, int F, int64_t sy, int64_t sg, int64_t so,
                     int act, int io_dtype, cudaStream_t stream);

BASED_WEAK int launch_rotary_qkv_cache(void* qkv, int B, int L, int H, int hd, int64_t sb, int64_t sl, int64_t s3, int64_t sh,
                            const void* rcos, const void* rsin, void* cache, int64_t cb, int64_t cl,
                            cudaStream_t stream);
int launch_decode_linear(const void* x, const void* w, const void* bias, void* out, int M, int N, int K, int64_t sx,
                         int64_t so, int epilogue, int act, void* conv_state, const void* conv_weight,
                         const void* conv_bias, int conv_k, int conv_w_dtype, cudaStream_t stream);

BASED_WEAK int launch_tp_outproj_allreduce(const void* const* x, const void* const* w, const void* bias, void* const* out,
                                void* const* workspaces, int M, int N, int K, int64_t sx, int64_t so, int Mmax,
                                int rank, int world, int emulate, cudaStream_t stream);
BASED_WEAK size_t tp_outproj_workspace_bytes(int world, int Mmax, int N);
BASED_WEAK int read_tp_status(unsigned int* out, int reset);      // fused output projection + all-reduce

BASED_WEAK int read_tc_status(unsigned int* out, int reset);      // linear-attention prefill kernel
BASED_WEAK int read_tc_status_swa(unsigned int* out, int reset);  // sliding-window prefill kernel

BASED_WEAK int launch_swa_prefill_simt(const void* q, const void* k, const void* v, void* o, int B, int L, int H, int hd,
                            Strides3 sq, Strides3 sk, Strides3 sv, Strides3 so, int window_left, float scale,
                            int io_dtype, cudaStream_t stream);

BASED_WEAK int launch_swa_prefill_tc(const void* q, const void* k, const void* v, void* o, int B, int L, int H, int hd,
                          Strides3 sq, Strides3 sk, Strides3 sv, Strides3 so, int window_left, float scale,
                          cudaStream_t stream);

BASED_WEAK int launch_rotary(void* x, int B, int L, int H, Strides3 sx, const void* rcos, const void* rsin, int rotary_dim,
                  const int32_t* offsets, int offset_scalar, int io_dtype, cudaStream_t stream);

BASED_WEAK int launch_swa_decode(const void* q, const void* k_new, const void* v_new, void* o, void* kv_cache,
                      const int32_t* cache_seqlens, int cache_seqlen_scalar, const void* rotary_cos,
                      const void* rotary_sin, int rotary_dim, int B, int H, int hd, int max_seqlen,
                      Strides2 sq, Strides2 sk, Strides2 sv, Strides2 so, int window_left, float scale,
                      int io_dtype, cudaStream_t stream);

// What an attention kernel may do beyond softmax(q k^T) v with a gate per head.
struct AttentionOptions {
  const float* key_factor = nullptr;   // [B, key heads, keys]: factor of a key's scores (strides fb, fh, 1)
  int64_t fb = 0, fh = 0;
  int group = 1;                       // query heads that share a key head
  float sink = 0.f;                    // added to the softmax sum as that many scores of 0 without a value
  int gate_per_element = 0;            // gate [B, L, H * dv] instead of [B, L, H]
};

// Stateful mixers of the hybrid stacks.  offsets (device, one per batch row) or offset: position of a call's first token.
int launch_stream_norm(const int64_t* tokens, const void* table, const void* table_norm, int64_t V, const void* branch,
                       int64_t branch_stride, float mult, float* residual, const void* w1, const void* w2, void* out1,
                       void* out2, int64_t M, int D, float eps, int io_dtype, cudaStream_t stream);
int launch_rmsnorm(const void* x, const void* w, void* out, int64_t M, int D, int64_t sx, int64_t so, float eps,
                   int io_dtype, cudaStream_t stream);
BASED_WEAK int launch_short_conv(const void* x, void* y, void* ring, const void* w, const void* bias, int B, int L, int C, int taps,
                      Strides2 sx, Strides2 sy, const int32_t* offsets, int offset, int silu, int io_dtype,
                      cudaStream_t stream);
BASED_WEAK int launch_latent_prepare(const void* z, const void* norm_w, void* cache, void* q, const float* cosv, const float* sinv,
                          int table_len, int B, int L, int H, int r, int rd, int d, int max_len, int64_t zb, int64_t zl,
                          int64_t cb, int64_t cl, int64_t qb, int64_t ql, const int32_t* offsets, int offset, float eps,
                          int io_dtype, cudaStream_t stream);
BASED_WEAK int launch_split_key_attention(const void* q1, const void* q2, const void* k1, const void* k2, const void* v,
                               const void* gate, void* out, int B, int L, int H, int d1, int d2, int dv, Strides3 sq1,
                               Strides3 sq2, Strides3 sk1, Strides3 sk2, Strides3 sv, Strides3 so, int64_t gb, int64_t gl,
                               const int32_t* offsets, int offset, float scale, AttentionOptions x, int io_dtype,
                               cudaStream_t stream);
BASED_WEAK int launch_delta_recurrent(const void* q, const void* k, const void* v, const void* z, const float* a, const float* b,
                           const float* A_log, const float* dt_bias, const void* norm_w, float* state, void* out, int B,
                           int L, int H, int Hk, int d, int dv, Strides2 sq, Strides2 sk, Strides2 sv, Strides2 sz,
                           Strides2 sg, Strides2 so, const int32_t* offsets, int offset, float eps, int io_dtype,
                           cudaStream_t stream);
BASED_WEAK int launch_delta_step(const void* x, const void* conv_w, void* ring, const float* a, const float* b, const float* A_log,
                      const float* dt_bias, const void* norm_w, float* state, void* out, int B, int H, int Hk, int d,
                      int dv, int taps, int64_t sx, int64_t sg, int64_t so, const int32_t* offsets, int offset, float eps,
                      int io_dtype, cudaStream_t stream);
BASED_WEAK int launch_rglru(const void* u, const void* y, const float* gates, const void* rb, const void* ib, const float* lam,
                 float* state, void* out, int B, int L, int W, int bw, Strides2 su, Strides2 sy, Strides2 so,
                 int64_t g_block, int64_t g_row, const int32_t* offsets, int offset, int io_dtype, cudaStream_t stream);

BASED_WEAK int launch_latent_prefill_tc(const void* q1, const void* q2, const void* k1, const void* k2, const void* v,
                             const void* gate, void* out, int B, int L, int T, int H, int d1, int d2, int dv, Strides3 sq1,
                             Strides3 sq2, Strides3 sk1, Strides3 sk2, Strides3 sv, Strides3 so, int64_t gb, int64_t gl,
                             const int32_t* offsets, int offset, float scale, cudaStream_t stream);
BASED_WEAK int read_tc_status_latent(unsigned int* out, int reset);
BASED_WEAK int latent_decode_splits(int B, int R, int max_len);
BASED_WEAK size_t latent_decode_scratch_bytes(int B, int R, int r, int max_len);
BASED_WEAK int launch_latent_decode(const void* q1, const void* q2, const void* cache, const void* gate, void* out, void* scratch,
                         size_t scratch_bytes, int B, int L, int H, int r, int rd, int max_len, Strides3 sq1, Strides3 sq2,
                         int64_t cb, int64_t cl, Strides3 so, int64_t gb, int64_t gl, const int32_t* offsets, int offset,
                         float scale, cudaStream_t stream);

BASED_WEAK int launch_delta_chunk(const void* q, const void* k, const void* v, const void* z, const float* a, const float* b,
                       const float* A_log, const float* dt_bias, const void* norm_w, float* state, void* out, void* scratch,
                       size_t scratch_bytes, int B, int L, int H, int Hk, int d, int dv, Strides2 sq, Strides2 sk,
                       Strides2 sv, Strides2 sz, Strides2 sg, Strides2 so, const int32_t* offsets, int offset, float eps,
                       cudaStream_t stream);
BASED_WEAK size_t delta_chunk_scratch_bytes(int B, int L, int H, int d, int dv);
BASED_WEAK int read_tc_status_delta(unsigned int* out, int reset);

BASED_WEAK int launch_rglru_tc(const void* u, const void* y, const void* w, const void* rb, const void* ib, const float* lam,
                    float* state, void* out, int B, int L, int W, int n, Strides2 su, Strides2 sy, Strides2 so,
                    const int32_t* offsets, int offset, cudaStream_t stream);
BASED_WEAK int read_tc_status_rglru(unsigned int* out, int reset);

// Post-norm stream, grouped attention over keys that are the values, linear attention with a constant decay.
int launch_stream_post_norm(const void* branch, int64_t sb, const void* w, float* residual, const void* w_out, void* out,
                            int64_t M, int D, float eps, int io_dtype, cudaStream_t stream);
int launch_stream_embed(const int64_t* tokens, const void* table, int64_t V, float scale, const void* pos, int64_t P,
                        float* residual, void* out, int B, int L, int D, const int32_t* offsets, int offset, int io_dtype,
                        cudaStream_t stream);
int launch_norm_gate(const void* x, int64_t sx, const void* w, const void* gate, int64_t sg, void* out, int64_t so, int64_t M,
                     int D, float eps, int io_dtype, cudaStream_t stream);
int launch_token_gate(const void* z, int64_t sz, const int64_t* tokens, const void* table, int64_t V, int64_t st,
                      int64_t column, void* out, int64_t M, int n, int io_dtype, cudaStream_t stream);
BASED_WEAK int launch_token_side(const void* x, int64_t sx, const int64_t* tokens, const void* wg, const void* wp, const void* table,
                                 int64_t V, int64_t st, int64_t column, const void* norm, float* residual, const void* out_norm,
                                 void* out, int M, int W, int n, float eps, cudaStream_t stream);
BASED_WEAK int launch_tied_prepare(void* q, const void* k, const void* wq, const void* wk, void* cache, float* factor, int B,
                                   int L, int H, int G, int d, int max_len, int64_t qb, int64_t ql, int64_t kb, int64_t kl,
                                   int64_t cb, int64_t cl, int64_t fb, int64_t fh, const int32_t* offsets, int offset,
                                   float eps, float coef, float every, int io_dtype, cudaStream_t stream);
BASED_WEAK int launch_tied_prefill_tc(const void* q, const void* cache, const float* factor, const void* gate, void* out, int B,
                                      int L, int H, int G, int d, int64_t qb, int64_t ql, int64_t cb, int64_t cl, int64_t fb,
                                      int64_t fh, int64_t gb, int64_t gl, int64_t ob, int64_t ol, int offset, float scale,
                                      float sink, cudaStream_t stream);
BASED_WEAK int read_tc_status_tied(unsigned int* out, int reset);
BASED_WEAK int read_tc_status_tied_decode(unsigned int* out, int reset);
BASED_WEAK size_t tied_decode_scratch_bytes(int B, int R, int G, int d, int max_len);
BASED_WEAK int launch_tied_decode(const void* q, const void* cache, const float* factor, const void* gate, void* out,
                                  void* scratch, size_t scratch_bytes, int* count, int count_len, int B, int L, int H, int G,
                                  int d, int max_len, int64_t qb, int64_t ql, int64_t cb, int64_t cl, int64_t fb, int64_t fh,
                                  int64_t gb, int64_t gl, int64_t ob, int64_t ol, const int32_t* offsets, int offset,
                                  float scale, float sink, cudaStream_t stream);
BASED_WEAK int launch_lightning_recurrent(const void* q, const void* k, const void* v, const float* decay, float* state,
                                          void* out, int B, int L, int H, int d, int dv, Strides2 sq, Strides2 sk, Strides2 sv,
                                          Strides2 so, const int32_t* offsets, int offset, int io_dtype, cudaStream_t stream);
BASED_WEAK int launch_lightning_tc(const void* q, const void* k, const void* v, const float* decay, float* state, void* out, int B,
                                   int L, int H, int d, int dv, Strides2 sq, Strides2 sk, Strides2 sv, Strides2 so,
                                   const int32_t* offsets, int offset, cudaStream_t stream);
BASED_WEAK int read_tc_status_lightning(unsigned int* out, int reset);
BASED_WEAK int launch_lightning_step(const void* q, const void* k, const void* v, const void* gate, int64_t sx,
                                     const float* decay, const void* norm_w, float* state, float* read, int* count, void* out,
                                     int64_t so, int B, int H, int d, int dv, const int32_t* offsets, int offset, float eps,
                                     int io_dtype, cudaStream_t stream);

}  // namespace based
