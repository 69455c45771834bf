// Real-gated linear recurrent unit, fp32 state, one channel per thread:
//   r = sigmoid(gr + br), i = sigmoid(gi + bi), log a = -8 r softplus(lam), a = exp(log a)
//   S <- a S + sqrt(1 - a^2) i u,     out = S * gelu_tanh(y)
// gr, gi are the fp32 products of the block-diagonal gate matrices with u (biases are added here).  Any L; a call
// whose first token is position 0 starts from zero whatever the state buffer holds.
#include <initializer_list>

#include "seq_common.cuh"

namespace based {
namespace {

using namespace seq;

struct RgP {
  const void *u, *y, *rb, *ib;
  const float *gates, *lam;
  float* state;                  // [B, W]
  void* out;
  const int32_t* offsets;
  int offset, B, L, W, bw;       // bw: width of one block
  Strides2 su, sy, so;           // .b batch, .h token
  int64_t g_block, g_row;        // gates: (block, row = b L + l, r_0..r_bw-1 i_0..i_bw-1)
};

constexpr int kThreads = 64;

template <typename T, int U>
__global__ void __launch_bounds__(kThreads) rglru_kernel(const RgP p) {
  const int c = blockIdx.x * kThreads + threadIdx.x, b = blockIdx.y;
  if (c >= p.W) return;
  const int blk = c / p.bw, j = c - blk * p.bw;
  const T* u = static_cast<const T*>(p.u) + b * p.su.b + c;
  const T* y = static_cast<const T*>(p.y) + b * p.sy.b + c;
  T* out = static_cast<T*>(p.out) + b * p.so.b + c;
  const float* gt = p.gates + blk * p.g_block + (int64_t)b * p.L * p.g_row + j;
  const float rb = to_float<T>(static_cast<const T*>(p.rb)[c]), ib = to_float<T>(static_cast<const T*>(p.ib)[c]);
  const float decay = -8.0f * softplus_acc(p.lam[c]);
  float S = position0(p.offsets, p.offset, b) == 0 ? 0.f : p.state[(int64_t)b * p.W + c];
  for (int l0 = 0; l0 < p.L; l0 += U) {
    float uv[U], yv[U], gr[U], gi[U];
#pragma unroll
    for (int t = 0; t < U; ++t)
      if (l0 + t < p.L) {
        uv[t] = to_float<T>(u[(l0 + t) * p.su.h]);
        yv[t] = to_float<T>(y[(l0 + t) * p.sy.h]);
        gr[t] = gt[(l0 + t) * p.g_row];
        gi[t] = gt[(l0 + t) * p.g_row + p.bw];
      }
#pragma unroll
    for (int t = 0; t < U; ++t)
      if (l0 + t < p.L) {
        const float la = decay * sigmoid_acc(gr[t] + rb);
        const float in = sqrtf(-expm1f(2.0f * la)) * sigmoid_acc(gi[t] + ib) * uv[t];
        S = fmaf(expf(la), S, in);
        out[(l0 + t) * p.so.h] = from_float<T>(S * gelu_tanh_t<T>(yv[t]));
      }
  }
  p.state[(int64_t)b * p.W + c] = S;
}

}  // namespace

int launch_rglru(const void* u, const void* y, const float* gates, const void* rb, const void* ib, const float* lam,
                 float* state, void* out, int B, int L, int W, int bw, Strides2 su, Strides2 sy, Strides2 so,
                 int64_t g_block, int64_t g_row, const int32_t* offsets, int offset, int io_dtype, cudaStream_t stream) {
  if (B > 65535) return BASED_ERR_TOO_LARGE;
  const RgP p{u, y, rb, ib, gates, lam, state, out, offsets, offset, B, L, W, bw, su, sy, so, g_block, g_row};
  const dim3 grid((W + kThreads - 1) / kThreads, B);
  if (io_dtype == BASED_BF16) {
    if (L == 1) rglru_kernel<__nv_bfloat16, 1><<<grid, kThreads, 0, stream>>>(p);
    else rglru_kernel<__nv_bfloat16, 8><<<grid, kThreads, 0, stream>>>(p);
  } else {
    if (L == 1) rglru_kernel<float, 1><<<grid, kThreads, 0, stream>>>(p);
    else rglru_kernel<float, 8><<<grid, kThreads, 0, stream>>>(p);
  }
  return (int)cudaGetLastError();
}

}  // namespace based
