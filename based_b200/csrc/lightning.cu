// Linear attention with one constant decay per head, fp32 state, on CUDA cores.  With q, k, v = silu of the projections:
//   S_t = decay S_(t-1) + k_t v_t^T;   o_t = S_t^T q_t
//  * lightning_recurrent: token by token for any sizes (fp32 models, short portions, sizes the chunked kernel does not
//    take).  A CTA owns 32 value columns of one head, lane = column, and keeps its part of the state in registers.
//  * lightning_step: a decode step from the packed projection to the normed, gated output in ONE launch.  HBM-bound: one
//    read and one write of the state, all loads of a thread in flight first.  The output norm runs over all heads of a
//    token, so the CTA that finishes a token's last columns does it; the others have left (nobody waits).
// A sequence's first token (position 0) starts from zero whatever the state buffer holds.
#include <initializer_list>

#include "seq_common.cuh"

namespace based {
namespace {

using namespace seq;

constexpr int kThreads = 256, kWarps = kThreads / 32;

struct RecP {
  const void *q, *k, *v;       // [B, L, H * d], [B, L, H * d], [B, L, H * dv], before silu
  const float* decay;          // [H]
  float* state;                // [B, H, d, dv]
  void* out;                   // [B, L, H * dv]
  const int32_t* offsets;
  int offset, L, H, d, dv;
  Strides2 sq, sk, sv, so;     // .b batch, .h token
};

// ROWS: state rows per warp, d <= 8 * ROWS
template <typename T, int ROWS>
__global__ void __launch_bounds__(kThreads) lightning_recurrent_kernel(const RecP p) {
  constexpr int kTok = ROWS > 32 ? 4 : 16;   // tokens per shared-memory chunk
  __shared__ float qs[kTok][kWarps * ROWS], ks[kTok][kWarps * ROWS], part[kTok][kWarps][32];
  const int h = blockIdx.x, b = blockIdx.y, e = blockIdx.z * 32 + (threadIdx.x & 31), lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const bool live = e < p.dv;
  const int i0 = warp * ROWS;
  float* st = p.state + (((int64_t)b * p.H + h) * p.d) * p.dv + e;
  const bool fresh = position0(p.offsets, p.offset, b) == 0;
  const float g = p.decay[h];
  float S[ROWS];
#pragma unroll
  for (int i = 0; i < ROWS; ++i) S[i] = !fresh && live && i0 + i < p.d ? st[(int64_t)(i0 + i) * p.dv] : 0.f;
  const T* q = static_cast<const T*>(p.q) + b * p.sq.b + (int64_t)h * p.d;
  const T* k = static_cast<const T*>(p.k) + b * p.sk.b + (int64_t)h * p.d;
  const T* v = static_cast<const T*>(p.v) + b * p.sv.b + (int64_t)h * p.dv + e;
  T* out = static_cast<T*>(p.out) + b * p.so.b + (int64_t)h * p.dv;
  for (int l0 = 0; l0 < p.L; l0 += kTok) {
    const int n = min(kTok, p.L - l0);
    for (int t = 0; t < n; ++t)
      for (int c = threadIdx.x; c < kWarps * ROWS; c += kThreads) {   // rows past d stay zero
        qs[t][c] = c < p.d ? silu_t<T>(to_float<T>(q[(l0 + t) * p.sq.h + c])) : 0.f;
        ks[t][c] = c < p.d ? silu_t<T>(to_float<T>(k[(l0 + t) * p.sk.h + c])) : 0.f;
      }
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      const float x = live ? silu_t<T>(to_float<T>(v[(l0 + t) * p.sv.h])) : 0.f;
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < ROWS; ++i) {
        S[i] = fmaf(ks[t][i0 + i], x, g * S[i]);
        o = fmaf(S[i], qs[t][i0 + i], o);
      }
      part[t][warp][lane] = o;
    }
    __syncthreads();
    for (int c = threadIdx.x; c < n * 32; c += kThreads) {
      const int t = c >> 5, j = c & 31, col = blockIdx.z * 32 + j;
      float o = 0.f;
#pragma unroll
      for (int w = 0; w < kWarps; ++w) o += part[t][w][j];
      if (col < p.dv) out[(l0 + t) * p.so.h + col] = from_float<T>(o);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < ROWS; ++i)
    if (live && i0 + i < p.d) st[(int64_t)(i0 + i) * p.dv] = S[i];
}

template <typename T>
int launch_rec_t(const RecP& p, int B, cudaStream_t st) {
  const dim3 grid(p.H, B, (p.dv + 31) / 32);
  if (p.d <= 32) lightning_recurrent_kernel<T, 4><<<grid, kThreads, 0, st>>>(p);
  else if (p.d <= 64) lightning_recurrent_kernel<T, 8><<<grid, kThreads, 0, st>>>(p);
  else if (p.d <= 128) lightning_recurrent_kernel<T, 16><<<grid, kThreads, 0, st>>>(p);
  else if (p.d <= 256) lightning_recurrent_kernel<T, 32><<<grid, kThreads, 0, st>>>(p);
  else if (p.d <= 512) lightning_recurrent_kernel<T, 64><<<grid, kThreads, 0, st>>>(p);
  else return BASED_ERR_SHAPE;
  return (int)cudaGetLastError();
}

struct StepP {
  const void *q, *k, *v, *gate, *norm_w;   // [B, H d], [B, H d], [B, H dv], [B, H dv] (rows sx apart), [H dv]
  const float* decay;
  float *state, *read;                     // [B, H, d, dv]; [B, H dv] read-outs before the norm
  int* count;                              // [B], zero between launches
  void* out;                               // [B, H dv], rows so apart
  const int32_t* offsets;
  int64_t sx, so;
  int offset, H, d, dv, cols, late;
  float eps;
};

// A CTA owns p.cols value columns of one head (a multiple of 4), a thread four of them in every R-th state row.  Up to V rows
// are in flight.
template <typename T, int V>
__global__ void __launch_bounds__(kThreads, V <= 8 ? 3 : 2) lightning_step_kernel(const StepP p) {
  extern __shared__ float sm[];
  const int h = blockIdx.x, b = blockIdx.y, col0 = blockIdx.z * p.cols, tid = threadIdx.x;
  const int quads = p.cols / 4, R = kThreads / quads, row4 = p.dv / 4;
  const int c = tid % quads, rg = tid / quads;
  const bool mine = rg < R;
  float *qs = sm, *ks = qs + p.d, *vs = ks + p.d, *part = vs + p.cols;   // part [R][cols]
  float4* st = reinterpret_cast<float4*>(p.state + ((int64_t)b * p.H + h) * p.d * p.dv + col0) + c;
  float4 s[V];
  auto fetch = [&](int i0) {
#pragma unroll
    for (int v = 0; v < V; ++v) {
      const int i = i0 + rg + v * R;
      s[v] = mine && i < p.d ? st[(int64_t)i * row4] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  fetch(0);                            // whatever the position: a sequence that starts drops the values
  // few CTAs: a state that is whole in registers is stored behind the read-out, off its way
  const bool keep = p.late && p.d <= V * R;
  if (tid < (p.cols * (int)sizeof(T) + 127) / 128)   // for whichever CTA will need them
    asm volatile("prefetch.global.L2 [%0];" ::"l"(static_cast<const char*>(p.norm_w) + ((int64_t)h * p.dv + col0) * sizeof(T) + tid * 128));
  const T *q = static_cast<const T*>(p.q) + b * p.sx + (int64_t)h * p.d, *k = static_cast<const T*>(p.k) + b * p.sx + (int64_t)h * p.d;
  const T* v = static_cast<const T*>(p.v) + b * p.sx + (int64_t)h * p.dv + col0;
  for (int i = tid; i < 2 * p.d + p.cols; i += kThreads) {
    const T* src = i < p.d ? q + i : i < 2 * p.d ? k + (i - p.d) : v + (i - 2 * p.d);
    sm[i] = silu_t<T>(to_float<T>(*src));
  }
  const bool fresh = position0(p.offsets, p.offset, b) == 0;
  __syncthreads();
  const float g = p.decay[h];
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  if (mine) {
    const float4 x = make_float4(vs[4 * c], vs[4 * c + 1], vs[4 * c + 2], vs[4 * c + 3]);
    for (int i0 = 0; i0 < p.d; i0 += V * R) {
      if (i0) fetch(i0);
#pragma unroll
      for (int n = 0; n < V; ++n) {
        const int i = i0 + rg + n * R;
        if (i < p.d) {
          const float kk = ks[i], qq = qs[i];
          if (fresh) s[n] = make_float4(0.f, 0.f, 0.f, 0.f);
          s[n].x = fmaf(kk, x.x, g * s[n].x); s[n].y = fmaf(kk, x.y, g * s[n].y);
          s[n].z = fmaf(kk, x.z, g * s[n].z); s[n].w = fmaf(kk, x.w, g * s[n].w);
          if (!keep) st[(int64_t)i * row4] = s[n];
          o.x = fmaf(s[n].x, qq, o.x); o.y = fmaf(s[n].y, qq, o.y);
          o.z = fmaf(s[n].z, qq, o.z); o.w = fmaf(s[n].w, qq, o.w);
        }
      }
    }
    float* dst = part + rg * p.cols + 4 * c;
    dst[0] = o.x; dst[1] = o.y; dst[2] = o.z; dst[3] = o.w;
  }
  __syncthreads();
  const int D = p.H * p.dv;
  float* read = p.read + (int64_t)b * D;
  for (int e = tid; e < p.cols; e += kThreads) {
    float y = 0.f;
    for (int r = 0; r < R; ++r) y += part[r * p.cols + e];
    read[h * p.dv + col0 + e] = y;
  }
  // the CTA that gets here last norms the token
  __shared__ int last;
  __shared__ float red[kWarps];
  __threadfence();
  __syncthreads();
  if (tid == 0) {
    last = atomicAdd(p.count + b, 1) == p.H * (int)gridDim.z - 1;
    if (last) p.count[b] = 0;
  }
  if (keep && mine) {
#pragma unroll
    for (int n = 0; n < V; ++n)
      if (rg + n * R < p.d) st[(int64_t)(rg + n * R) * row4] = s[n];
  }
  __syncthreads();
  if (!last) return;
  __threadfence();
  const T* gate = static_cast<const T*>(p.gate) + b * p.sx;
  const T* w = static_cast<const T*>(p.norm_w);
  T* out = static_cast<T*>(p.out) + b * p.so;
  constexpr int kHeld = 8;             // of a thread's values: asked for together
  float y[kHeld], z[kHeld], u[kHeld], ss = 0.f;
#pragma unroll
  for (int i = 0; i < kHeld; ++i) {
    const int e = tid + i * kThreads;
    y[i] = e < D ? __ldcg(read + e) : 0.f;
    z[i] = e < D ? to_float<T>(gate[e]) : 0.f;
    u[i] = e < D ? to_float<T>(w[e]) : 0.f;
  }
#pragma unroll
  for (int i = 0; i < kHeld; ++i) ss = fmaf(y[i], y[i], ss);
  for (int e = tid + kHeld * kThreads; e < D; e += kThreads) { const float x = __ldcg(read + e); ss = fmaf(x, x, ss); }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < kWarps; ++i) ss += red[i];
  const float rstd = rsqrtf(ss / (float)D + p.eps);
#pragma unroll
  for (int i = 0; i < kHeld; ++i)
    if (tid + i * kThreads < D) out[tid + i * kThreads] = from_float<T>(y[i] * rstd * u[i] * sigmoid_t<T>(z[i]));
  for (int e = tid + kHeld * kThreads; e < D; e += kThreads)
    out[e] = from_float<T>(__ldcg(read + e) * rstd * to_float<T>(w[e]) * sigmoid_t<T>(to_float<T>(gate[e])));
}

template <typename T>
int launch_step_t(const StepP& p, int B, cudaStream_t st) {
  const int quads = p.cols / 4, R = kThreads / quads, rows = (p.d + R - 1) / R;
  const size_t smem = sizeof(float) * (2 * p.d + p.cols + (size_t)R * p.cols);
  const dim3 grid(p.H, B, p.dv / p.cols);
  if (rows <= 2) lightning_step_kernel<T, 2><<<grid, kThreads, smem, st>>>(p);
  else if (rows <= 4) lightning_step_kernel<T, 4><<<grid, kThreads, smem, st>>>(p);
  else if (rows <= 8) lightning_step_kernel<T, 8><<<grid, kThreads, smem, st>>>(p);
  else lightning_step_kernel<T, 16><<<grid, kThreads, smem, st>>>(p);
  return (int)cudaGetLastError();
}

}  // namespace

int launch_lightning_recurrent(const void* q, const void* k, const void* v, const float* decay, float* state, void* out, int B,
                               int L, int H, int d, int dv, Strides2 sq, Strides2 sk, Strides2 sv, Strides2 so,
                               const int32_t* offsets, int offset, int io_dtype, cudaStream_t stream) {
  if (B > 65535 || (dv + 31) / 32 > 65535) return BASED_ERR_TOO_LARGE;
  const RecP p{q, k, v, decay, state, out, offsets, offset, L, H, d, dv, sq, sk, sv, so};
  return io_dtype == BASED_BF16 ? launch_rec_t<__nv_bfloat16>(p, B, stream) : launch_rec_t<float>(p, B, stream);
}

int launch_lightning_step(const void* q, const void* k, const void* v, const void* gate, int64_t sx, const float* decay,
                          const void* norm_w, float* state, float* read, int* count, void* out, int64_t so, int B, int H, int d,
                          int dv, const int32_t* offsets, int offset, float eps, int io_dtype, cudaStream_t stream) {
  if (dv % 4 || dv > 4 * kThreads || d > 1024 || H > 65535 || !aligned16(state)) return BASED_ERR_IMPL;
  if (B > 65535) return BASED_ERR_TOO_LARGE;
  const bool few = (int64_t)B * H < 8 * 148;
  int cols = dv;   // few heads: slices of their columns, several CTAs per SM
  while (few && cols % 8 == 0 && cols / 2 >= 64) cols /= 2;
  const StepP p{q, k, v, gate, norm_w, decay, state, read, count, out, offsets, sx, so, offset, H, d, dv, cols, few, eps};
  return io_dtype == BASED_BF16 ? launch_step_t<__nv_bfloat16>(p, B, stream) : launch_step_t<float>(p, B, stream);
}

}  // namespace based
