// Gated delta rule on CUDA cores, fp32 state.  Per head, with unit vectors k and q (q also times d^-1/2):
//   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q;   g = exp(-exp(A_log) softplus(a + dt_bias))
// followed by the output norm and gate: out = o / rms(o) * w * silu(z).  Head h uses query / key head h / (H / Hk).
//
//  * delta_recurrent: token by token for any L and any sizes (fp32 models, sizes the chunked kernel does not take).
//  * delta_step: a decode step from the packed projection to the gated output in ONE launch: short convolution over
//    the input ring, silu, unit norms, gates, state update, read-out, output norm and gate.  One read and one write
//    of the state (HBM-bound); every state load is in flight before the first dependent instruction.
// A sequence's first token (position 0) starts from zero whatever the state and ring buffers hold.
#include <initializer_list>

#include "seq_common.cuh"

namespace based {
namespace {

using namespace seq;

constexpr float kUnitEps = 1e-6f;
constexpr int kThreads = 256;

__device__ __forceinline__ float block_sum256(float v, float* part) {  // every thread gets the sum; part: 8 floats
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int w = 0; w < kThreads / 32; ++w) t += part[w];
  return t;
}

struct DeltaP {
  const void *q, *k, *v, *z, *norm_w;
  const float *a, *b, *A_log, *dt_bias;   // a, b: [B, L, H] pre-activations
  float* state;                           // [B, H, d, dv]
  void* out;
  const int32_t* offsets;
  int offset, B, L, H, Hk, d, dv, state_in_smem;
  Strides2 sq, sk, sv, sz, sg, so;        // .b batch, .h token; heads contiguous inside a token
  float eps;
};

template <typename T>
__global__ void __launch_bounds__(kThreads) delta_recurrent_kernel(const DeltaP p) {
  extern __shared__ float sm[];
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int hk = h / (p.H / p.Hk);
  const int d = p.d, dv = p.dv;
  const int Cw = min(dv, kThreads), R = max(1, kThreads / dv);
  const int e0 = tid % Cw, rg = tid / Cw;
  const bool active = rg < R;
  float* ks = sm;             // [d]
  float* qs = ks + d;         // [d]
  float* os = qs + d;         // [dv]
  float* part = os + dv;      // [R][dv]
  float* red = part + R * dv; // [8]
  float* gst = p.state + ((int64_t)b * p.H + h) * d * dv;
  float* S = p.state_in_smem ? red + 8 : gst;
  const bool fresh = position0(p.offsets, p.offset, b) == 0;
  if (p.state_in_smem || fresh)
    for (int i = tid; i < d * dv; i += kThreads) S[i] = fresh ? 0.f : gst[i];
  __syncthreads();
  const float A = expf(p.A_log[h]), dt = p.dt_bias[h], qscale = rsqrtf((float)d);
  for (int l = 0; l < p.L; ++l) {
    const T* q = static_cast<const T*>(p.q) + b * p.sq.b + l * p.sq.h + (int64_t)hk * d;
    const T* k = static_cast<const T*>(p.k) + b * p.sk.b + l * p.sk.h + (int64_t)hk * d;
    const T* v = static_cast<const T*>(p.v) + b * p.sv.b + l * p.sv.h + (int64_t)h * dv;
    float nq = 0.f, nk = 0.f;
    for (int i = tid; i < d; i += kThreads) {
      const float x = to_float<T>(q[i]), y = to_float<T>(k[i]);
      qs[i] = x; ks[i] = y;
      nq = fmaf(x, x, nq); nk = fmaf(y, y, nk);
    }
    nq = rsqrtf(block_sum256(nq, red) + kUnitEps) * qscale;
    nk = rsqrtf(block_sum256(nk, red) + kUnitEps);
    const int64_t gi = b * p.sg.b + l * p.sg.h + h;
    const float g = expf(-A * softplus_acc(p.a[gi] + dt)), beta = sigmoid_acc(p.b[gi]);
    if (active)
      for (int e = e0; e < dv; e += Cw) {
        float s = 0.f;
        for (int i = rg; i < d; i += R) s = fmaf(S[(int64_t)i * dv + e], ks[i], s);
        part[rg * dv + e] = s;
      }
    __syncthreads();
    float u_keep = 0.f;
    if (active)
      for (int e = e0; e < dv; e += Cw) {
        float s = 0.f;
        for (int r = 0; r < R; ++r) s += part[r * dv + e];
        const float u = beta * (to_float<T>(v[e]) - g * nk * s);
        float o = 0.f;
        for (int i = rg; i < d; i += R) {
          const float x = fmaf(ks[i] * nk, u, g * S[(int64_t)i * dv + e]);
          S[(int64_t)i * dv + e] = x;
          o = fmaf(x, qs[i], o);
        }
        if (R == 1) os[e] = o * nq;
        u_keep = o;
      }
    if (R > 1) {
      __syncthreads();   // every partial sum has been read
      if (active) part[rg * dv + e0] = u_keep;
      __syncthreads();
      if (tid < dv) {
        float o = 0.f;
        for (int r = 0; r < R; ++r) o += part[r * dv + tid];
        os[tid] = o * nq;
      }
    }
    __syncthreads();
    float ss = 0.f;
    for (int e = tid; e < dv; e += kThreads) ss = fmaf(os[e], os[e], ss);
    const float rstd = rsqrtf(block_sum256(ss, red) / (float)dv + p.eps);
    const T* z = static_cast<const T*>(p.z) + b * p.sz.b + l * p.sz.h + (int64_t)h * dv;
    T* out = static_cast<T*>(p.out) + b * p.so.b + l * p.so.h + (int64_t)h * dv;
    for (int e = tid; e < dv; e += kThreads)
      out[e] = from_float<T>(os[e] * rstd * to_float<T>(static_cast<const T*>(p.norm_w)[e]) * silu_t<T>(to_float<T>(z[e])));
    __syncthreads();
  }
  if (p.state_in_smem)
    for (int i = tid; i < d * dv; i += kThreads) gst[i] = S[i];
}

// ------------------------------------------------------------------ decode step
struct StepP {
  const void *x, *conv_w, *norm_w;        // x [B, 2 Hk d + 2 H dv]: q | k | v | z; conv_w [2 Hk d + H dv, taps]
  void* ring;                             // [B, taps, 2 Hk d + H dv]
  const float *a, *b, *A_log, *dt_bias;   // a, b: [B, H]
  float* state;
  void* out;
  const int32_t* offsets;
  int offset, B, H, Hk, d, dv, taps;
  int64_t sx, sg, so;
  float eps;
};

// NR float4 rows of the state per thread; thread t owns columns 4 (t mod dv/4) .. +3 of rows t / (dv/4), + R, ...
template <typename T, int NR>
__global__ void __launch_bounds__(kThreads, NR <= 8 ? 3 : NR <= 16 ? 2 : 1) delta_step_kernel(const StepP p) {
  extern __shared__ float sm[];
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int hk = h / (p.H / p.Hk);
  const int d = p.d, dv = p.dv, C4 = dv / 4, R = kThreads / C4;
  const int c4 = tid % C4, rg = tid / C4;
  const bool active = rg < R;
  const int pos = position0(p.offsets, p.offset, b);
  float4* st = reinterpret_cast<float4*>(p.state + ((int64_t)b * p.H + h) * d * dv);
  float4 s[NR];
#pragma unroll
  for (int n = 0; n < NR; ++n) {
    const int i = rg + n * R;
    s[n] = (active && i < d && pos > 0) ? __ldcs(st + (int64_t)i * C4 + c4) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  float* ks = sm;              // [d]
  float* qs = ks + d;          // [d]
  float* vs = qs + d;          // [dv]
  float* red = vs + dv;        // [24]: three 8-entry reductions
  float4* part = reinterpret_cast<float4*>(red + 24);  // [R][C4]
  const int C = 2 * p.Hk * d + p.H * dv;
  const T* x = static_cast<const T*>(p.x) + b * p.sx;
  T* ring = static_cast<T*>(p.ring) + (int64_t)b * p.taps * C;
  float nq = 0.f, nk = 0.f;
  for (int n = tid; n < 2 * d + dv; n += kThreads) {
    const int c = n < d ? hk * d + n : n < 2 * d ? p.Hk * d + hk * d + (n - d) : 2 * p.Hk * d + h * dv + (n - 2 * d);
    const T* w = static_cast<const T*>(p.conv_w) + (int64_t)c * p.taps;
    const T xc = x[c];
    float y = 0.f;
    for (int j = 0; j < p.taps - 1; ++j) {
      const int pp = pos - (p.taps - 1) + j;
      if (pp >= 0) y = fmaf(to_float<T>(w[j]), to_float<T>(ring[(int64_t)(pp % p.taps) * C + c]), y);
    }
    y = fmaf(to_float<T>(w[p.taps - 1]), to_float<T>(xc), y);
    y = to_float<T>(from_float<T>(silu_t<T>(y)));   // the prompt pass stores this value in the activations' dtype
    ring[(int64_t)(pos % p.taps) * C + c] = xc;     // heads that share a query / key head store the same value
    if (n < d) { qs[n] = y; nq = fmaf(y, y, nq); }
    else if (n < 2 * d) { ks[n - d] = y; nk = fmaf(y, y, nk); }
    else vs[n - 2 * d] = y;
  }
  nq = warp_sum(nq); nk = warp_sum(nk);
  if ((tid & 31) == 0) { red[tid >> 5] = nq; red[8 + (tid >> 5)] = nk; }
  const float A = expf(p.A_log[h]);
  const float g = expf(-A * softplus_acc(p.a[b * p.sg + h] + p.dt_bias[h])), beta = sigmoid_acc(p.b[b * p.sg + h]);
  __syncthreads();
  nq = 0.f; nk = 0.f;
#pragma unroll
  for (int w = 0; w < kThreads / 32; ++w) { nq += red[w]; nk += red[8 + w]; }
  nq = rsqrtf(nq + kUnitEps) * rsqrtf((float)d);
  nk = rsqrtf(nk + kUnitEps);
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int n = 0; n < NR; ++n) {
    const int i = rg + n * R;
    if (active && i < d) {
      const float k = ks[i];
      s[n].x *= g; s[n].y *= g; s[n].z *= g; s[n].w *= g;
      acc.x = fmaf(s[n].x, k, acc.x); acc.y = fmaf(s[n].y, k, acc.y);
      acc.z = fmaf(s[n].z, k, acc.z); acc.w = fmaf(s[n].w, k, acc.w);
    }
  }
  if (active) part[rg * C4 + c4] = acc;
  __syncthreads();
  float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
  if (active) {
    for (int r = 0; r < R; ++r) {
      const float4 t = part[r * C4 + c4];
      u.x += t.x; u.y += t.y; u.z += t.z; u.w += t.w;
    }
    // u holds S^T k; now the written value, with the unit norm of k folded into it for the outer product
    u.x = beta * (vs[4 * c4] - nk * u.x) * nk; u.y = beta * (vs[4 * c4 + 1] - nk * u.y) * nk;
    u.z = beta * (vs[4 * c4 + 2] - nk * u.z) * nk; u.w = beta * (vs[4 * c4 + 3] - nk * u.w) * nk;
  }
  acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int n = 0; n < NR; ++n) {
    const int i = rg + n * R;
    if (active && i < d) {
      const float k = ks[i], q = qs[i];
      s[n].x = fmaf(k, u.x, s[n].x); s[n].y = fmaf(k, u.y, s[n].y);
      s[n].z = fmaf(k, u.z, s[n].z); s[n].w = fmaf(k, u.w, s[n].w);
      __stcs(st + (int64_t)i * C4 + c4, s[n]);
      acc.x = fmaf(s[n].x, q, acc.x); acc.y = fmaf(s[n].y, q, acc.y);
      acc.z = fmaf(s[n].z, q, acc.z); acc.w = fmaf(s[n].w, q, acc.w);
    }
  }
  __syncthreads();
  if (active) part[rg * C4 + c4] = acc;
  __syncthreads();
  float ss = 0.f;
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  if (tid < C4) {
    for (int r = 0; r < R; ++r) {
      const float4 t = part[r * C4 + tid];
      o.x += t.x; o.y += t.y; o.z += t.z; o.w += t.w;
    }
    o.x *= nq; o.y *= nq; o.z *= nq; o.w *= nq;
    ss = o.x * o.x + o.y * o.y + o.z * o.z + o.w * o.w;
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[16 + (tid >> 5)] = ss;
  __syncthreads();
  if (tid < C4) {
    float tot = 0.f;
#pragma unroll
    for (int w = 0; w < kThreads / 32; ++w) tot += red[16 + w];
    const float rstd = rsqrtf(tot / (float)dv + p.eps);
    const T* z = x + C + (int64_t)h * dv + 4 * tid;
    const T* nw = static_cast<const T*>(p.norm_w) + 4 * tid;
    T* out = static_cast<T*>(p.out) + b * p.so + (int64_t)h * dv + 4 * tid;
    const float ov[4] = {o.x, o.y, o.z, o.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) out[e] = from_float<T>(ov[e] * rstd * to_float<T>(nw[e]) * silu_t<T>(to_float<T>(z[e])));
  }
}

template <typename T>
int launch_step_t(const StepP& p, cudaStream_t st) {
  const int C4 = p.dv / 4, R = kThreads / C4, nr = (p.d + R - 1) / R;
  const size_t smem = sizeof(float) * (2 * p.d + p.dv + 24) + sizeof(float4) * R * C4;
  const dim3 grid(p.H, p.B);
  if (nr <= 1) delta_step_kernel<T, 1><<<grid, kThreads, smem, st>>>(p);
  else if (nr <= 2) delta_step_kernel<T, 2><<<grid, kThreads, smem, st>>>(p);
  else if (nr <= 4) delta_step_kernel<T, 4><<<grid, kThreads, smem, st>>>(p);
  else if (nr <= 8) delta_step_kernel<T, 8><<<grid, kThreads, smem, st>>>(p);
  else if (nr <= 16) delta_step_kernel<T, 16><<<grid, kThreads, smem, st>>>(p);
  else delta_step_kernel<T, 32><<<grid, kThreads, smem, st>>>(p);
  return (int)cudaGetLastError();
}

template <typename T>
int launch_recurrent_t(DeltaP p, cudaStream_t st) {
  const int R = p.dv < kThreads ? kThreads / p.dv : 1;
  size_t floats = 2 * (size_t)p.d + p.dv + (size_t)R * p.dv + 8;
  p.state_in_smem = (floats + (size_t)p.d * p.dv) * 4 <= 200 * 1024;
  if (p.state_in_smem) floats += (size_t)p.d * p.dv;
  if (floats * 4 > 200 * 1024) return BASED_ERR_SHAPE;
  const cudaError_t e = cudaFuncSetAttribute(delta_recurrent_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
  if (e != cudaSuccess) return (int)e;
  delta_recurrent_kernel<T><<<dim3(p.H, p.B), kThreads, floats * 4, st>>>(p);
  return (int)cudaGetLastError();
}

}  // namespace

int launch_delta_recurrent(const void* q, const void* k, const void* v, const void* z, const float* a, const float* b,
                           const float* A_log, const float* dt_bias, const void* norm_w, float* state, void* out, int B,
                           int L, int H, int Hk, int d, int dv, Strides2 sq, Strides2 sk, Strides2 sv, Strides2 sz,
                           Strides2 sg, Strides2 so, const int32_t* offsets, int offset, float eps, int io_dtype,
                           cudaStream_t stream) {
  if (B > 65535) return BASED_ERR_TOO_LARGE;
  const DeltaP p{q, k, v, z, norm_w, a, b, A_log, dt_bias, state, out, offsets, offset, B, L, H, Hk, d, dv, 0,
                 sq, sk, sv, sz, sg, so, eps};
  return io_dtype == BASED_BF16 ? launch_recurrent_t<__nv_bfloat16>(p, stream) : launch_recurrent_t<float>(p, stream);
}

int launch_delta_step(const void* x, const void* conv_w, void* ring, const float* a, const float* b, const float* A_log,
                      const float* dt_bias, const void* norm_w, float* state, void* out, int B, int H, int Hk, int d,
                      int dv, int taps, int64_t sx, int64_t sg, int64_t so, const int32_t* offsets, int offset, float eps,
                      int io_dtype, cudaStream_t stream) {
  if (B > 65535) return BASED_ERR_TOO_LARGE;
  if (dv % 4 != 0 || dv > 4 * kThreads || !aligned16(state)) return BASED_ERR_IMPL;
  const int R = kThreads / (dv / 4);
  if ((d + R - 1) / R > 32 || sizeof(float) * (2 * d + dv + 24 + 4 * kThreads) > 47 * 1024) return BASED_ERR_IMPL;
  // red (24 floats) is followed by a float4 array: keep it 16-byte aligned
  if ((2 * d + dv) % 4 != 0) return BASED_ERR_IMPL;
  const StepP p{x, conv_w, norm_w, ring, a, b, A_log, dt_bias, state, out, offsets, offset, B, H, Hk, d, dv, taps,
                sx, sg, so, eps};
  return io_dtype == BASED_BF16 ? launch_step_t<__nv_bfloat16>(p, stream) : launch_step_t<float>(p, stream);
}

}  // namespace based
