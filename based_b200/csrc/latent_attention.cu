// Latent attention, everything but the tensor-core kernels:
//  * latent_prepare: one launch between the projections and the attention of a layer.  Per token: RMSNorm of the
//    kv_rank latent values, rotation of the shared key part, both appended to the cache row of the token's position;
//    rotation of the rotated part of every query head in place.  Rotation tables are fp32 and so is the arithmetic.
//  * split_key_attention: causal softmax attention whose score is a sum of two dot products,
//    s = (q1 . k1 + q2 . k2) * scale, on CUDA cores with fp32 arithmetic, any sizes.  With k1 = per-head keys and
//    k2 = the shared rotated part it is the expanded form; with q1 = W_uk^T q and k1 = v = the cached latent
//    (head stride 0) it is the absorbed form.  fp32 models and sizes the tensor-core kernels do not take run here.
//    Options: groups of query heads that share a key head, a factor per key on its scores, a sink (a score of 0 without
//    a value in the softmax sum), an output gate per head or per element.
#include <initializer_list>

#include "seq_common.cuh"

namespace based {
namespace {

using namespace seq;

constexpr int kPrepThreads = 128;

struct PrepP {
  const void *z, *norm_w;      // [B, L, r + rd] or null (the layer reads another layer's cache)
  void *cache, *q;             // cache [B, maxL, r + rd]; q [B, L, H, d + rd] or null
  const float *cosv, *sinv;    // [table_len, rd / 2]
  const int32_t* offsets;
  int offset, B, L, H, r, rd, d, max_len, table_len;
  int64_t zb, zl, cb, cl, qb, ql;
  float eps;
};

template <typename T>
__global__ void __launch_bounds__(kPrepThreads) latent_prepare_kernel(const PrepP p) {
  const int l = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int pos = position0(p.offsets, p.offset, b) + l;
  if (pos < 0 || pos >= p.max_len || pos >= p.table_len) return;
  const int half = p.rd / 2;
  const float *cs = p.cosv + (int64_t)pos * half, *sn = p.sinv + (int64_t)pos * half;
  if (p.z) {
    const T* z = static_cast<const T*>(p.z) + b * p.zb + l * p.zl;
    T* row = static_cast<T*>(p.cache) + b * p.cb + (int64_t)pos * p.cl;
    float ss = 0.f;
    for (int c = tid; c < p.r; c += kPrepThreads) { const float v = to_float<T>(z[c]); ss = fmaf(v, v, ss); }
    ss = warp_sum(ss);
    __shared__ float part[kPrepThreads / 32];
    if ((tid & 31) == 0) part[tid >> 5] = ss;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int w = 0; w < kPrepThreads / 32; ++w) tot += part[w];
    const float rstd = rsqrtf(tot / (float)p.r + p.eps);
    for (int c = tid; c < p.r; c += kPrepThreads)
      row[c] = from_float<T>(to_float<T>(z[c]) * rstd * to_float<T>(static_cast<const T*>(p.norm_w)[c]));
    for (int i = tid; i < half; i += kPrepThreads) {
      const float u = to_float<T>(z[p.r + i]), v = to_float<T>(z[p.r + half + i]);
      row[p.r + i] = from_float<T>(u * cs[i] - v * sn[i]);
      row[p.r + half + i] = from_float<T>(v * cs[i] + u * sn[i]);
    }
  }
  if (p.q) {
    T* q = static_cast<T*>(p.q) + b * p.qb + l * p.ql + p.d;
    for (int e = tid; e < p.H * half; e += kPrepThreads) {
      const int h = e / half, i = e - h * half;
      T* x = q + (int64_t)h * (p.d + p.rd);
      const float u = to_float<T>(x[i]), v = to_float<T>(x[half + i]);
      x[i] = from_float<T>(u * cs[i] - v * sn[i]);
      x[half + i] = from_float<T>(v * cs[i] + u * sn[i]);
    }
  }
}

// ------------------------------------------------------------------ CUDA-core attention
constexpr int kWarps = 4;

struct AttnP {
  const void *q1, *q2, *k1, *k2, *v, *gate;
  void* out;
  const int32_t* offsets;
  int offset, B, L, H, d1, d2, dv;
  Strides3 sq1, sq2, sk1, sk2, sv, so;  // b, h, l
  int64_t gb, gl;                       // gate [B, L, H], or [B, L, H * dv] with x.gate_per_element
  float scale;
  AttentionOptions x;
};

// One warp per (query, head).  Lanes own keys for the scores of 32 keys at a time, then output channels for the
// weighted sum; running maximum and sum as usual.  NJ = ceil(dv / 32).
template <typename T, int NJ>
__global__ void __launch_bounds__(kWarps * 32) split_key_attention_kernel(const AttnP p) {
  extern __shared__ float sm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int dq = p.d1 + p.d2;
  float* q = sm + warp * dq;
  const int l = blockIdx.x * kWarps + warp, h = blockIdx.y, b = blockIdx.z;
  if (l >= p.L) return;
  const T* q1 = static_cast<const T*>(p.q1) + b * p.sq1.b + h * p.sq1.h + l * p.sq1.l;
  const T* q2 = static_cast<const T*>(p.q2) + b * p.sq2.b + h * p.sq2.h + l * p.sq2.l;
  for (int c = lane; c < dq; c += 32) q[c] = to_float<T>(c < p.d1 ? q1[c] : q2[c - p.d1]);
  __syncwarp();
  const int nk = position0(p.offsets, p.offset, b) + l + 1;
  const int g = h / p.x.group;
  const T* k1 = static_cast<const T*>(p.k1) + b * p.sk1.b + g * p.sk1.h;
  const T* k2 = static_cast<const T*>(p.k2) + b * p.sk2.b + g * p.sk2.h;
  const T* v = static_cast<const T*>(p.v) + b * p.sv.b + g * p.sv.h;
  const float* kf = p.x.key_factor ? p.x.key_factor + b * p.x.fb + g * p.x.fh : nullptr;
  float m = p.x.sink > 0.f ? 0.f : -INFINITY, sum = lane == 0 ? p.x.sink : 0.f, acc[NJ];
#pragma unroll
  for (int j = 0; j < NJ; ++j) acc[j] = 0.f;
  for (int t0 = 0; t0 < nk; t0 += 32) {
    const int t = t0 + lane;
    float s = -INFINITY;
    if (t < nk) {
      const T *a = k1 + (int64_t)t * p.sk1.l, *r = k2 + (int64_t)t * p.sk2.l;
      float x = 0.f;
      for (int c = 0; c < p.d1; ++c) x = fmaf(q[c], to_float<T>(a[c]), x);
      for (int c = 0; c < p.d2; ++c) x = fmaf(q[p.d1 + c], to_float<T>(r[c]), x);
      s = x * p.scale * (kf ? kf[t] : 1.0f);
    }
    const float mn = fmaxf(m, warp_max(s));
    const float corr = expf(m - mn), pr = expf(s - mn);
    sum = sum * corr + pr;   // this lane's share; lanes are added at the end
    m = mn;
#pragma unroll
    for (int j = 0; j < NJ; ++j) acc[j] *= corr;
    const int n = min(32, nk - t0);
    for (int u = 0; u < n; ++u) {
      const float pu = __shfl_sync(0xffffffffu, pr, u);
      const T* vr = v + (int64_t)(t0 + u) * p.sv.l;
#pragma unroll
      for (int j = 0; j < NJ; ++j)
        if (lane + 32 * j < p.dv) acc[j] = fmaf(pu, to_float<T>(vr[lane + 32 * j]), acc[j]);
    }
  }
  sum = warp_sum(sum);
  float f = 1.0f / sum;
  const T* gate = p.gate ? static_cast<const T*>(p.gate) + b * p.gb + l * p.gl : nullptr;
  if (gate && !p.x.gate_per_element) { f *= sigmoid_acc(to_float<T>(gate[h])); gate = nullptr; }
  if (gate) gate += (int64_t)h * p.dv;
  T* o = static_cast<T*>(p.out) + b * p.so.b + h * p.so.h + l * p.so.l;
#pragma unroll
  for (int j = 0; j < NJ; ++j)
    if (lane + 32 * j < p.dv) {
      const float gf = gate ? sigmoid_acc(to_float<T>(gate[lane + 32 * j])) : 1.0f;
      o[lane + 32 * j] = from_float<T>(acc[j] * f * gf);
    }
}

template <typename T>
int launch_attn_t(const AttnP& p, cudaStream_t st) {
  const dim3 grid((p.L + kWarps - 1) / kWarps, p.H, p.B);
  const size_t smem = sizeof(float) * kWarps * (p.d1 + p.d2);
  const int nj = (p.dv + 31) / 32;
  if (nj <= 2) split_key_attention_kernel<T, 2><<<grid, kWarps * 32, smem, st>>>(p);
  else if (nj <= 4) split_key_attention_kernel<T, 4><<<grid, kWarps * 32, smem, st>>>(p);
  else if (nj <= 8) split_key_attention_kernel<T, 8><<<grid, kWarps * 32, smem, st>>>(p);
  else if (nj <= 16) split_key_attention_kernel<T, 16><<<grid, kWarps * 32, smem, st>>>(p);
  else split_key_attention_kernel<T, 32><<<grid, kWarps * 32, smem, st>>>(p);
  return (int)cudaGetLastError();
}

}  // namespace

int launch_latent_prepare(const void* z, const void* norm_w, void* cache, void* q, const float* cosv, const float* sinv,
                          int table_len, int B, int L, int H, int r, int rd, int d, int max_len, int64_t zb, int64_t zl,
                          int64_t cb, int64_t cl, int64_t qb, int64_t ql, const int32_t* offsets, int offset, float eps,
                          int io_dtype, cudaStream_t stream) {
  if (B > 65535) return BASED_ERR_TOO_LARGE;
  const PrepP p{z, norm_w, cache, q, cosv, sinv, offsets, offset, B, L, H, r, rd, d, max_len, table_len,
                zb, zl, cb, cl, qb, ql, eps};
  const dim3 grid(L, B);
  if (io_dtype == BASED_BF16) latent_prepare_kernel<__nv_bfloat16><<<grid, kPrepThreads, 0, stream>>>(p);
  else latent_prepare_kernel<float><<<grid, kPrepThreads, 0, stream>>>(p);
  return (int)cudaGetLastError();
}

int launch_split_key_attention(const void* q1, const void* q2, const void* k1, const void* k2, const void* v,
                               const void* gate, void* out, int B, int L, int H, int d1, int d2, int dv, Strides3 sq1,
                               Strides3 sq2, Strides3 sk1, Strides3 sk2, Strides3 sv, Strides3 so, int64_t gb, int64_t gl,
                               const int32_t* offsets, int offset, float scale, AttentionOptions x, int io_dtype,
                               cudaStream_t stream) {
  if (B > 65535 || H > 65535) return BASED_ERR_TOO_LARGE;
  if (dv > 1024 || d1 + d2 > 2560) return BASED_ERR_SHAPE;
  const AttnP p{q1, q2, k1, k2, v, gate, out, offsets, offset, B, L, H, d1, d2, dv, sq1, sq2, sk1, sk2, sv, so, gb, gl, scale, x};
  return io_dtype == BASED_BF16 ? launch_attn_t<__nv_bfloat16>(p, stream) : launch_attn_t<float>(p, stream);
}

}  // namespace based
