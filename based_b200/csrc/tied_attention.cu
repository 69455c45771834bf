// Between the projections and the attention of a layer whose values are its keys as projected, before their norm
// (grouped query heads, unit-RMS queries and keys with weights, a query temperature that grows with the position).
//
// The cache holds the projected keys alone: a normed key is k * rstd(k) * w_k, so rstd(k) is kept as one fp32 factor per
// key (it multiplies the key's scores) and w_k goes into the query together with w_q and the temperature:
//   q <- q rstd(q) w_q w_k (1 + coef ln(floor((p + 1) / every) + 1))      in place
//   cache row of the token's position <- k;   factor[b, g, position] <- rstd(k)
// One read of the cache then serves scores and values.  A group of 16 lanes owns one head of one token.
#include "seq_common.cuh"

namespace based {
namespace {

using namespace seq;

constexpr int kLanes = 16, kThreads = 256;

struct PrepP {
  void* q;                       // [B, L, H * d], rewritten
  const void *k, *wq, *wk;       // [B, L, G * d], [d], [d]
  void* cache;                   // [B, max_len, G * d]
  float* factor;                 // [B, G, max_len]
  const int32_t* offsets;
  int64_t tasks, qb, ql, kb, kl, cb, cl, fb, fh;
  int offset, L, H, G, d, max_len;
  float eps, coef, every;
};

template <typename T, int N, int VPT>
__global__ void __launch_bounds__(kThreads) tied_prepare_kernel(const PrepP p) {
  const int64_t task = (int64_t)blockIdx.x * (kThreads / kLanes) + threadIdx.x / kLanes;
  const int lane = threadIdx.x % kLanes, heads = p.H + p.G;
  const bool live = task < p.tasks;     // every lane stays for the reductions
  const int64_t token = live ? task / heads : 0;
  const int head = live ? (int)(task - token * heads) : 0;
  const int b = (int)(token / p.L), l = (int)(token - (int64_t)b * p.L);
  const bool key = head >= p.H;
  T* src = key ? const_cast<T*>(static_cast<const T*>(p.k)) + b * p.kb + l * p.kl + (int64_t)(head - p.H) * p.d
               : static_cast<T*>(p.q) + b * p.qb + l * p.ql + (int64_t)head * p.d;
  const int packs = p.d / N;
  float z[VPT][N], ss = 0.f;
#pragma unroll
  for (int v = 0; v < VPT; ++v) {
    const int c = lane + v * kLanes;
    if (c < packs) {
      Pack<T, N>::load(src + c * N, z[v]);
#pragma unroll
      for (int i = 0; i < N; ++i) ss = fmaf(z[v][i], z[v][i], ss);
    }
  }
#pragma unroll
  for (int o = kLanes / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if (!live) return;
  const float rstd = rsqrtf(ss / (float)p.d + p.eps);
  const int pos = position0(p.offsets, p.offset, b) + l;
  if (key) {
    if (pos < 0 || pos >= p.max_len) return;
    T* row = static_cast<T*>(p.cache) + b * p.cb + (int64_t)pos * p.cl + (int64_t)(head - p.H) * p.d;
#pragma unroll
    for (int v = 0; v < VPT; ++v) {
      const int c = lane + v * kLanes;
      if (c < packs) Pack<T, N>::store(row + c * N, z[v]);
    }
    if (lane == 0) p.factor[b * p.fb + (head - p.H) * p.fh + pos] = rstd;
    return;
  }
  const float f = p.coef == 0.f ? rstd : rstd * fmaf(p.coef, logf(floorf(__fdiv_rn((float)(pos + 1), p.every)) + 1.0f), 1.0f);
#pragma unroll
  for (int v = 0; v < VPT; ++v) {
    const int c = lane + v * kLanes;
    if (c < packs) {
      float a[N], w[N];
      Pack<T, N>::load(static_cast<const T*>(p.wq) + c * N, a);
      Pack<T, N>::load(static_cast<const T*>(p.wk) + c * N, w);
#pragma unroll
      for (int i = 0; i < N; ++i) z[v][i] *= f * (a[i] * w[i]);
      Pack<T, N>::store(src + c * N, z[v]);
    }
  }
}

template <typename T>
int launch_t(const PrepP& p, cudaStream_t st) {
  const int64_t blocks = (p.tasks + kThreads / kLanes - 1) / (kThreads / kLanes);
  if (blocks > 2147483647LL) return BASED_ERR_TOO_LARGE;
  const unsigned grid = (unsigned)blocks;
  const bool vec = p.d % 8 == 0 && aligned16(p.q) && aligned16(p.k) && aligned16(p.wq) && aligned16(p.wk) && aligned16(p.cache) &&
                   p.qb % 8 == 0 && p.ql % 8 == 0 && p.kb % 8 == 0 && p.kl % 8 == 0 && p.cb % 8 == 0 && p.cl % 8 == 0;
  if (vec && p.d <= 128) tied_prepare_kernel<T, 8, 1><<<grid, kThreads, 0, st>>>(p);
  else if (vec && p.d <= 256) tied_prepare_kernel<T, 8, 2><<<grid, kThreads, 0, st>>>(p);
  else if (vec && p.d <= 512) tied_prepare_kernel<T, 8, 4><<<grid, kThreads, 0, st>>>(p);
  else if (p.d <= 128) tied_prepare_kernel<T, 1, 8><<<grid, kThreads, 0, st>>>(p);
  else if (p.d <= 512) tied_prepare_kernel<T, 1, 32><<<grid, kThreads, 0, st>>>(p);
  else return BASED_ERR_SHAPE;
  return (int)cudaGetLastError();
}

}  // namespace

int launch_tied_prepare(void* q, const void* k, const void* wq, const void* wk, void* cache, float* factor, int B, int L, int H,
                        int G, int d, int max_len, int64_t qb, int64_t ql, int64_t kb, int64_t kl, int64_t cb, int64_t cl,
                        int64_t fb, int64_t fh, const int32_t* offsets, int offset, float eps, float coef, float every,
                        int io_dtype, cudaStream_t stream) {
  const PrepP p{q, k, wq, wk, cache, factor, offsets, (int64_t)B * L * (H + G), qb, ql, kb, kl, cb, cl, fb, fh,
                offset, L, H, G, d, max_len, eps, coef, every};
  return io_dtype == BASED_BF16 ? launch_t<__nv_bfloat16>(p, stream) : launch_t<float>(p, stream);
}

}  // namespace based
