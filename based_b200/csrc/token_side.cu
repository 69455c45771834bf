// A layer's own input per token, for the few rows of a decode step, in one launch (bf16):
//   g = gelu_tanh(W_gate x) * table[token, column ..];  y = W_proj g;  stream <- stream + y / rms(y) * norm
// and the new stream in bf16, plain or with a norm of its own.  The two products depend on one another through every
// element, so a cluster of eight CTAs owns 16 rows: each takes an eighth of the gate's outputs, hands them to the others
// through distributed shared memory, takes an eighth of the projection's outputs, and the sums of squares go the same way.
// Everything that comes from memory is asked for at the start (what registers cannot hold, into L2), so that one memory
// latency is paid.
// mma.sync m16n8k16 with a common permutation of K in both operands: a thread loads 16 bytes of a row at a time.
#include <cooperative_groups.h>

#include <utility>

#include "seq_common.cuh"
#include "tcgen05.cuh"

namespace based {
namespace {

namespace cg = cooperative_groups;
using bf16 = __nv_bfloat16;

constexpr int kCluster = 8, kWarps = 8, kThreads = kWarps * 32, kRows = 16, kMaxGateTiles = 4;   // gate tiles per CTA

struct P {
  const bf16 *x, *wg, *wp, *table, *norm, *out_norm;   // x [M, W] rows sx apart; wg [n, W], wp [W, n] contiguous
  const int64_t* tokens;
  float* residual;                                     // [M, W]
  bf16* out;                                           // [M, W]
  int64_t V, st, column, sx;
  int M, W, n;
  float eps;
};

__device__ __forceinline__ void mma16816(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
// 32 values of K: lo / hi are 8 consecutive ones of rows g and g + 8, b of a column
__device__ __forceinline__ void mma32(float (&c)[4], const uint4& lo, const uint4& hi, const uint4& b) {
  mma16816(c, lo.x, hi.x, lo.y, hi.y, b.x, b.y);
  mma16816(c, lo.z, hi.z, lo.w, hi.w, b.z, b.w);
}
__device__ __forceinline__ uint4 load16(const bf16* p, bool ok) { return ok ? __ldg(reinterpret_cast<const uint4*>(p)) : make_uint4(0, 0, 0, 0); }

// NT: projection tiles of 8 columns per warp
template <int NT>
__global__ void __cluster_dims__(kCluster, 1, 1) __launch_bounds__(kThreads) token_side_kernel(const P p) {
  extern __shared__ __align__(16) uint8_t smem[];
  cg::cluster_group cluster = cg::this_cluster();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
  const int rank = (int)cluster.block_rank(), row0 = (blockIdx.x / kCluster) * kRows;
  const int ldg = p.n + 8;                                                    // rows of G: an odd number of 16-byte units
  bf16* G = reinterpret_cast<bf16*>(smem);                                    // [16][ldg]
  float* part = reinterpret_cast<float*>(smem + kRows * ldg * 2);             // [warps][16][kMaxGateTiles * 8]
  float* ss = part + kWarps * kRows * kMaxGateTiles * 8;                      // [2][cluster][16]
  float* red = ss + 2 * kCluster * kRows;                                     // [warps][16]
  const int gt = p.n / 8, pt = p.W / 8;                                       // tiles of 8 outputs
  const int tile0 = (rank * kWarps + warp) * NT;                              // this warp's projection tiles

  auto started = cluster.barrier_arrive();   // the others' shared memory is written below
  // weights of the projection into L2
  for (int i = lane; i < NT * 8 * ((p.n + 63) / 64); i += 32) {
    const int r = i % (NT * 8), c = i / (NT * 8), row = tile0 * 8 + r;
    if (row < p.W) asm volatile("prefetch.global.L2 [%0];" ::"l"(p.wp + (int64_t)row * p.n + c * 64));
  }
  // the token vectors' values this thread will multiply by
  constexpr int ldp = kMaxGateTiles * 8, kMine = kRows * ldp / kThreads;
  float ev[kMine];
#pragma unroll
  for (int i = 0; i < kMine; ++i) {
    const int e = tid + i * kThreads, r = e / ldp, j = e - r * ldp, t = rank + (j >> 3) * kCluster;
    ev[i] = 0.f;
    if (t < gt && row0 + r < p.M) {
      const int64_t tok = p.tokens[row0 + r];
      if (tok >= 0 && tok < p.V) ev[i] = __bfloat162float(p.table[tok * p.st + p.column + t * 8 + (j & 7)]);
    }
  }
  // the projection's first 64 of K, and the stream (small tiles only)
  constexpr bool kEarly = NT <= 4;
  constexpr int kAhead = kEarly ? 2 : 0;
  uint4 wa[kAhead > 0 ? kAhead : 1][NT];
  float2 rs[kEarly ? NT : 1][2];
  if (kEarly) {
#pragma unroll
    for (int b = 0; b < kAhead; ++b)
#pragma unroll
      for (int i = 0; i < NT; ++i) wa[b][i] = load16(p.wp + (int64_t)((tile0 + i) * 8 + g) * p.n + b * 32 + t4 * 8, b * 32 + t4 * 8 < p.n && tile0 + i < pt);
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int row = row0 + g + 8 * half;
        rs[i][half] = row < p.M && tile0 + i < pt ? *reinterpret_cast<const float2*>(p.residual + (int64_t)row * p.W + (tile0 + i) * 8 + 2 * t4)
                                                  : make_float2(0.f, 0.f);
      }
  }
  // gate: this CTA's tiles rank, rank + 8, ..; the warps share K in blocks of 32
  float acc[kMaxGateTiles][4] = {};
  const bf16 *xa = p.x + (int64_t)min(row0 + g, p.M - 1) * p.sx, *xb = p.x + (int64_t)min(row0 + g + 8, p.M - 1) * p.sx;
#pragma unroll 4
  for (int k0 = warp * 32; k0 < p.W; k0 += kWarps * 32) {
    const int k = k0 + t4 * 8;
    const bool ok = k < p.W;
    const uint4 lo = load16(xa + k, ok), hi = load16(xb + k, ok);
    uint4 w[kMaxGateTiles];
#pragma unroll
    for (int i = 0; i < kMaxGateTiles; ++i) {
      const int t = rank + i * kCluster;
      w[i] = load16(p.wg + (int64_t)(t * 8 + g) * p.W + k, ok && t < gt);
    }
#pragma unroll
    for (int i = 0; i < kMaxGateTiles; ++i)
      if (rank + i * kCluster < gt) mma32(acc[i], lo, hi, w[i]);
  }
#pragma unroll
  for (int i = 0; i < kMaxGateTiles; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) part[(warp * kRows + g + 8 * (e >> 1)) * ldp + 8 * i + 2 * t4 + (e & 1)] = acc[i][e];
  __syncthreads();
  cluster.barrier_wait(std::move(started));
#pragma unroll
  for (int i = 0; i < kMine; ++i) {
    const int e = tid + i * kThreads, r = e / ldp, j = e - r * ldp, t = rank + (j >> 3) * kCluster, c = t * 8 + (j & 7);
    if (t >= gt) continue;
    float z = 0.f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) z += part[(w * kRows + r) * ldp + j];
    const bf16 v = __float2bfloat16_rn(seq::gelu_tanh_t<bf16>(z) * ev[i]);
#pragma unroll
    for (int q = 0; q < kCluster; ++q) cluster.map_shared_rank(G, q)[r * ldg + c] = v;
  }
  cluster.sync();
  // projection: NT tiles of 8 outputs per warp
  float y[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) y[i][e] = 0.f;
  auto product = [&](int k0, const uint4 (&w)[NT]) {
    const int k = k0 + t4 * 8;
    uint4 lo = make_uint4(0, 0, 0, 0), hi = lo;
    if (k < p.n) {
      lo = *reinterpret_cast<const uint4*>(G + g * ldg + k);
      hi = *reinterpret_cast<const uint4*>(G + (g + 8) * ldg + k);
    }
#pragma unroll
    for (int i = 0; i < NT; ++i) mma32(y[i], lo, hi, w[i]);
  };
#pragma unroll
  for (int b = 0; b < kAhead; ++b)
    if (b * 32 < p.n) product(b * 32, wa[b]);
#pragma unroll 2
  for (int k0 = kAhead * 32; k0 < p.n; k0 += 32) {
    uint4 w[NT];
#pragma unroll
    for (int i = 0; i < NT; ++i) w[i] = load16(p.wp + (int64_t)((tile0 + i) * 8 + g) * p.n + k0 + t4 * 8, k0 + t4 * 8 < p.n && tile0 + i < pt);
    product(k0, w);
  }
  // rows g and g + 8: sums over this CTA's columns, then over the cluster
  auto row_sums = [&](float a, float b, float* dst, float& ta, float& tb) {
    a += __shfl_xor_sync(0xffffffffu, a, 1);
    a += __shfl_xor_sync(0xffffffffu, a, 2);
    b += __shfl_xor_sync(0xffffffffu, b, 1);
    b += __shfl_xor_sync(0xffffffffu, b, 2);
    if (t4 == 0) { red[warp * kRows + g] = a; red[warp * kRows + g + 8] = b; }
    __syncthreads();
    if (tid < kRows) {
      float s = 0.f;
#pragma unroll
      for (int w = 0; w < kWarps; ++w) s += red[w * kRows + tid];
#pragma unroll
      for (int q = 0; q < kCluster; ++q) cluster.map_shared_rank(dst, q)[rank * kRows + tid] = s;
    }
    cluster.sync();
    ta = tb = 0.f;
#pragma unroll
    for (int q = 0; q < kCluster; ++q) { ta += dst[q * kRows + g]; tb += dst[q * kRows + g + 8]; }
  };
  float sa = 0.f, sb = 0.f, ta, tb;
#pragma unroll
  for (int i = 0; i < NT; ++i) {
    sa = fmaf(y[i][0], y[i][0], fmaf(y[i][1], y[i][1], sa));
    sb = fmaf(y[i][2], y[i][2], fmaf(y[i][3], y[i][3], sb));
  }
  row_sums(sa, sb, ss, ta, tb);
  const float ra = rsqrtf(ta / (float)p.W + p.eps), rb = rsqrtf(tb / (float)p.W + p.eps);
  sa = sb = 0.f;
#pragma unroll
  for (int i = 0; i < NT; ++i) {
    const int c = (tile0 + i) * 8 + 2 * t4;
    if (tile0 + i >= pt) continue;
    const float w0 = __bfloat162float(p.norm[c]), w1 = __bfloat162float(p.norm[c + 1]);
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int row = row0 + g + 8 * half;
      if (row >= p.M) continue;
      float2* dst = reinterpret_cast<float2*>(p.residual + (int64_t)row * p.W + c);
      float2 v = kEarly ? rs[kEarly ? i : 0][half] : *dst;
      const float f = half ? rb : ra;
      v.x = fmaf(y[i][2 * half] * f, w0, v.x);
      v.y = fmaf(y[i][2 * half + 1] * f, w1, v.y);
      *dst = v;
      y[i][2 * half] = v.x;
      y[i][2 * half + 1] = v.y;
      if (half) sb = fmaf(v.x, v.x, fmaf(v.y, v.y, sb));
      else sa = fmaf(v.x, v.x, fmaf(v.y, v.y, sa));
    }
  }
  float fa = 1.f, fb = 1.f;
  if (p.out_norm) {
    row_sums(sa, sb, ss + kCluster * kRows, ta, tb);
    fa = rsqrtf(ta / (float)p.W + p.eps);
    fb = rsqrtf(tb / (float)p.W + p.eps);
  }
#pragma unroll
  for (int i = 0; i < NT; ++i) {
    const int c = (tile0 + i) * 8 + 2 * t4;
    if (tile0 + i >= pt) continue;
    float w0 = 1.f, w1 = 1.f;
    if (p.out_norm) { w0 = __bfloat162float(p.out_norm[c]); w1 = __bfloat162float(p.out_norm[c + 1]); }
    if (row0 + g < p.M) *reinterpret_cast<uint32_t*>(p.out + (int64_t)(row0 + g) * p.W + c) = seq::bf16x2_bits(y[i][0] * fa * w0, y[i][1] * fa * w1);
    if (row0 + g + 8 < p.M) *reinterpret_cast<uint32_t*>(p.out + (int64_t)(row0 + g + 8) * p.W + c) = seq::bf16x2_bits(y[i][2] * fb * w0, y[i][3] * fb * w1);
  }
}

template <int NT>
int launch_nt(const P& p, cudaStream_t st) {
  const size_t smem = (size_t)kRows * (p.n + 8) * 2 + sizeof(float) * (kWarps * kRows * kMaxGateTiles * 8 + 2 * kCluster * kRows + kWarps * kRows);
  token_side_kernel<NT><<<(p.M + kRows - 1) / kRows * kCluster, kThreads, smem, st>>>(p);
  return (int)cudaGetLastError();
}

}  // namespace

// BASED_ERR_IMPL: sizes or alignment this kernel does not take.
int launch_token_side(const void* x, int64_t sx, const int64_t* tokens, const void* wg, const void* wp, const void* table, int64_t V,
                      int64_t st, int64_t column, const void* norm, float* residual, const void* out_norm, void* out, int M, int W,
                      int n, float eps, cudaStream_t stream) {
  constexpr int kColumns = kCluster * kWarps * 8;   // of one tile per warp
  if (W % 8 || n % 8 || n > 8 * kCluster * kMaxGateTiles || W > 16 * kColumns || sx % 8) return BASED_ERR_IMPL;
  if (!aligned16(x) || !aligned16(wg) || !aligned16(wp) || !aligned16(residual) || !aligned16(out)) return BASED_ERR_IMPL;
  const P p{static_cast<const bf16*>(x), static_cast<const bf16*>(wg), static_cast<const bf16*>(wp), static_cast<const bf16*>(table),
            static_cast<const bf16*>(norm), static_cast<const bf16*>(out_norm), tokens, residual, static_cast<bf16*>(out), V, st, column,
            sx, M, W, n, eps};
  const int nt = (W + kColumns - 1) / kColumns;
  if (nt <= 1) return launch_nt<1>(p, stream);
  if (nt <= 2) return launch_nt<2>(p, stream);
  if (nt <= 4) return launch_nt<4>(p, stream);
  if (nt <= 8) return launch_nt<8>(p, stream);
  return launch_nt<16>(p, stream);
}

}  // namespace based
