// Attention of a few query rows over a cache whose rows are keys and values at once (a decode step, or a short portion of a
// prompt), bf16, HBM-bound on the cache.
//   s[t, r] = (k_t . q_r) factor_t scale;   out_r = sum_t exp(s[t, r]) k_t / (sink + sum_t exp(s[t, r])) * sigmoid(gate_r)
// The query heads of a group (times the call's tokens) are the rows; 8 or 16 of them share a read of the keys.  Both products
// are taken transposed (mma.sync m16n8k16: keys by rows, then dimensions by rows), so that a step with up to 8 rows wastes
// nothing on a 16-row tile.  A warp walks tiles of 32 keys of its own through its own ring of TMA copies (64-column atoms,
// 128-byte swizzle), with its own running maximum and sum, so a CTA meets only at the end; a tile in shared memory is the
// left operand of both products.  Several CTAs split the keys of a sequence; the one that finishes last adds the parts up
// (nobody waits).  The split follows the sequence's current length, read on the device.
#include <initializer_list>
#include <mutex>

#include "seq_common.cuh"
#include "tcgen05.cuh"
#include "tma.cuh"

namespace based {

__device__ unsigned int g_tc_status_tied_decode = 0;

namespace {

using namespace tc;

constexpr int kWarps = 4, kThreads = kWarps * 32, kTile = 32, kStages = 3, kMaxSplits = 592;
constexpr uint32_t kAtom = kTile * 128;   // bytes of 32 keys x 64 columns

struct P {
  CUtensorMap mk;              // cache [B][G][max_len][d]
  const __nv_bfloat16 *q, *gate;
  const float* factor;
  __nv_bfloat16* out;
  float *part, *ms;            // [splits][B * G][padded rows][d] and [..][2]: weighted sums, maximum and sum
  int* count;                  // [B * G * row tiles], zero between launches
  const int32_t* offsets;
  int offset, B, L, G, group, d, splits, max_len;
  int64_t qb, ql, fb, fh, gb, gl, ob, ol;
  float scale_log2e, sink;
  unsigned int* status;
};

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ uint32_t transpose8(uint32_t x) {
  asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %0;\n" : "+r"(x));
  return x;
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void bulk_load(uint32_t dst, const void* src, uint32_t bytes, uint32_t mbar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];\n" ::"r"(dst), "l"(src),
               "r"(bytes), "r"(mbar)
               : "memory");
}
__device__ __forceinline__ float ex2(float x) { float r; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x)); return r; }
__device__ __forceinline__ float weight(float m, float base) { return m == -INFINITY ? 0.f : exp2f(m - base); }

// d <= 16 * NK, a multiple of 16; 8 * NR rows per CTA
template <int NK, int NR>
__global__ void __launch_bounds__(kThreads, NK <= 4 ? 4 : (NK <= 8 ? 2 : 1)) tied_decode_kernel(const __grid_constant__ P p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
  constexpr int kRows = 8 * NR;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
  const int split = blockIdx.x, rt = blockIdx.y, row0 = rt * kRows, bg = blockIdx.z, b = bg / p.G, kh = bg - b * p.G;
  const int d = p.d, nk = d / 16, na = (d + 63) / 64, R = p.L * p.group;
  const uint32_t stage_bytes = na * kAtom;
  const uint32_t ring = smem_u32(smem) + warp * kStages * stage_bytes;                  // this warp's
  uint8_t* tail = smem + kWarps * kStages * stage_bytes;
  float* F = reinterpret_cast<float*>(tail) + warp * kStages * kTile;
  const uint32_t bar = smem_u32(tail + kWarps * kStages * kTile * 4) + warp * kStages * 8;
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tail + kWarps * kStages * (kTile * 4 + 8));
  const int pos0 = seq::position0(p.offsets, p.offset, b);
  const int len = min(pos0 + p.L, p.max_len);
  const int tiles = (len + kTile - 1) / kTile, per = (tiles + p.splits - 1) / p.splits;
  const int t0 = min(split * per, tiles), t1 = min(t0 + per, tiles);

  if (lane == 0) {
#pragma unroll
    for (int s = 0; s < kStages; ++s) mbar_init(bar + 8 * s, 1);
    if (warp == 0) *abort_flag = 0;
    fence_mbar_init();
    fence_proxy_async();
  }
  __syncthreads();
  const float* factor = p.factor + b * p.fb + kh * p.fh;
  auto fetch = [&](int t, int s) {   // one lane
    tma::mbar_expect_tx(bar + 8 * s, stage_bytes + kTile * 4);
    for (int a = 0; a < na; ++a) tma::load_4d(ring + s * stage_bytes + a * kAtom, &p.mk, bar + 8 * s, 64 * a, t * kTile, kh, b);
    bulk_load(smem_u32(F + s * kTile), factor + t * kTile, kTile * 4, bar + 8 * s);
  };
  if (lane == 0) {
#pragma unroll
    for (int s = 0; s < kStages; ++s)
      if (t0 + warp + s * kWarps < t1) fetch(t0 + warp + s * kWarps, s);
  }
  // queries as the right operand: registers of row 8 n + g, dimensions 16 k + 2 t4 .. and 16 k + 8 + 2 t4 ..
  uint32_t qb[NK][NR][2];
#pragma unroll
  for (int n = 0; n < NR; ++n) {
    const int row = row0 + 8 * n + g, l = row / p.group, h = kh * p.group + row - l * p.group;
    const uint32_t* src = reinterpret_cast<const uint32_t*>(p.q + b * p.qb + l * p.ql + (int64_t)h * d);
#pragma unroll
    for (int k = 0; k < NK; ++k) {
      const bool ok = k < nk && row < R;
      qb[k][n][0] = ok ? src[8 * k + t4] : 0u;
      qb[k][n][1] = ok ? src[8 * k + 4 + t4] : 0u;
    }
  }
  float acc[NK][NR][4];        // dimensions 16 k + g (+ 8), rows 8 n + 2 t4 (+ 1)
#pragma unroll
  for (int k = 0; k < NK; ++k)
#pragma unroll
    for (int n = 0; n < NR; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[k][n][e] = 0.f;
  float m[NR][2], sum[NR][2];
  int last[NR][2];             // last key rows 8 n + 2 t4 (+ 1) see
#pragma unroll
  for (int n = 0; n < NR; ++n)
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int row = row0 + 8 * n + 2 * t4 + i;
      m[n][i] = -INFINITY;
      sum[n][i] = 0.f;
      last[n][i] = row < R ? pos0 + row / p.group : -1;
    }
  // ldmatrix addresses: rows of a tile are 128 bytes, the 16-byte piece c of row r is at c ^ (r & 7)
  const int kr = (lane & 7) + ((lane >> 3) & 1) * 8, kc = lane >> 4;     // scores: keys 0-15, dimensions low / high
  const int vr = (lane & 7) + (lane >> 4) * 8, vc = (lane >> 3) & 1;     // sums: dimensions low / high, keys 0-7 / 8-15
  int stage = 0, phase = 0;
  for (int t = t0 + warp; t < t1; t += kWarps) {
    mbar_wait_bounded(bar + 8 * stage, phase, abort_flag, p.status, 1u << 20);
    const uint32_t K = ring + stage * stage_bytes;
    const bool whole = t * kTile + kTile - 1 <= pos0;      // every row sees every key
    if (t * kTile + kTile > len) {                         // rows past the sequence may hold anything
      const int first = len - t * kTile;
      for (int e = lane; e < na * (kTile - first) * 8; e += 32) {
        const int a = e / ((kTile - first) * 8), r = e - a * (kTile - first) * 8;
        *reinterpret_cast<uint4*>(smem + (K - smem_u32(smem)) + a * kAtom + (first + (r >> 3)) * 128 + (r & 7) * 16) = make_uint4(0, 0, 0, 0);
      }
      __syncwarp();
    }
    float s[2][NR][4];
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int n = 0; n < NR; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[x][n][e] = 0.f;
#pragma unroll
    for (int k = 0; k < NK; ++k) {
      if (k < nk) {
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          uint32_t a[4];
          ldsm4(a, K + (k >> 2) * kAtom + (16 * x + kr) * 128 + (((2 * (k & 3) + kc) ^ (kr & 7)) << 4));
#pragma unroll
          for (int n = 0; n < NR; ++n) mma16816(s[x][n], a, qb[k][n][0], qb[k][n][1]);
        }
      }
    }
    // s[x][n]: keys 16 x + g (+ 8 for elements 2, 3), rows 8 n + 2 t4 (+ 1 for elements 1, 3)
    const float* Ft = F + stage * kTile;
    float fk[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) fk[i] = Ft[8 * i + g] * p.scale_log2e;
    uint32_t pb[2][NR][2];
    float f[NR][2];
    bool moved = false;
#pragma unroll
    for (int n = 0; n < NR; ++n) {
      float mt[2] = {-INFINITY, -INFINITY};
#pragma unroll
      for (int x = 0; x < 2; ++x)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          s[x][n][e] *= fk[2 * x + (e >> 1)];
          if (!whole && t * kTile + 16 * x + 8 * (e >> 1) + g > last[n][e & 1]) s[x][n][e] = -INFINITY;
          mt[e & 1] = fmaxf(mt[e & 1], s[x][n][e]);
        }
#pragma unroll
      for (int i = 0; i < 2; ++i) {
#pragma unroll
        for (int o = 4; o < 32; o <<= 1) mt[i] = fmaxf(mt[i], __shfl_xor_sync(0xffffffffu, mt[i], o));
        const float mn = fmaxf(m[n][i], mt[i]), base = mn == -INFINITY ? 0.f : mn;
        f[n][i] = ex2(m[n][i] - base);
        moved |= mn != m[n][i];
        m[n][i] = mn;
        float add = 0.f;
#pragma unroll
        for (int x = 0; x < 2; ++x)
#pragma unroll
          for (int e = i; e < 4; e += 2) {
            s[x][n][e] = ex2(s[x][n][e] - base);
            add += s[x][n][e];
          }
        sum[n][i] = fmaf(sum[n][i], f[n][i], add);   // this lane's share
      }
#pragma unroll
      for (int x = 0; x < 2; ++x) {                  // to the right operand's layout: keys along the registers
        pb[x][n][0] = transpose8(seq::bf16x2_bits(s[x][n][0], s[x][n][1]));
        pb[x][n][1] = transpose8(seq::bf16x2_bits(s[x][n][2], s[x][n][3]));
      }
    }
    if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
      for (int k = 0; k < NK; ++k)
#pragma unroll
        for (int n = 0; n < NR; ++n) { acc[k][n][0] *= f[n][0]; acc[k][n][1] *= f[n][1]; acc[k][n][2] *= f[n][0]; acc[k][n][3] *= f[n][1]; }
    }
#pragma unroll
    for (int k = 0; k < NK; ++k) {
      if (k < nk) {
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          uint32_t a[4];
          ldsm4t(a, K + (k >> 2) * kAtom + (16 * x + vr) * 128 + (((2 * (k & 3) + vc) ^ (vr & 7)) << 4));
#pragma unroll
          for (int n = 0; n < NR; ++n) mma16816(acc[k][n], a, pb[x][n][0], pb[x][n][1]);
        }
      }
    }
    __syncwarp();   // every lane has read this stage
    if (lane == 0 && t + kStages * kWarps < t1) fetch(t + kStages * kWarps, stage);
    if (++stage == kStages) { stage = 0; phase ^= 1; }
  }
  __syncthreads();   // the rings are free: they take the warps' results
  float* O = reinterpret_cast<float*>(smem);                   // [warps][rows][d + 4]
  const int lo = d + 4;
  float* MS = O + kWarps * kRows * lo;                         // [warps][rows][2]
#pragma unroll
  for (int n = 0; n < NR; ++n)
#pragma unroll
    for (int i = 0; i < 2; ++i) {
#pragma unroll
      for (int o = 4; o < 32; o <<= 1) sum[n][i] += __shfl_xor_sync(0xffffffffu, sum[n][i], o);
      const int rr = warp * kRows + 8 * n + 2 * t4 + i;
      if (g == 0) { MS[2 * rr] = m[n][i]; MS[2 * rr + 1] = sum[n][i]; }
#pragma unroll
      for (int k = 0; k < NK; ++k)
        if (k < nk) { O[rr * lo + 16 * k + g] = acc[k][n][i]; O[rr * lo + 16 * k + 8 + g] = acc[k][n][2 + i]; }
    }
  __syncthreads();
  const int rows = min(kRows, R - row0), quads = d / 4;
  const int64_t prow = (int64_t)p.G * p.B * gridDim.y * kRows;                 // rows of one split's part
  const int64_t at = ((int64_t)bg * gridDim.y + rt) * kRows;
  auto finish = [&](int row, int c, float4 x, float mt, float total) {
    const int l = row / p.group, h = kh * p.group + row - l * p.group;
    const float f = 1.0f / (p.sink > 0.f ? fmaf(p.sink, exp2f(-mt), total) : total);
    const int64_t e = (int64_t)h * d + c;
    float y[4] = {x.x * f, x.y * f, x.z * f, x.w * f};
    if (p.gate) {
      float z[4];
      seq::Pack<__nv_bfloat16, 4>::load(p.gate + b * p.gb + l * p.gl + e, z);
#pragma unroll
      for (int i = 0; i < 4; ++i) y[i] *= seq::sigmoid_t<__nv_bfloat16>(z[i]);
    }
    seq::Pack<__nv_bfloat16, 4>::store(p.out + b * p.ob + l * p.ol + e, y);
  };
  for (int e = tid; e < rows * quads; e += kThreads) {
    const int rr = e / quads, c = (e - rr * quads) * 4;
    float mw[kWarps], mt = p.splits == 1 && p.sink > 0.f ? 0.f : -INFINITY;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) { mw[w] = MS[(w * kRows + rr) * 2]; mt = fmaxf(mt, mw[w]); }
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
    float y = 0.f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
      const float f = weight(mw[w], mt);
      const float4 v = *reinterpret_cast<const float4*>(O + (w * kRows + rr) * lo + c);
      x.x = fmaf(f, v.x, x.x); x.y = fmaf(f, v.y, x.y); x.z = fmaf(f, v.z, x.z); x.w = fmaf(f, v.w, x.w);
      y = fmaf(f, MS[(w * kRows + rr) * 2 + 1], y);
    }
    if (p.splits == 1) {
      finish(row0 + rr, c, x, mt, y);
    } else {
      const int64_t r = (int64_t)split * prow + at + rr;
      *reinterpret_cast<float4*>(p.part + r * d + c) = x;
      if (c == 0) *reinterpret_cast<float2*>(p.ms + 2 * r) = make_float2(mt, y);
    }
  }
  if (p.splits == 1) return;
  __shared__ int done;
  __threadfence();
  __syncthreads();
  if (tid == 0) {
    int* count = p.count + bg * gridDim.y + rt;
    done = atomicAdd(count, 1) == p.splits - 1;
    if (done) *count = 0;
  }
  __syncthreads();
  if (!done) return;
  __threadfence();
  // weights of the splits, per row, in shared memory
  float* W = reinterpret_cast<float*>(smem);                   // [rows][splits], then [rows] maxima and sums
  float* T = W + rows * p.splits;
  for (int rr = warp; rr < rows; rr += kWarps) {
    const float2* src = reinterpret_cast<const float2*>(p.ms) + at + rr;
    float mt = p.sink > 0.f ? 0.f : -INFINITY;
    for (int s = lane; s < p.splits; s += 32) mt = fmaxf(mt, __ldcg(src + s * prow).x);
    mt = warp_max(mt);
    float y = 0.f;
    for (int s = lane; s < p.splits; s += 32) {
      const float2 v = __ldcg(src + s * prow);
      const float w = weight(v.x, mt);
      W[rr * p.splits + s] = w;
      y = fmaf(w, v.y, y);
    }
    y = warp_sum(y);
    if (lane == 0) { T[2 * rr] = mt; T[2 * rr + 1] = y; }
  }
  __syncthreads();
  for (int e = tid; e < rows * quads; e += kThreads) {
    const int rr = e / quads, c = (e - rr * quads) * 4;
    const float* src = p.part + (at + rr) * d + c;
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int s = 0; s < p.splits; ++s) {
      const float w = W[rr * p.splits + s];
      const float4 v = __ldcg(reinterpret_cast<const float4*>(src + s * prow * d));
      x.x = fmaf(w, v.x, x.x); x.y = fmaf(w, v.y, x.y); x.z = fmaf(w, v.z, x.z); x.w = fmaf(w, v.w, x.w);
    }
    finish(row0 + rr, c, x, T[2 * rr], T[2 * rr + 1]);
  }
}

int rows_per_cta(int R) { return R <= 8 ? 8 : 16; }

size_t smem_bytes(int d) {
  const size_t na = (d + 63) / 64;
  const size_t ring = kWarps * kStages * (na * kAtom + kTile * 4 + 8) + 16;
  const size_t merge = (size_t)kWarps * 16 * (d + 4 + 2) * 4, parts = (size_t)16 * (kMaxSplits + 2) * 4;
  return 1024 + (ring > merge ? (ring > parts ? ring : parts) : (merge > parts ? merge : parts));
}

template <int NK, int NR>
int launch_k(const P& p, cudaStream_t st) {
  const cudaError_t e = cudaFuncSetAttribute(tied_decode_kernel<NK, NR>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_bytes(16 * NK));
  if (e != cudaSuccess) return (int)e;
  const int rows = 8 * NR;
  tied_decode_kernel<NK, NR><<<dim3(p.splits, (p.L * p.group + rows - 1) / rows, p.B * p.G), kThreads, smem_bytes(p.d), st>>>(p);
  return (int)cudaGetLastError();
}

}  // namespace

int read_tc_status_tied_decode(unsigned int* out, int reset) {
  unsigned int v = 0;
  cudaError_t e = cudaMemcpyFromSymbol(&v, g_tc_status_tied_decode, sizeof(v));
  if (e != cudaSuccess) return (int)e;
  if (out) *out = v;
  if (reset && v != 0) {
    v = 0;
    e = cudaMemcpyToSymbol(g_tc_status_tied_decode, &v, sizeof(v));
  }
  return (int)e;
}

int tied_decode_splits(int B, int R, int G, int d, int max_len) {
  const int rows = rows_per_cta(R), slots = 148 * (d <= 64 ? 4 : (d <= 128 ? 2 : 1));
  const int64_t ctas = (int64_t)B * G * ((R + rows - 1) / rows);
  int s = (int)(slots / (ctas > 0 ? ctas : 1));
  const int most = (max_len + kWarps * kTile - 1) / (kWarps * kTile);   // a tile per warp at full length
  if (s > most) s = most;
  return s < 1 ? 1 : s;
}

size_t tied_decode_scratch_bytes(int B, int R, int G, int d, int max_len) {
  const int s = tied_decode_splits(B, R, G, d, max_len), rows = rows_per_cta(R);
  return s > 1 ? (size_t)s * B * G * ((R + rows - 1) / rows * rows) * (d + 2) * sizeof(float) : 0;
}

// factor rows may be read up to the next multiple of 32 keys.  BASED_ERR_IMPL: sizes or strides this kernel does not take.
int launch_tied_decode(const void* q, const void* cache, const float* factor, const void* gate, void* out, void* scratch,
                       size_t scratch_bytes, int* count, int count_len, int B, int L, int H, int G, int d, int max_len,
                       int64_t qb, int64_t ql, int64_t cb, int64_t cl, int64_t fb, int64_t fh, int64_t gb, int64_t gl,
                       int64_t ob, int64_t ol, const int32_t* offsets, int offset, float scale, float sink,
                       cudaStream_t stream) {
  const int group = H / G, R = L * group, rows = rows_per_cta(R), tiles = (R + rows - 1) / rows;
  if (d % 16 || d > 256 || (int64_t)B * G > 65535 || tiles > 65535) return BASED_ERR_IMPL;
  if (!aligned16(q) || !aligned16(cache) || !aligned16(factor)) return BASED_ERR_IMPL;
  const uintptr_t io = reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(gate);
  auto fix = [](int64_t s, int extent) { return extent == 1 ? (int64_t)8 : s; };
  for (int64_t s : {fix(qb, B), fix(ql, L), fix(cb, B), fix(cl, max_len), fix(ob, B), fix(ol, L), gate ? fix(gb, B) : 8, gate ? fix(gl, L) : 8})
    if (s % 8 || s <= 0) return BASED_ERR_IMPL;
  if (io % 8) return BASED_ERR_IMPL;
  if ((G > 1 && fh % 4) || (B > 1 && fb % 4) || fh < (max_len + kTile - 1) / kTile * kTile) return BASED_ERR_IMPL;
  int splits = tied_decode_splits(B, R, G, d, max_len);
  if (!count || count_len < (int64_t)B * G * tiles) splits = 1;   // many rows fill the machine without a split
  if (splits > 1 && (!scratch || !aligned16(scratch) || scratch_bytes < tied_decode_scratch_bytes(B, R, G, d, max_len)))
    return BASED_ERR_SCRATCH;
  P p;
  static tma::MapCache maps;
  const tma::MapKey key = tma::make_key(cache, d, max_len, G, B, 0, fix(cl, max_len), d, fix(cb, B), 0, 64, kTile, 0, 4);
  if (!maps.find(key, &p.mk)) {
    if (tma::encode_bf16_4d_sw128(&p.mk, cache, d, max_len, G, B, fix(cl, max_len), d, fix(cb, B), 64, kTile)) return BASED_ERR_IMPL;
    maps.put(key, p.mk);
  }
  p.q = static_cast<const __nv_bfloat16*>(q);
  p.gate = static_cast<const __nv_bfloat16*>(gate);
  p.factor = factor;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.part = static_cast<float*>(scratch);
  p.ms = p.part + (size_t)splits * B * G * tiles * rows * d;
  p.count = count; p.offsets = offsets; p.offset = offset;
  p.B = B; p.L = L; p.G = G; p.group = group; p.d = d; p.splits = splits; p.max_len = max_len;
  p.qb = qb; p.ql = ql; p.fb = fb; p.fh = fh; p.gb = gb; p.gl = gl; p.ob = ob; p.ol = ol;
  p.scale_log2e = scale * 1.4426950408889634f;
  p.sink = sink;
  {
    constexpr int kMaxDevices = 64;
    static std::mutex mu;
    static unsigned int* status[kMaxDevices] = {};
    int dev = 0;
    cudaError_t e = cudaGetDevice(&dev);
    if (e != cudaSuccess) return (int)e;
    if (dev < 0 || dev >= kMaxDevices) return BASED_ERR_TOO_LARGE;
    std::lock_guard<std::mutex> lock(mu);
    if (status[dev] == nullptr) {
      unsigned int* addr = nullptr;
      e = cudaGetSymbolAddress(reinterpret_cast<void**>(&addr), g_tc_status_tied_decode);
      if (e != cudaSuccess) return (int)e;
      status[dev] = addr;
    }
    p.status = status[dev];
  }
  if (rows == 8) {
    if (d <= 64) return launch_k<4, 1>(p, stream);
    if (d <= 128) return launch_k<8, 1>(p, stream);
    return launch_k<16, 1>(p, stream);
  }
  if (d <= 64) return launch_k<4, 2>(p, stream);
  if (d <= 128) return launch_k<8, 2>(p, stream);
  return launch_k<16, 2>(p, stream);
}

}  // namespace based
