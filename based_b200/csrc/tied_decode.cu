// Attention of a few query rows over a cache whose rows are keys and values at once (a decode step, or a short portion of a
// prompt), bf16, HBM-bound on the cache.
//   s[r, t] = (q_r . k_t) factor_t scale;   out_r = sum_t exp(s[r, t]) k_t / (sink + sum_t exp(s[r, t])) * sigmoid(gate_r)
// The query heads of a group (times the call's tokens) are the rows; 16 of them, one mma.sync tile, share a read of the
// keys.  A warp walks key tiles of its own through its own cp.async ring, with its own running maximum and sum, so a CTA
// meets only at the end: a tile of keys in shared memory is the B operand of both products, and the score accumulator is
// the A operand of the second.  Several CTAs split the keys of a sequence; the one that finishes last adds the parts up
// (nobody waits).  The split follows the sequence's current length, read on the device.
#include <initializer_list>

#include "seq_common.cuh"
#include "tcgen05.cuh"

namespace based {
namespace {

constexpr int kWarps = 4, kThreads = kWarps * 32, kTile = 32, kStages = 3, kPad = 8, kRowTile = 16;

struct P {
  const __nv_bfloat16 *q, *cache, *gate;
  const float* factor;
  __nv_bfloat16* out;
  float* part;                 // [splits][B * G][rows padded to 16][d + 2]
  int* count;                  // [B * G * row tiles], zero between launches
  const int32_t* offsets;
  int offset, B, L, G, group, d, splits, max_len;
  int64_t qb, ql, cb, cl, fb, fh, gb, gl, ob, ol;
  float scale_log2e, sink;
};

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void wait_but(int) { asm volatile("cp.async.wait_group %0;\n" ::"n"(kStages - 1) : "memory"); }
__device__ __forceinline__ float weight(float m, float base) { return m == -INFINITY ? 0.f : exp2f(m - base); }

// d <= 16 * NK, a multiple of 16
template <int NK>
__global__ void __launch_bounds__(kThreads, NK <= 8 ? 2 : 1) tied_decode_kernel(const P p) {
  extern __shared__ __align__(16) uint8_t smem[];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
  const int split = blockIdx.x, rt = blockIdx.y, row0 = rt * kRowTile, bg = blockIdx.z, b = bg / p.G, kh = bg - b * p.G;
  const int d = p.d, nk = d / 16, ld = d + kPad, R = p.L * p.group;   // ld: an odd number of 16-byte units
  __nv_bfloat16* Q = reinterpret_cast<__nv_bfloat16*>(smem);                                  // [16][ld]
  __nv_bfloat16* K = Q + kRowTile * ld + warp * (kStages * kTile) * ld;                       // this warp's ring
  float* F = reinterpret_cast<float*>(Q + (kRowTile + kWarps * kStages * kTile) * ld) + warp * kStages * kTile;
  const int pos0 = seq::position0(p.offsets, p.offset, b);
  const int len = min(pos0 + p.L, p.max_len);
  const int tiles = (len + kTile - 1) / kTile, per = (tiles + p.splits - 1) / p.splits;
  const int t0 = min(split * per, tiles), t1 = min(t0 + per, tiles);
  const int chunks = d / 8;

  const __nv_bfloat16* cache = p.cache + b * p.cb + (int64_t)kh * d;
  const float* factor = p.factor + b * p.fb + kh * p.fh;
  const int i0 = lane / chunks, c0 = lane - i0 * chunks, di = 32 / chunks, dc = 32 - di * chunks;
  auto fetch = [&](int t, int s) {
    if (t < t1) {
      const uint32_t dst = tc::smem_u32(K + s * kTile * ld);
      for (int i = i0, c = c0; i < kTile;) {   // 16-byte piece c of key i, then the 32nd after it
        const int key = t * kTile + i;
        tc::cp_async16(dst + (i * ld + c * 8) * 2, cache + (int64_t)(key < len ? key : 0) * p.cl + c * 8, key < len);
        i += di;
        c += dc;
        if (c >= chunks) { c -= chunks; ++i; }
      }
      if (lane < kTile / 4) tc::cp_async16(tc::smem_u32(F + s * kTile + lane * 4), factor + t * kTile + lane * 4, true);
    }
    tc::cp_async_commit();
  };
#pragma unroll
  for (int s = 0; s < kStages - 1; ++s) fetch(t0 + warp + s * kWarps, s);

  for (int e = tid; e < kRowTile * chunks; e += kThreads) {
    const int i = e / chunks, c = (e - i * chunks) * 8, row = row0 + i;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (row < R) {
      const int l = row / p.group, h = kh * p.group + row - l * p.group;
      v = *reinterpret_cast<const uint4*>(p.q + b * p.qb + l * p.ql + (int64_t)h * d + c);
    }
    *reinterpret_cast<uint4*>(Q + i * ld + c) = v;
  }
  __syncthreads();
  constexpr bool kQRegs = NK <= 8;
  uint32_t qa[kQRegs ? NK : 1][4];
  const uint32_t qaddr = tc::smem_u32(Q + (lane & 15) * ld + (lane >> 4) * 8);
  if (kQRegs) {
#pragma unroll
    for (int k = 0; k < NK; ++k)
      if (k < nk) ldsm4(qa[k], qaddr + k * 32);
  }
  float acc[2 * NK][4];
#pragma unroll
  for (int i = 0; i < 2 * NK; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, sum[2] = {0.f, 0.f};
  int last[2];   // last key rows g and g + 8 see
#pragma unroll
  for (int i = 0; i < 2; ++i) last[i] = row0 + g + 8 * i < R ? pos0 + (row0 + g + 8 * i) / p.group : -1;

  int stage = 0;
  for (int t = t0 + warp; t < t1; t += kWarps) {
    fetch(t + (kStages - 1) * kWarps, stage == 0 ? kStages - 1 : stage - 1);
    wait_but(0);
    __syncwarp();
    const __nv_bfloat16* Kt = K + stage * kTile * ld;
    const float* Ft = F + stage * kTile;
    float s[kTile / 8][4];
#pragma unroll
    for (int n = 0; n < kTile / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[n][e] = 0.f;
    // keys 16 n2 .. + 15 in one load: matrices (keys 0-7, k low), (keys 0-7, k high), (keys 8-15, ..), ..
    const uint32_t ka = tc::smem_u32(Kt + ((lane & 7) + (lane >> 4) * 8) * ld) + ((lane >> 3) & 1) * 16;
#pragma unroll
    for (int k = 0; k < NK; ++k) {
      if (k < nk) {
        uint32_t a[4];
        if (kQRegs) {
#pragma unroll
          for (int e = 0; e < 4; ++e) a[e] = qa[kQRegs ? k : 0][e];
        } else {
          ldsm4(a, qaddr + k * 32);
        }
#pragma unroll
        for (int n2 = 0; n2 < kTile / 16; ++n2) {
          uint32_t bb[4];
          ldsm4(bb, ka + n2 * 16 * ld * 2 + k * 32);
          mma16816(s[2 * n2], a, bb[0], bb[1]);
          mma16816(s[2 * n2 + 1], a, bb[2], bb[3]);
        }
      }
    }
    float mt[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int n = 0; n < kTile / 8; ++n) {
      const float2 f = *reinterpret_cast<const float2*>(Ft + 8 * n + 2 * t4);
      const int key = t * kTile + 8 * n + 2 * t4;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float x = s[n][e] * ((e & 1) ? f.y : f.x) * p.scale_log2e;
        s[n][e] = key + (e & 1) <= last[e >> 1] ? x : -INFINITY;
        mt[e >> 1] = fmaxf(mt[e >> 1], s[n][e]);
      }
    }
    float f[2], base[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      mt[i] = fmaxf(mt[i], __shfl_xor_sync(0xffffffffu, mt[i], 1));
      mt[i] = fmaxf(mt[i], __shfl_xor_sync(0xffffffffu, mt[i], 2));
      const float mn = fmaxf(m[i], mt[i]);
      base[i] = mn == -INFINITY ? 0.f : mn;
      f[i] = exp2f(m[i] - base[i]);
      m[i] = mn;
      sum[i] *= f[i];
    }
    uint32_t pa[kTile / 16][4];
#pragma unroll
    for (int n = 0; n < kTile / 8; ++n) {
      float e0 = exp2f(s[n][0] - base[0]), e1 = exp2f(s[n][1] - base[0]), e2 = exp2f(s[n][2] - base[1]), e3 = exp2f(s[n][3] - base[1]);
      sum[0] += e0 + e1;
      sum[1] += e2 + e3;
      pa[n >> 1][(n & 1) * 2] = seq::bf16x2_bits(e0, e1);
      pa[n >> 1][(n & 1) * 2 + 1] = seq::bf16x2_bits(e2, e3);
    }
    if (__any_sync(0xffffffffu, f[0] != 1.f || f[1] != 1.f)) {
#pragma unroll
      for (int i = 0; i < 2 * NK; ++i) { acc[i][0] *= f[0]; acc[i][1] *= f[0]; acc[i][2] *= f[1]; acc[i][3] *= f[1]; }
    }
#pragma unroll
    for (int n = 0; n < 2 * NK; ++n) {
      if (n < 2 * nk) {
        uint32_t bb[4];
        ldsm4t(bb, tc::smem_u32(Kt + lane * ld + n * 8));   // keys 0-31 of 8 columns
        mma16816(acc[n], pa[0], bb[0], bb[1]);
        mma16816(acc[n], pa[1], bb[2], bb[3]);
      }
    }
    __syncwarp();   // every lane has read this stage
    stage = stage == kStages - 1 ? 0 : stage + 1;
  }
  tc::cp_async_wait_all();
  __syncthreads();   // the rings are free: they take the warps' results
  float* O = reinterpret_cast<float*>(Q + kRowTile * ld);      // [warps][16][d + 4]
  const int lo = d + 4;
  float* MS = O + kWarps * kRowTile * lo;                      // [warps][16][2]
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 1);
    sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 2);
    const int rr = g + 8 * i;
    if (t4 == 0) { MS[(warp * kRowTile + rr) * 2] = m[i]; MS[(warp * kRowTile + rr) * 2 + 1] = sum[i]; }
    float* dst = O + (warp * kRowTile + rr) * lo + 2 * t4;
#pragma unroll
    for (int n = 0; n < 2 * NK; ++n)
      if (n < 2 * nk) *reinterpret_cast<float2*>(dst + 8 * n) = make_float2(acc[n][2 * i], acc[n][2 * i + 1]);
  }
  __syncthreads();
  const int rows = min(kRowTile, R - row0);
  const int64_t prow = (int64_t)p.G * p.B * gridDim.y * kRowTile;              // rows of one split's part
  const int64_t at = ((int64_t)bg * gridDim.y + rt) * kRowTile;
  auto finish = [&](int row, int c, float x, float mt, float sum_) {
    const int l = row / p.group, h = kh * p.group + row - l * p.group;
    x *= 1.0f / (p.sink > 0.f ? fmaf(p.sink, exp2f(-mt), sum_) : sum_);
    const int64_t e = (int64_t)h * d + c;
    if (p.gate) x *= seq::sigmoid_t<__nv_bfloat16>(__bfloat162float(p.gate[b * p.gb + l * p.gl + e]));
    p.out[b * p.ob + l * p.ol + e] = __float2bfloat16_rn(x);
  };
  for (int e = tid; e < rows * d; e += kThreads) {
    const int rr = e / d, c = e - rr * d;
    float mw[kWarps], mt = -INFINITY;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) { mw[w] = MS[(w * kRowTile + rr) * 2]; mt = fmaxf(mt, mw[w]); }
    if (p.splits == 1 && p.sink > 0.f) mt = fmaxf(mt, 0.f);
    const float base = mt == -INFINITY ? 0.f : mt;
    float x = 0.f, y = 0.f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
      const float f = weight(mw[w], base);
      x = fmaf(f, O[(w * kRowTile + rr) * lo + c], x);
      y = fmaf(f, MS[(w * kRowTile + rr) * 2 + 1], y);
    }
    if (p.splits == 1) {
      finish(row0 + rr, c, x, base, y);
    } else {
      float* dst = p.part + ((int64_t)split * prow + at + rr) * (d + 2);
      dst[c] = x;
      if (c == 0) { dst[d] = mt; dst[d + 1] = y; }
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
  float* W = reinterpret_cast<float*>(smem);                   // [rows][splits], then [rows] sums and maxima
  float* T = W + rows * p.splits;
  const int64_t step = prow * (d + 2);
  for (int rr = warp; rr < rows; rr += kWarps) {
    const float* src = p.part + (at + rr) * (d + 2) + d;
    float mt = p.sink > 0.f ? 0.f : -INFINITY;
    for (int s = lane; s < p.splits; s += 32) mt = fmaxf(mt, __ldcg(src + s * step));
    mt = warp_max(mt);
    float y = 0.f;
    for (int s = lane; s < p.splits; s += 32) {
      const float w = weight(__ldcg(src + s * step), mt);
      W[rr * p.splits + s] = w;
      y = fmaf(w, __ldcg(src + s * step + 1), y);
    }
    y = warp_sum(y);
    if (lane == 0) { T[2 * rr] = mt; T[2 * rr + 1] = y; }
  }
  __syncthreads();
  for (int e = tid; e < rows * d; e += kThreads) {
    const int rr = e / d, c = e - rr * d;
    const float* src = p.part + (at + rr) * (d + 2) + c;
    float x = 0.f;
#pragma unroll 8
    for (int s = 0; s < p.splits; ++s) x = fmaf(W[rr * p.splits + s], __ldcg(src + s * step), x);
    finish(row0 + rr, c, x, T[2 * rr], T[2 * rr + 1]);
  }
}

constexpr int kMaxSplits = 296;

size_t smem_bytes(int d) {
  const size_t ring = (size_t)(kRowTile + kWarps * kStages * kTile) * (d + kPad) * 2 + kWarps * kStages * kTile * 4;
  const size_t merge = (size_t)kRowTile * (d + kPad) * 2 + (size_t)kWarps * kRowTile * (d + 4 + 2) * 4;
  const size_t parts = (size_t)kRowTile * (kMaxSplits + 2) * 4;
  return ring > merge ? (ring > parts ? ring : parts) : (merge > parts ? merge : parts);
}

template <int NK>
int launch_nk(const P& p, cudaStream_t st) {
  const cudaError_t e = cudaFuncSetAttribute(tied_decode_kernel<NK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_bytes(16 * NK));
  if (e != cudaSuccess) return (int)e;
  tied_decode_kernel<NK><<<dim3(p.splits, (p.L * p.group + kRowTile - 1) / kRowTile, p.B * p.G), kThreads, smem_bytes(p.d), st>>>(p);
  return (int)cudaGetLastError();
}

}  // namespace

int tied_decode_splits(int B, int R, int G, int max_len) {
  const int64_t ctas = (int64_t)B * G * ((R + kRowTile - 1) / kRowTile);
  int s = (int)(kMaxSplits / (ctas > 0 ? ctas : 1));           // two CTAs per SM
  const int most = (max_len + kWarps * kTile - 1) / (kWarps * kTile);   // a tile per warp at full length
  if (s > most) s = most;
  return s < 1 ? 1 : s;
}

size_t tied_decode_scratch_bytes(int B, int R, int G, int d, int max_len) {
  const int s = tied_decode_splits(B, R, G, max_len);
  return s > 1 ? (size_t)s * B * G * ((R + kRowTile - 1) / kRowTile * kRowTile) * (d + 2) * sizeof(float) : 0;
}

// factor rows may be read up to the next multiple of 32 keys.  BASED_ERR_IMPL: sizes or strides this kernel does not take.
int launch_tied_decode(const void* q, const void* cache, const float* factor, const void* gate, void* out, void* scratch,
                       size_t scratch_bytes, int* count, int count_len, int B, int L, int H, int G, int d, int max_len,
                       int64_t qb, int64_t ql, int64_t cb, int64_t cl, int64_t fb, int64_t fh, int64_t gb, int64_t gl,
                       int64_t ob, int64_t ol, const int32_t* offsets, int offset, float scale, float sink,
                       cudaStream_t stream) {
  const int group = H / G, R = L * group, tiles = (R + kRowTile - 1) / kRowTile;
  if (d % 16 || d > 256 || (int64_t)B * G > 65535 || tiles > 65535 || smem_bytes(d) > 227 * 1024) return BASED_ERR_IMPL;
  if (!aligned16(q) || !aligned16(cache) || !aligned16(factor)) return BASED_ERR_IMPL;
  const int64_t in[] = {B > 1 ? qb : 0, L > 1 ? ql : 0, B > 1 ? cb : 0, cl};
  for (int64_t s : in)
    if (s % 8) return BASED_ERR_IMPL;
  if ((G > 1 && fh % 4) || (B > 1 && fb % 4) || fh < (max_len + kTile - 1) / kTile * kTile) return BASED_ERR_IMPL;
  int splits = tied_decode_splits(B, R, G, max_len);
  if (!count || count_len < (int64_t)B * G * tiles) splits = 1;   // many rows fill the machine without a split
  if (splits > 1 && (!scratch || !aligned16(scratch) || scratch_bytes < tied_decode_scratch_bytes(B, R, G, d, max_len)))
    return BASED_ERR_SCRATCH;
  const P p{static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(cache),
            static_cast<const __nv_bfloat16*>(gate), factor, static_cast<__nv_bfloat16*>(out), static_cast<float*>(scratch),
            count, offsets, offset, B, L, G, group, d, splits, max_len, qb, ql, cb, cl, fb, fh, gb, gl, ob, ol,
            scale * 1.4426950408889634f, sink};
  if (d <= 64) return launch_nk<4>(p, stream);
  if (d <= 128) return launch_nk<8>(p, stream);
  return launch_nk<16>(p, stream);
}

}  // namespace based
