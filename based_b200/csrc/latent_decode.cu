// Latent attention in its absorbed form for a few query rows: every head of every query attends over the SAME cached
// rows [latent | rotated key], so 16 (query, head) rows share one read of the cache.
//   s[row, t] = (qa[row] . c_t + qr[row] . kr_t) * scale,   ctx[row] = sigmoid(gate[row]) * sum_t softmax(s)[row, t] c_t
// HBM-bound on the cache.  A CTA of 8 warps walks its share of the keys in tiles of 32, two tiles in flight
// (cp.async), two CTAs per SM so that one's products run under the other's waits; scores and context use mma.sync m16n8k16 (16 rows are exactly the tile height, the operands are a few
// hundred flops per cached byte at most), softmax in fp32.  Several CTAs split the keys of a sequence; a second launch
// merges their partial results.  The split follows the sequence's current length, read on the device.
#include <initializer_list>

#include "seq_common.cuh"
#include "tcgen05.cuh"

namespace based {
namespace {

constexpr int kWarps = 8, kThreads = kWarps * 32, kTile = 32, kPad = 8;
constexpr int kRows = 16 / kWarps;   // softmax rows per warp

struct P {
  const __nv_bfloat16 *q1, *q2, *cache, *gate;
  __nv_bfloat16* out;
  float* part;                 // [splits][B][R][r + 2]
  const int32_t* offsets;
  int offset, B, L, H, R, r, rd, splits, max_len;
  Strides3 sq1, sq2, so;
  int64_t cb, cl, gb, gl;
  float scale_log2e;
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

// NW: 8-column groups of the context per warp
template <int NW>
__global__ void __launch_bounds__(kThreads, 2) latent_decode_kernel(const P p) {
  extern __shared__ __align__(16) uint8_t smem[];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int split = blockIdx.x, row0 = blockIdx.y * 16, b = blockIdx.z;
  const int D = p.r + p.rd, ld = D + kPad;      // row stride: an odd number of 16-byte units, so ldmatrix has no conflicts
  __nv_bfloat16* Q = reinterpret_cast<__nv_bfloat16*>(smem);                 // [16][ld]
  __nv_bfloat16* K = Q + 16 * ld;                                            // [2][32][ld]
  float* S = reinterpret_cast<float*>(K + 2 * kTile * ld);                   // [2][16][32 + 4]: two halves of the dims
  __nv_bfloat16* Pm = reinterpret_cast<__nv_bfloat16*>(S + 32 * (kTile + 4)); // [16][32 + 8]
  float* corr = reinterpret_cast<float*>(Pm + 16 * (kTile + 8));             // [16]
  float* msum = corr + 16;                                                   // [16][2]
  const int pos0 = seq::position0(p.offsets, p.offset, b);
  const int len = min(pos0 + p.L, p.max_len);
  const int tiles = (len + kTile - 1) / kTile, per = (tiles + p.splits - 1) / p.splits;
  const int t0 = min(split * per, tiles), t1 = min(t0 + per, tiles);

  const int chunks = D / 8;
  for (int e = tid; e < 16 * chunks; e += kThreads) {
    const int i = e / chunks, c = (e - i * chunks) * 8, row = row0 + i;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (row < p.R) {
      const int l = row / p.H, h = row - l * p.H;
      v = c < p.r ? *reinterpret_cast<const uint4*>(p.q1 + b * p.sq1.b + l * p.sq1.l + h * p.sq1.h + c)
                  : *reinterpret_cast<const uint4*>(p.q2 + b * p.sq2.b + l * p.sq2.l + h * p.sq2.h + (c - p.r));
    }
    *reinterpret_cast<uint4*>(Q + i * ld + c) = v;
  }
  const __nv_bfloat16* cache = p.cache + b * p.cb;
  auto fetch = [&](int t, int buf) {
#pragma unroll
    for (int n = 0; n < kTile / kWarps; ++n) {   // a warp copies whole rows, a lane every 32nd 16-byte piece
      const int i = n * kWarps + warp, key = t * kTile + i;
      const __nv_bfloat16* src = cache + (int64_t)(key < len ? key : 0) * p.cl;
      const uint32_t dst = tc::smem_u32(K + (buf * kTile + i) * ld);
      for (int c = lane; c < chunks; c += 32) tc::cp_async16(dst + c * 16, src + c * 8, key < len);
    }
    tc::cp_async_commit();
  };
  float acc[NW][4];
#pragma unroll
  for (int i = 0; i < NW; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
  // rows kRows * warp .. of the softmax belong to this warp; every lane keeps a copy of the maximum
  float m[kRows], sum[kRows];
#pragma unroll
  for (int i = 0; i < kRows; ++i) { m[i] = -INFINITY; sum[i] = 0.f; }
  if (t0 < t1) fetch(t0, 0);
  const int g = lane >> 2, t4 = lane & 3;
  for (int t = t0; t < t1; ++t) {
    const int buf = (t - t0) & 1;
    if (t + 1 < t1) {
      fetch(t + 1, buf ^ 1);
      tc::cp_async_wait_1();
    } else {
      tc::cp_async_wait_all();
    }
    __syncthreads();
    const __nv_bfloat16* Kt = K + buf * kTile * ld;
    {  // scores of keys 8 (warp mod 4) .. + 7 over one half of the dims, in pairs of 16
      const int kq = warp & 3, pairs = (D / 16 + 1) / 2, kb = (warp >> 2) ? (pairs + 1) / 2 : 0, ke = (warp >> 2) ? pairs : (pairs + 1) / 2;
      float s[2][4] = {};
      const uint32_t qa = tc::smem_u32(Q + (lane & 15) * ld + (lane >> 4) * 8);
      const uint32_t krow = tc::smem_u32(Kt + (8 * kq + (lane & 7)) * ld), ka = krow + (lane >> 3) * 16;   // four k-halves
#pragma unroll 3
      for (int k = kb; k < ke; ++k) {
        uint32_t a0[4], a1[4], bb[4];
        ldsm4(a0, qa + k * 64);
        if (2 * k + 1 < D / 16) {
          ldsm4(a1, qa + k * 64 + 32);
          ldsm4(bb, ka + k * 64);
          mma16816(s[0], a0, bb[0], bb[1]);
          mma16816(s[1], a1, bb[2], bb[3]);
        } else {   // the last 16 of an odd number: the upper lanes repeat their addresses
          ldsm4(bb, krow + ((lane >> 3) & 1) * 16 + k * 64);
          mma16816(s[0], a0, bb[0], bb[1]);
        }
      }
      float* Sh = S + (warp >> 2) * 16 * (kTile + 4);
      const int c = 8 * kq + 2 * t4;
      *reinterpret_cast<float2*>(Sh + g * (kTile + 4) + c) = make_float2(s[0][0] + s[1][0], s[0][1] + s[1][1]);
      *reinterpret_cast<float2*>(Sh + (g + 8) * (kTile + 4) + c) = make_float2(s[0][2] + s[1][2], s[0][3] + s[1][3]);
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      const int rr = kRows * warp + i, row = row0 + rr;
      const int last = row < p.R ? pos0 + row / p.H : -1;   // last key this row sees
      const int key = t * kTile + lane;
      const float a = key <= last ? (S[rr * (kTile + 4) + lane] + S[(16 + rr) * (kTile + 4) + lane]) * p.scale_log2e : -INFINITY;
      const float mn = fmaxf(m[i], warp_max(a));
      const float base = mn == -INFINITY ? 0.f : mn;
      const float ea = exp2f(a - base), f = exp2f(m[i] - base);
      sum[i] = fmaf(sum[i], f, ea);     // this lane's share
      m[i] = mn;
      Pm[rr * (kTile + 8) + lane] = __float2bfloat16_rn(ea);
      if (lane == 0) corr[rr] = f;
    }
    __syncthreads();
    const float f0 = corr[g], f1 = corr[g + 8];
    uint32_t pa[kTile / 16][4];
#pragma unroll
    for (int k = 0; k < kTile / 16; ++k) ldsm4(pa[k], tc::smem_u32(Pm + (lane & 15) * (kTile + 8) + k * 16 + (lane >> 4) * 8));
#pragma unroll
    for (int i = 0; i < NW; ++i) {
      const int n = warp * NW + i;
      if (n * 8 < p.r) {
        acc[i][0] *= f0; acc[i][1] *= f0; acc[i][2] *= f1; acc[i][3] *= f1;
#pragma unroll
        for (int k = 0; k < kTile / 16; k += 2) {
          uint32_t bb[4];
          ldsm4t(bb, tc::smem_u32(Kt + (k * 16 + lane) * ld + n * 8));
          mma16816(acc[i], pa[k], bb[0], bb[1]);
          mma16816(acc[i], pa[k + 1], bb[2], bb[3]);
        }
      }
    }
    __syncthreads();   // this tile's buffer, S and P are free
  }
#pragma unroll
  for (int i = 0; i < kRows; ++i) {
    const float s = warp_sum(sum[i]);
    if (lane == 0) { msum[2 * (kRows * warp + i)] = m[i]; msum[2 * (kRows * warp + i) + 1] = s; }
  }
  __syncthreads();
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int rr = g + 8 * half, row = row0 + rr;
    if (row >= p.R) continue;
    const int l = row / p.H, h = row - l * p.H;
    if (p.splits > 1) {
      float* dst = p.part + (((int64_t)split * p.B + b) * p.R + row) * (p.r + 2);
      if (warp == 0 && t4 == 0) { dst[p.r] = msum[2 * rr]; dst[p.r + 1] = msum[2 * rr + 1]; }
#pragma unroll
      for (int i = 0; i < NW; ++i) {
        const int c = (warp * NW + i) * 8 + 2 * t4;
        if (c < p.r) *reinterpret_cast<float2*>(dst + c) = make_float2(acc[i][2 * half], acc[i][2 * half + 1]);
      }
    } else {
      float f = 1.0f / msum[2 * rr + 1];
      if (p.gate) f *= seq::sigmoid_acc(__bfloat162float(p.gate[b * p.gb + l * p.gl + h]));
      __nv_bfloat16* dst = p.out + b * p.so.b + l * p.so.l + h * p.so.h;
#pragma unroll
      for (int i = 0; i < NW; ++i) {
        const int c = (warp * NW + i) * 8 + 2 * t4;
        if (c < p.r) *reinterpret_cast<uint32_t*>(dst + c) = seq::bf16x2_bits(acc[i][2 * half] * f, acc[i][2 * half + 1] * f);
      }
    }
  }
}

// G groups of splits times 128 / G column pairs per block; grid (R, B, ceil(r / (256 / G)))
template <int G>
__global__ void __launch_bounds__(128) latent_decode_merge_kernel(const P p) {
  constexpr int W = 128 / G;
  const int row = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, grp = tid / W, lane = tid % W;
  const int c = blockIdx.z * 2 * W + 2 * lane;
  const int64_t stride = (int64_t)p.B * p.R * (p.r + 2);
  const float* src = p.part + ((int64_t)b * p.R + row) * (p.r + 2);
  float m = -INFINITY;
  if (G > 1) {
    __shared__ float red[4];
    for (int s = tid; s < p.splits; s += 128) m = fmaxf(m, src[s * stride + p.r]);
    m = warp_max(m);
    if ((tid & 31) == 0) red[tid >> 5] = m;
    __syncthreads();
    m = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
  } else {
    for (int s = 0; s < p.splits; ++s) m = fmaxf(m, src[s * stride + p.r]);
  }
  float sum = 0.f, x = 0.f, y = 0.f;
#pragma unroll 4
  for (int s = grp; s < p.splits; s += G) {
    const float ms = src[s * stride + p.r];
    const float w = ms == -INFINITY ? 0.f : exp2f(ms - m);   // a split without keys wrote zeros
    sum = fmaf(w, src[s * stride + p.r + 1], sum);
    if (c < p.r) {
      const float2 v = *reinterpret_cast<const float2*>(src + s * stride + c);
      x = fmaf(w, v.x, x);
      y = fmaf(w, v.y, y);
    }
  }
  if (G > 1) {
    __shared__ float wsum[G], acc[G][2 * W];
    if (lane == 0) wsum[grp] = sum;
    acc[grp][2 * lane] = x;
    acc[grp][2 * lane + 1] = y;
    __syncthreads();
    if (grp != 0) return;
    sum = x = y = 0.f;
#pragma unroll
    for (int i = 0; i < G; ++i) { sum += wsum[i]; x += acc[i][2 * lane]; y += acc[i][2 * lane + 1]; }
  }
  if (c >= p.r) return;
  const int l = row / p.H, h = row - l * p.H;
  float f = 1.0f / sum;
  if (p.gate) f *= seq::sigmoid_acc(__bfloat162float(p.gate[b * p.gb + l * p.gl + h]));
  *reinterpret_cast<uint32_t*>(p.out + b * p.so.b + l * p.so.l + h * p.so.h + c) = seq::bf16x2_bits(x * f, y * f);
}

size_t smem_bytes(int D) {
  return (size_t)(16 + 2 * kTile) * (D + kPad) * 2 + 32 * (kTile + 4) * 4 + 16 * (kTile + 8) * 2 + 16 * 3 * 4;
}
constexpr int kMaxSmem = 227 * 1024;

template <int NW>
int launch_nw(const P& p, cudaStream_t st) {
  const cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<NW>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxSmem);
  if (e != cudaSuccess) return (int)e;
  latent_decode_kernel<NW><<<dim3(p.splits, (p.R + 15) / 16, p.B), kThreads, smem_bytes(p.r + p.rd), st>>>(p);
  if (p.splits > 16) latent_decode_merge_kernel<8><<<dim3(p.R, p.B, (p.r + 31) / 32), 128, 0, st>>>(p);
  else if (p.splits > 1) latent_decode_merge_kernel<1><<<dim3(p.R, p.B, (p.r + 255) / 256), 128, 0, st>>>(p);
  return (int)cudaGetLastError();
}

}  // namespace

int latent_decode_splits(int B, int R, int max_len) {
  const int64_t ctas = (int64_t)B * ((R + 15) / 16);
  int s = (int)(2 * 148 / (ctas > 0 ? ctas : 1));
  const int most = (max_len + 4 * kTile - 1) / (4 * kTile);   // at least four tiles per CTA at full length
  if (s > most) s = most;
  return s < 1 ? 1 : s;
}

size_t latent_decode_scratch_bytes(int B, int R, int r, int max_len) {
  const int s = latent_decode_splits(B, R, max_len);
  return s > 1 ? (size_t)s * B * R * (r + 2) * sizeof(float) : 0;
}

int launch_latent_decode(const void* q1, const void* q2, const void* cache, const void* gate, void* out, void* scratch,
                         size_t scratch_bytes, int B, int L, int H, int r, int rd, int max_len, Strides3 sq1, Strides3 sq2,
                         int64_t cb, int64_t cl, Strides3 so, int64_t gb, int64_t gl, const int32_t* offsets, int offset,
                         float scale, cudaStream_t stream) {
  const int D = r + rd;
  if (r % 8 || D % 16 || r > 512 || smem_bytes(D) > kMaxSmem || B > 65535 || (int64_t)L * H > 65535 * 16) return BASED_ERR_IMPL;
  if (!aligned16(q1) || !aligned16(q2) || !aligned16(cache) || (reinterpret_cast<uintptr_t>(out) & 3)) return BASED_ERR_IMPL;
  const int64_t in[] = {B > 1 ? sq1.b : 0, L > 1 ? sq1.l : 0, H > 1 ? sq1.h : 0, B > 1 ? sq2.b : 0, L > 1 ? sq2.l : 0,
                        H > 1 ? sq2.h : 0, B > 1 ? cb : 0, cl};
  for (int64_t s : in)
    if (s % 8) return BASED_ERR_IMPL;
  if (so.b % 2 || so.l % 2 || so.h % 2) return BASED_ERR_IMPL;
  const int R = L * H, splits = latent_decode_splits(B, R, max_len);
  if (splits > 1 && (!scratch || scratch_bytes < latent_decode_scratch_bytes(B, R, r, max_len) || !aligned16(scratch)))
    return BASED_ERR_SCRATCH;
  const P p{static_cast<const __nv_bfloat16*>(q1), static_cast<const __nv_bfloat16*>(q2),
            static_cast<const __nv_bfloat16*>(cache), static_cast<const __nv_bfloat16*>(gate),
            static_cast<__nv_bfloat16*>(out), static_cast<float*>(scratch), offsets, offset, B, L, H, R, r, rd, splits,
            max_len, sq1, sq2, so, cb, cl, gb, gl, scale * 1.4426950408889634f};
  const int nw = (r / 8 + kWarps - 1) / kWarps;
  if (nw <= 1) return launch_nw<1>(p, stream);
  if (nw <= 2) return launch_nw<2>(p, stream);
  if (nw <= 4) return launch_nw<4>(p, stream);
  return launch_nw<8>(p, stream);
}

}  // namespace based
