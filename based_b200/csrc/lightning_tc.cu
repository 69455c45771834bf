// Linear attention with one constant decay g per head over prompts and portions, in chunks of 128 tokens on the sm_100a
// tensor cores.  With q, k, v = silu of the projections, i, j places in a chunk of n tokens, S0 the state before it:
//   o_i = g^(i+1) S0^T q_i + sum_{j <= i} g^(i-j) (q_i . k_j) v_j
//   S   = g^n S0 + sum_j k_j (g^(n-1-j) v_j)^T
// One CTA walks the chunks of one (batch, head) (or of a slice of its value columns) with the state as a TMEM accumulator:
//   warps 0-3    scores: (Q K^T)_ij times g^(i-j) to P (bf16, in the scores' columns); read-out: O = P V + g^(i+1) Q S0
//   warps 4-7    state: S0 (TMEM) to the bf16 operand of Q S0, and g^n S0 back to TMEM
//   warps 8, 9   MMA issue; TMA loads of v and prefetches into L2
//   warps 12-27  operands: silu of the next chunk while the tensor cores work on this one.  q and k wait in registers, the
//                second buffer that shared memory has no room for; v arrives by TMA in one of two buffers and is replaced
//                by its silu in place.  When a chunk's read-out is complete its v buffer takes the output tile on its way
//                to a TMA store
// 32-bit in the recurrence: the state is the fp32 accumulator and is scaled in fp32; g^(n-1-j) v_j enters as a bf16 pair
// hi + lo (16 mantissa bits) against k as the activation stored it.  Scores and decays are fp32 until P, and nothing feeds
// the read-out back.
#include <initializer_list>
#include <mutex>

#include "seq_common.cuh"
#include "tcgen05.cuh"
#include "tma.cuh"

namespace based {

__device__ unsigned int g_tc_status_lightning = 0;

namespace {

using namespace tc;
using bf16 = __nv_bfloat16;

constexpr int C = 128;                      // tokens per chunk
constexpr int kLoaders = 512, NT = 12 * 32 + kLoaders;   // seven warpgroups; warps 10 and 11 are idle
// registers per thread: 72 at launch; the loaders take what the others leave (7 * 72 = 72 + 40 + 40 + 4 * 88)
constexpr int kStateRegs = 40, kMmaRegs = 40, kLoadRegs = 88;
constexpr int kItems = C * 16 / kLoaders;   // 16-byte pieces per thread and tensor at 128 columns
constexpr uint32_t kAtom = 128 * 128;       // bytes of 128 rows x 64 columns
constexpr int kTables = 32 + 132 + 32;

struct Params {
  CUtensorMap mq, mk, mv, mo;               // [B][H][L][.]; q and k for prefetches into L2
  const bf16 *q, *k;
  const float* decay;
  float* state;
  bf16* out;
  const int32_t* offsets;
  int64_t qb, ql, kb, kl, ob, ol;
  int offset, L, H, d, dv, cols, tma_out;   // cols: value columns per CTA
  unsigned int* status;
};

__device__ __forceinline__ float ex2(float x) { float r; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x)); return r; }
__device__ __forceinline__ float rcp(float x) { float r; asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x)); return r; }

// two fp32 values in one 64-bit register, for the packed arithmetic instructions
__device__ __forceinline__ uint64_t pair(float lo, float hi) { uint64_t r; asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi)); return r; }
__device__ __forceinline__ void split(uint64_t v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) { uint64_t r; asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b)); return r; }
__device__ __forceinline__ uint64_t add2(uint64_t a, uint64_t b) { uint64_t r; asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b)); return r; }
__device__ __forceinline__ uint32_t pack2(uint64_t v) { float lo, hi; split(v, lo, hi); return pack_bf16(lo, hi); }

// volatile: stays where it is written, a chunk ahead of its use
__device__ __forceinline__ uint4 load16(const bf16* src) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.b32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(src));
  return v;
}

// silu of four packed values; the four sigmoids share one reciprocal.  Below -20 silu counts as its value there, -4e-8.
__device__ __forceinline__ void silu4(uint32_t& u, uint32_t& w) {
  asm("max.bf16x2 %0, %0, %1;" : "+r"(u) : "r"(0xc1a0c1a0u));
  asm("max.bf16x2 %0, %0, %1;" : "+r"(w) : "r"(0xc1a0c1a0u));
  const uint64_t x = pair(seq::bf16_lo(u), seq::bf16_hi(u)), y = pair(seq::bf16_lo(w), seq::bf16_hi(w));
  const uint64_t nl = pair(-1.4426950408889634f, -1.4426950408889634f), one = pair(1.f, 1.f);
  float a, b, c, d;
  split(mul2(x, nl), a, b);
  split(mul2(y, nl), c, d);
  split(add2(pair(ex2(a), ex2(b)), one), a, b);    // at most 2^29 each
  split(add2(pair(ex2(c), ex2(d)), one), c, d);
  const float ab = a * b, cd = c * d, r = rcp(ab * cd), rab = r * cd, rcd = r * ab;
  u = pack2(mul2(x, mul2(pair(rab, rab), pair(b, a))));
  w = pack2(mul2(y, mul2(pair(rcd, rcd), pair(d, c))));
}

__global__ void __launch_bounds__(NT, 1) lightning_tc_kernel(const __grid_constant__ Params p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
  const uint32_t sb = smem_u32(smem);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.x, b = blockIdx.y, col0 = blockIdx.z * p.cols;
  const int cols = min(p.cols, p.dv - col0);
  const int nc = (p.L + C - 1) / C;
  const int aq = (p.d + 63) / 64, av = (p.cols + 63) / 64;
  // shared memory: Q, K (always two atoms: its transpose is a 128-row operand), two of V, hi and lo of the decayed V, S0
  const uint32_t SM_K = aq * kAtom, SM_V = SM_K + 2 * kAtom, SM_W = SM_V + 2 * av * kAtom, SM_S = SM_W + 2 * av * kAtom,
                 SM_POW = SM_S + av * kAtom, SM_BAR = SM_POW + kTables * 4;
  float* pz = reinterpret_cast<float*>(smem + SM_POW);   // 32 zeros, g^0 .. g^128
  float* pw = pz + 32;
  float* pr = pw + 132;                                  // g^31 .. g^0
  const uint32_t B_FULL = sb + SM_BAR, B_A = B_FULL + 8, B_P = B_FULL + 16, B_S0 = B_FULL + 24, B_S = B_FULL + 32,
                 B_O = B_FULL + 40, B_OF = B_FULL + 48, B_VF = B_FULL + 56, B_R = B_FULL + 64;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem + SM_BAR + 80);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  if (tid == 0) {
    mbar_init(B_FULL, kLoaders); mbar_init(B_A, 1); mbar_init(B_P, 128); mbar_init(B_S0, 128); mbar_init(B_S, 1);
    mbar_init(B_O, 1); mbar_init(B_OF, 128); mbar_init(B_VF, 1); mbar_init(B_R, 1); mbar_init(B_R + 8, 1);
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (tid <= C) {   // powers by squaring
    float r = 1.f, x = p.decay[h];
    for (int e = tid; e > 0; e >>= 1) { if (e & 1) r *= x; x *= x; }
    pw[tid] = r;
    if (tid < 32) { pz[tid] = 0.f; pr[31 - tid] = r; }
  }
  for (uint32_t i = tid * 16; i < 2 * kAtom; i += NT * 16) *reinterpret_cast<uint4*>(smem + SM_K + i) = make_uint4(0, 0, 0, 0);
  fence_proxy_async();
  if (warp == 8) tmem_alloc(smem_u32(tmem_slot), 512);
  fence_before_sync();
  __syncthreads();
  fence_after_sync();
  const uint32_t tmem = *tmem_slot;
  constexpr uint32_t TM_A = 0, TM_S = 128, TM_O = 256, TM_I = 384;

  if (warp >= 12) {
    asm volatile("setmaxnreg.inc.sync.aligned.u32 %0;" ::"n"(kLoadRegs));
    // ---------------- loads, silu, operands
    // a thread keeps one 16-byte column and takes every `step`-th row of it; a row's columns are padded to a power of two
    const int t = tid - 12 * 32;
    const int cq = p.d / 8, cv = cols / 8;
    const int wq = 32 - __clz(cq - 1), wv = 32 - __clz(cv - 1);           // log2 of the padded widths
    const int rowq = t >> wq, rowv = t >> wv, colq = t & ((1 << wq) - 1), colv = t & ((1 << wv) - 1);
    const int stepq = kLoaders >> wq, stepv = kLoaders >> wv;
    const bool onq = colq < cq && rowq < C, onv = colv < cv && rowv < C;
    const bf16* q = p.q + b * p.qb + (int64_t)h * p.d + rowq * p.ql + colq * 8;
    const bf16* k = p.k + b * p.kb + (int64_t)h * p.d + rowq * p.kl + colq * 8;
    // steps are multiples of 8 rows (or there is one row only): the swizzle is the same for all of a thread's rows
    const uint32_t atq = (colq >> 3) * kAtom + tma::sw128_offset(rowq & (C - 1), colq & 7), atv = (colv >> 3) * kAtom + tma::sw128_offset(rowv & (C - 1), colv & 7);
    uint4 rq[kItems], rk[kItems];
    auto load = [&](uint4 (&r)[kItems], const bf16* src, int64_t stride, int row, int step, bool on, int n) {
#pragma unroll
      for (int i = 0; i < kItems; ++i)
        if (i * step < C) r[i] = on && row + i * step < n ? load16(src + i * step * stride) : make_uint4(0, 0, 0, 0);
    };
    auto act = [&](uint4 (&r)[kItems], int step) {
#pragma unroll
      for (int i = 0; i < kItems; ++i)
        if (i * step < C) { silu4(r[i].x, r[i].y); silu4(r[i].z, r[i].w); }
    };
    load(rq, q, p.ql, rowq, stepq, onq, min(C, p.L));
    load(rk, k, p.kl, rowq, stepq, onq, min(C, p.L));
    for (int c = 0; c < nc; ++c) {
      const int n = min(C, p.L - c * C);
      uint8_t* vb = smem + SM_V + (c & 1) * av * kAtom + atv;
      act(rq, stepq);
      act(rk, stepq);
      mbar_wait_bounded(B_R + 8 * (c & 1), (c >> 1) & 1, abort_flag, p.status, 1u << 10);
      if (onv) {
        uint4 rv[kItems];
#pragma unroll
        for (int i = 0; i < kItems; ++i)
          if (i * stepv < C) rv[i] = *reinterpret_cast<const uint4*>(vb + i * stepv * 128);
        act(rv, stepv);
#pragma unroll
        for (int i = 0; i < kItems; ++i)
          if (i * stepv < C) *reinterpret_cast<uint4*>(vb + i * stepv * 128) = rv[i];
      }
      if (c > 0) mbar_wait_bounded(B_S, (c - 1) & 1, abort_flag, p.status, 1u << 0);   // Q, K and W of the chunk before are free
      if (onq) {
#pragma unroll
        for (int i = 0; i < kItems; ++i)
          if (i * stepq < C) {
            *reinterpret_cast<uint4*>(smem + atq + i * stepq * 128) = rq[i];
            *reinterpret_cast<uint4*>(smem + SM_K + atq + i * stepq * 128) = rk[i];
          }
      }
      if (onv) {
#pragma unroll
        for (int i = 0; i < kItems; ++i)
          if (i * stepv < C) {
            uint8_t* dst = smem + SM_W + atv + i * stepv * 128;
            const uint4 r = *reinterpret_cast<const uint4*>(vb + i * stepv * 128);
            const float f = pw[max(n - 1 - rowv - i * stepv, 0)];      // rows past the end are zero
            const uint64_t f2 = pair(f, f);
            uint32_t hi[4], lo[4];
            const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
            for (int m = 0; m < 4; ++m) {
              float x, y;
              split(mul2(pair(seq::bf16_lo(w[m]), seq::bf16_hi(w[m])), f2), x, y);
              hi[m] = pack_bf16(x, y);
              lo[m] = pack_bf16(x - seq::bf16_lo(hi[m]), y - seq::bf16_hi(hi[m]));
            }
            *reinterpret_cast<uint4*>(dst) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
            *reinterpret_cast<uint4*>(dst + av * kAtom) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
          }
      }
      fence_proxy_async();
      mbar_arrive(B_FULL);
      if (c + 1 < nc) {
        q += C * p.ql;
        k += C * p.kl;
        load(rq, q, p.ql, rowq, stepq, onq, min(C, p.L - (c + 1) * C));
        load(rk, k, p.kl, rowq, stepq, onq, min(C, p.L - (c + 1) * C));
      }
    }
  } else if (warp >= 8) {
    asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(kMmaRegs));
    if (warp == 8) {
    // ---------------- MMA issue (converged warp, one elected lane)
    const uint32_t tm = __shfl_sync(0xffffffffu, tmem, 0);
    const bool leader = elect_one_sync();
    const uint32_t id_a = make_idesc_bf16(128, C, 0, 0), id_i = make_idesc_bf16(128, cols, 0, 1), id_s = make_idesc_bf16(128, cols, 1, 1);
    const uint64_t dk_t = make_smem_desc_sw128(sb + SM_K, kAtom, 1024), dv_[2] = {make_smem_desc_sw128(sb + SM_V, kAtom, 1024), make_smem_desc_sw128(sb + SM_V + av * kAtom, kAtom, 1024)};
    const uint64_t dw0 = make_smem_desc_sw128(sb + SM_W, kAtom, 1024), dw1 = make_smem_desc_sw128(sb + SM_W + av * kAtom, kAtom, 1024);
    const uint64_t ds = make_smem_desc_sw128(sb + SM_S, kAtom, 1024);
    const int ks = p.d / 16;
    for (int c = 0; c < nc; ++c) {
      const uint32_t ph = c & 1;
      mbar_wait_bounded(B_FULL, ph, abort_flag, p.status, 1u << 1);
      fence_after_sync();
      for (int k = 0; k < ks; ++k) {   // 16 columns are 32 bytes of a row, four to an atom
        const uint32_t at = (k >> 2) * kAtom + (k & 3) * 32;
        const uint64_t da = make_smem_desc_sw128(sb + at, 16, 1024), db = make_smem_desc_sw128(sb + SM_K + at, 16, 1024);
        if (leader) mma_ss(tm + TM_A, da, db, id_a, k > 0 ? 1u : 0u);
      }
      if (leader) mma_commit(B_A);
      __syncwarp();
      mbar_wait_bounded(B_S0, ph, abort_flag, p.status, 1u << 2);
      if (c > 0) mbar_wait_bounded(B_OF, ph ^ 1, abort_flag, p.status, 1u << 3);
      fence_after_sync();
      for (int k = 0; k < ks; ++k) {   // 16 rows of S0 are 2048 bytes
        const uint64_t da = make_smem_desc_sw128(sb + (k >> 2) * kAtom + (k & 3) * 32, 16, 1024);
        if (leader) mma_ss(tm + TM_I, da, ds + 128 * k, id_i, k > 0 ? 1u : 0u);
      }
      // the read-out before the state: its buffers have the longer way back
      mbar_wait_bounded(B_P, ph, abort_flag, p.status, 1u << 4);
      fence_after_sync();
#pragma unroll
      for (int k = 0; k < C / 16; ++k)
        if (leader) mma_ts(tm + TM_O, tm + TM_A + 8 * k, (ph ? dv_[1] : dv_[0]) + 128 * k, id_i, k > 0 ? 1u : 0u);
      if (leader) mma_commit(B_O);
#pragma unroll
      for (int k = 0; k < C / 16; ++k) {
        if (leader) mma_ss(tm + TM_S, dk_t + 128 * k, dw0 + 128 * k, id_s, 1u);
        if (leader) mma_ss(tm + TM_S, dk_t + 128 * k, dw1 + 128 * k, id_s, 1u);
      }
      if (leader) mma_commit(B_S);     // every operand of this chunk read
      __syncwarp();
    }
    } else if (warp == 9 && lane == 0) {
      // ---------------- v by TMA; the chunk after the next into L2
      for (int c = 0; c < nc; ++c) {
        if (c >= 2) mbar_wait_bounded<false>(B_VF, c & 1, abort_flag, p.status, 1u << 8);   // chunk c - 2 has given its output away
        const uint32_t full = B_R + 8 * (c & 1);
        tma::mbar_expect_tx(full, av * kAtom);
        for (int a = 0; a < av; ++a) tma::load_4d(sb + SM_V + ((c & 1) * av + a) * kAtom, &p.mv, full, col0 + 64 * a, c * C, h, b);
        if (c + 1 < nc) {
          for (int a = 0; a < av; ++a) tma::prefetch_4d(&p.mv, col0 + 64 * a, (c + 1) * C, h, b);
          for (int a = 0; a < aq; ++a) {
            tma::prefetch_4d(&p.mq, 64 * a, (c + 1) * C, h, b);
            tma::prefetch_4d(&p.mk, 64 * a, (c + 1) * C, h, b);
          }
        }
      }
    }
  } else if (warp >= 4) {
    asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(kStateRegs));
    // ---------------- state: one row (key dimension) per thread
    const int row = tid - 128;
    const uint32_t ts = tmem + ((uint32_t)((warp & 3) * 32) << 16) + TM_S;
    const bool live = row < p.d, fresh = seq::position0(p.offsets, p.offset, b) == 0;
    float* st = p.state + (((int64_t)b * p.H + h) * p.d + (live ? row : 0)) * p.dv + col0;
    for (int c = 0; c <= nc; ++c) {
      const float g = c < nc ? pw[min(C, p.L - c * C)] : 0.f;
      if (c > 0) {
        mbar_wait_bounded(B_S, (c - 1) & 1, abort_flag, p.status, 1u << 5);
        fence_after_sync();
      }
      for (int x = 0; x < cols; x += 16) {
        uint32_t s[16];
        if (c > 0) {
          tmem_ld16(ts + x, s);
          tmem_ld_wait();
        } else {
#pragma unroll
          for (int i = 0; i < 16; i += 4) {
            float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
            if (live && !fresh) f = *reinterpret_cast<const float4*>(st + x + i);
            s[i] = __float_as_uint(f.x); s[i + 1] = __float_as_uint(f.y); s[i + 2] = __float_as_uint(f.z); s[i + 3] = __float_as_uint(f.w);
          }
        }
        if (c == nc) {
          if (live) {
#pragma unroll
            for (int i = 0; i < 16; i += 4)
              *reinterpret_cast<float4*>(st + x + i) = make_float4(__uint_as_float(s[i]), __uint_as_float(s[i + 1]), __uint_as_float(s[i + 2]), __uint_as_float(s[i + 3]));
          }
        } else {
#pragma unroll
          for (int i = 0; i < 16; i += 8) {
            uint32_t w[4];
#pragma unroll
            for (int m = 0; m < 4; ++m) w[m] = pack_bf16(__uint_as_float(s[i + 2 * m]), __uint_as_float(s[i + 2 * m + 1]));
            const int cc = (x + i) >> 3;
            *reinterpret_cast<uint4*>(smem + SM_S + (cc >> 3) * kAtom + tma::sw128_offset(row, cc & 7)) = make_uint4(w[0], w[1], w[2], w[3]);
          }
#pragma unroll
          for (int i = 0; i < 16; ++i) s[i] = __float_as_uint(__uint_as_float(s[i]) * g);
          tmem_st16(ts + x, s);
        }
      }
      if (c < nc) {
        tmem_st_wait();
        fence_proxy_async();
        fence_before_sync();
        mbar_arrive(B_S0);
      }
    }
  } else {
    // ---------------- scores and read-out: one token per thread
    const int i = tid;
    const uint32_t tl = tmem + ((uint32_t)(warp * 32) << 16);
    bf16* out = p.out + b * p.ob + (int64_t)h * p.dv + col0;
    for (int c = 0; c < nc; ++c) {
      mbar_wait_bounded(B_A, c & 1, abort_flag, p.status, 1u << 6);
      fence_after_sync();
#pragma unroll
      for (int x = 0; x < 4; ++x) {   // 32 columns at a time: before, on and after this warp's diagonal block
        uint32_t w[16];
        if (x <= warp) {
          uint32_t r[32];
          tmem_ld32(tl + TM_A + 32 * x, r);
          tmem_ld_wait();
          if (x < warp) {             // g^(i-j) = g^(i-last column) g^(last column-j): no power of it is negative
            const float f = pw[i - 32 * x - 31];
            const uint64_t f2 = pair(f, f);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
              const float4 y = *reinterpret_cast<const float4*>(pr + 4 * j);
              w[2 * j] = pack2(mul2(pair(__uint_as_float(r[4 * j]), __uint_as_float(r[4 * j + 1])), mul2(f2, pair(y.x, y.y))));
              w[2 * j + 1] = pack2(mul2(pair(__uint_as_float(r[4 * j + 2]), __uint_as_float(r[4 * j + 3])), mul2(f2, pair(y.z, y.w))));
            }
          } else {
#pragma unroll
            for (int j = 0; j < 16; ++j)
              w[j] = pack_bf16(__uint_as_float(r[2 * j]) * pw[lane - 2 * j], __uint_as_float(r[2 * j + 1]) * pw[lane - 2 * j - 1]);
          }
        } else {
#pragma unroll
          for (int j = 0; j < 16; ++j) w[j] = 0u;
        }
        // P of columns 32 x .. goes to columns 16 x ..: already read by this thread
        tmem_st16(tl + TM_A + 16 * x, w);
      }
      tmem_st_wait();
      fence_before_sync();
      mbar_arrive(B_P);
      mbar_wait_bounded(B_O, c & 1, abort_flag, p.status, 1u << 7);
      fence_after_sync();
      const float g = pw[i + 1];
      const bool live = c * C + i < p.L;
      bf16* o = out + (int64_t)(c * C + i) * p.ol;
      uint8_t* tile = smem + SM_V + (c & 1) * av * kAtom;
      for (int x = 0; x < cols; x += 16) {
        uint32_t r0[16], r1[16], w[8];
        tmem_ld16(tl + TM_O + x, r0);
        tmem_ld16(tl + TM_I + x, r1);
        tmem_ld_wait();
#pragma unroll
        for (int m = 0; m < 8; ++m)
          w[m] = pack_bf16(fmaf(__uint_as_float(r1[2 * m]), g, __uint_as_float(r0[2 * m])),
                           fmaf(__uint_as_float(r1[2 * m + 1]), g, __uint_as_float(r0[2 * m + 1])));
        const uint4 lo = make_uint4(w[0], w[1], w[2], w[3]), hi = make_uint4(w[4], w[5], w[6], w[7]);
        if (p.tma_out) {
          uint8_t* atom = tile + (x >> 6) * kAtom;
          *reinterpret_cast<uint4*>(atom + tma::sw128_offset(i, (x & 63) >> 3)) = lo;
          *reinterpret_cast<uint4*>(atom + tma::sw128_offset(i, ((x & 63) >> 3) + 1)) = hi;
        } else if (live) {
          *reinterpret_cast<uint4*>(o + x) = lo;
          *reinterpret_cast<uint4*>(o + x + 8) = hi;
        }
      }
      fence_before_sync();
      mbar_arrive(B_OF);
      if (p.tma_out) fence_proxy_async();
      asm volatile("bar.sync 1, 128;" ::: "memory");   // these four warps
      if (tid == 0) {
        if (p.tma_out) {               // rows past the sequence and columns past the head are clipped
          for (int a = 0; a < av; ++a) tma::store_4d(&p.mo, sb + SM_V + ((c & 1) * av + a) * kAtom, col0 + 64 * a, c * C, h, b);
          bulk_commit();
          bulk_wait_read_all();
        }
        mbar_arrive(B_VF);
      }
    }
    if (tid == 0) bulk_wait_all();
  }
  __syncwarp();
  fence_before_sync();
  __syncthreads();
  if (warp == 8) {
    fence_after_sync();
    tmem_dealloc(tmem, 512);
  }
}

}  // namespace

int read_tc_status_lightning(unsigned int* out, int reset) {
  unsigned int v = 0;
  cudaError_t e = cudaMemcpyFromSymbol(&v, g_tc_status_lightning, sizeof(v));
  if (e != cudaSuccess) return (int)e;
  if (out) *out = v;
  if (reset && v != 0) {
    v = 0;
    e = cudaMemcpyToSymbol(g_tc_status_lightning, &v, sizeof(v));
  }
  return (int)e;
}

// BASED_ERR_IMPL: sizes or strides this kernel does not take.
int launch_lightning_tc(const void* q, const void* k, const void* v, const float* decay, float* state, void* out, int B, int L,
                        int H, int d, int dv, Strides2 sq, Strides2 sk, Strides2 sv, Strides2 so, const int32_t* offsets,
                        int offset, cudaStream_t stream) {
  if (d % 16 || d > 128 || dv % 16 || B > 65535) return BASED_ERR_IMPL;
  if (!aligned16(q) || !aligned16(k) || !aligned16(v) || !aligned16(out) || !aligned16(state)) return BASED_ERR_IMPL;
  for (const Strides2& s : {sq, sk, sv, so})
    if (s.h % 8 || (B > 1 && s.b % 8)) return BASED_ERR_IMPL;
  Params p{{}, {}, {}, {}, static_cast<const bf16*>(q), static_cast<const bf16*>(k), decay, state, static_cast<bf16*>(out), offsets,
           sq.b, sq.h, sk.b, sk.h, so.b, so.h, offset, L, H, d, dv, 0, 0, nullptr};
  // few (batch, head) pairs: their value columns over several CTAs, at least 32 each
  int slices = (dv + 127) / 128;
  while ((int64_t)B * H * slices * 2 <= 148 && dv / (slices * 2) >= 32) slices *= 2;
  p.cols = ((dv + slices - 1) / slices + 15) / 16 * 16;
  slices = (dv + p.cols - 1) / p.cols;
  const int aq = (d + 63) / 64, av = (p.cols + 63) / 64;
  constexpr int kMaxSmem = 227 * 1024;
  const int smem = (aq + 2 + 5 * av) * (int)kAtom + kTables * 4 + 88 + 1024;
  if (smem > kMaxSmem || slices > 65535) return BASED_ERR_IMPL;
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
      e = cudaGetSymbolAddress(reinterpret_cast<void**>(&addr), g_tc_status_lightning);
      if (e != cudaSuccess) return (int)e;
      e = cudaFuncSetAttribute(lightning_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxSmem);
      if (e != cudaSuccess) return (int)e;
      status[dev] = addr;
    }
    p.status = status[dev];
  }
  static tma::MapCache maps;
  auto fix = [](int64_t st, int extent) { return extent == 1 ? (int64_t)8 : st; };
  auto get_map = [&](CUtensorMap* m, const void* base, int w, const Strides2& st) -> int {
    const int64_t sl = fix(st.h, L), sbt = fix(st.b, B);
    if (sl <= 0 || sbt <= 0) return 1;
    const tma::MapKey key = tma::make_key(base, w, L, H, B, 0, sl, w, sbt, 0, 64, C, 0, 4);
    if (maps.find(key, m)) return 0;
    if (tma::encode_bf16_4d_sw128(m, base, w, L, H, B, sl, w, sbt, 64, C)) return 1;
    maps.put(key, *m);
    return 0;
  };
  if (get_map(&p.mq, q, d, sq) || get_map(&p.mk, k, d, sk) || get_map(&p.mv, v, dv, sv) || get_map(&p.mo, out, dv, so)) return BASED_ERR_IMPL;
  p.tma_out = slices == 1 || p.cols % 64 == 0;   // a slice's tile must not reach into the next one
  lightning_tc_kernel<<<dim3(H, B, slices), NT, smem, stream>>>(p);
  return (int)cudaGetLastError();
}

}  // namespace based
