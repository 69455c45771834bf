// Real-gated linear recurrent unit over prompts and portions with its gate products on the tensor cores (tcgen05),
// bf16 operands, fp32 gates and state: from u and y to the gated output in one pass, nothing in between leaves the SM.
//
// One CTA per (batch row, up to 128 channels of one gate block) walks the sequence in tiles of 64 tokens.  The product is
// taken transposed, D[channel, token] = W_gate[channel, :] u[token, :]^T, so that a TMEM lane is a channel and a thread
// finds the gate values of consecutive tokens of its channel in consecutive columns.  Four groups of 128 threads own 16
// tokens of a tile each: a thread computes a_t and b_t of its tokens and the scan of (a, b) from a zero state, takes the
// state at its first token from the thread of the group before (a ring of four mbarriers), hands on the state after its
// last, and only then writes S_t * gelu(y_t): the serial part is one multiply-add per 16 tokens.
// Warp 16 loads u by TMA (two stages) and issues the MMAs (two accumulator buffers); the weights stay in shared memory.
// Warp 17 loads the y tiles and stores the output tiles, which replace y's values in place.
#include <initializer_list>
#include <mutex>

#include "seq_common.cuh"
#include "tcgen05.cuh"
#include "tma.cuh"

namespace based {

__device__ unsigned int g_tc_status_rglru = 0;

namespace {

using namespace tc;
using bf16 = __nv_bfloat16;

constexpr int TT = 64, GROUPS = 4, TG = TT / GROUPS;   // tokens per tile, groups, tokens per group
constexpr int NC = 128 * GROUPS, NT = NC + 64;
constexpr uint32_t kWAtom = 128 * 128, kUAtom = TT * 128;   // bytes of 64 columns x 128 (64) rows
constexpr float kLog2e = 1.4426950408889634f;

struct Params {
  CUtensorMap mw, mu, my, mo;    // weights [blocks][2][n][n], u [B][1][L][W], y and out [B][blocks][L][n]
  const bf16 *rb, *ib;
  const float* lam;
  float* state;
  const int32_t* offsets;
  int offset, L, W, n, slices, atoms;
  unsigned int* status;
};

__device__ __forceinline__ float ex2(float x) { float r; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x)); return r; }
__device__ __forceinline__ float rcp(float x) { float r; asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x)); return r; }
__device__ __forceinline__ float sqrt_approx(float x) { float r; asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x)); return r; }

__global__ void __launch_bounds__(NT, 1) rglru_tc_kernel(const __grid_constant__ Params p) {
  extern __shared__ __align__(1024) uint8_t smem[];
  const uint32_t sb = smem_u32(smem);
  if (sb & 1023u) {   // the swizzled tiles need this alignment; there is no room for slack
    if (threadIdx.x == 0) atomicOr(p.status, 1u << 25);
    return;
  }
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int blk = blockIdx.x / p.slices, c0 = (blockIdx.x % p.slices) * 128, b = blockIdx.y;
  const int nt = (p.L + TT - 1) / TT;
  // shared memory: W_r, W_i (atoms each), u stages, y stages (two 64-channel atoms each), carries, barriers
  const uint32_t SM_U = 2u * p.atoms * kWAtom, SM_Y = SM_U + 2u * p.atoms * kUAtom, SM_C = SM_Y + 4u * kUAtom,
                 SM_BAR = SM_C + GROUPS * 128 * 4;
  const uint32_t B_W = sb + SM_BAR, B_FULL = B_W + 8, B_D = B_FULL + 16, B_EMPTY = B_D + 16, B_Y = B_EMPTY + 16,
                 B_OUT = B_Y + 16, B_CARRY = B_OUT + 16;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem + SM_BAR + 8 * (11 + GROUPS));
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  if (tid == 0) {
    mbar_init(B_W, 1);
    for (int i = 0; i < 2; ++i) { mbar_init(B_FULL + 8 * i, 1); mbar_init(B_D + 8 * i, 1); mbar_init(B_EMPTY + 8 * i, NC); mbar_init(B_Y + 8 * i, 1); mbar_init(B_OUT + 8 * i, NC); }
    for (int i = 0; i < GROUPS; ++i) mbar_init(B_CARRY + 8 * i, 128);
    *abort_flag = 0;
    fence_mbar_init();
    fence_proxy_async();
  }
  if (warp == NC / 32) tmem_alloc(smem_u32(tmem_slot), 256);
  fence_before_sync();
  __syncthreads();
  fence_after_sync();
  const uint32_t tmem = *tmem_slot;   // buffer x: r gates in columns 128 x .., i gates in columns 128 x + 64 ..

  if (warp == NC / 32) {
    const uint32_t tmem_u = __shfl_sync(0xffffffffu, tmem, 0);
    const bool leader = elect_one_sync();
    auto load = [&](int t) {
      if (leader) {
        tma::mbar_expect_tx(B_FULL + 8 * (t & 1), (uint32_t)p.atoms * kUAtom);
        for (int a = 0; a < p.atoms; ++a)
          tma::load_4d(sb + SM_U + ((t & 1) * p.atoms + a) * kUAtom, &p.mu, B_FULL + 8 * (t & 1), blk * p.n + 64 * a, t * TT, 0, b);
      }
    };
    if (leader) {
      tma::mbar_expect_tx(B_W, 2u * p.atoms * kWAtom);
      for (int m = 0; m < 2; ++m)
        for (int a = 0; a < p.atoms; ++a) tma::load_4d(sb + (m * p.atoms + a) * kWAtom, &p.mw, B_W, 64 * a, c0, m, blk);
    }
    __syncwarp();
    load(0);
    if (nt > 1) load(1);
    mbar_wait_bounded(B_W, 0, abort_flag, p.status, 1u << 18);
    const uint32_t idesc = make_idesc_bf16(128, TT, 0, 0);
    for (int t = 0; t < nt; ++t) {
      const int x = t & 1;
      mbar_wait_bounded(B_FULL + 8 * x, (t >> 1) & 1, abort_flag, p.status, 1u << 19);
      fence_after_sync();
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        for (int a = 0; a < p.atoms; ++a) {
          // a K step of 16 advances both start addresses by 32 bytes, 2 in descriptor units
          const uint64_t da = make_smem_desc_sw128(sb + (m * p.atoms + a) * kWAtom, 16, 1024);
          const uint64_t db = make_smem_desc_sw128(sb + SM_U + (x * p.atoms + a) * kUAtom, 16, 1024);
          const int ks = min(64, p.n - 64 * a) >> 4;
#pragma unroll
          for (int k = 0; k < 4; ++k)
            if (k < ks && leader) mma_ss(tmem_u + 128 * x + 64 * m, da + 2 * k, db + 2 * k, idesc, (a > 0 || k > 0) ? 1u : 0u);
        }
      }
      if (leader) mma_commit(B_D + 8 * x);
      __syncwarp();
      if (t >= 1 && t + 1 < nt) {   // tile t - 1 has been read: its stage takes tile t + 1
        mbar_wait_bounded(B_EMPTY + 8 * (x ^ 1), ((t - 1) >> 1) & 1, abort_flag, p.status, 1u << 20);
        load(t + 1);
      }
      __syncwarp();
    }
  } else if (warp == NC / 32 + 1) {
    if (lane == 0) {
      const int na = min(128, p.n - c0) > 64 ? 2 : 1;
      auto load_y = [&](int t) {
        tma::mbar_expect_tx(B_Y + 8 * (t & 1), (uint32_t)na * kUAtom);
        for (int a = 0; a < na; ++a)
          tma::load_4d(sb + SM_Y + ((t & 1) * 2 + a) * kUAtom, &p.my, B_Y + 8 * (t & 1), c0 + 64 * a, t * TT, blk, b);
      };
      load_y(0);
      if (nt > 1) load_y(1);
      for (int t = 0; t < nt; ++t) {
        mbar_wait_bounded<false>(B_OUT + 8 * (t & 1), (t >> 1) & 1, abort_flag, p.status, 1u << 23);
        for (int a = 0; a < na; ++a) tma::store_4d(&p.mo, sb + SM_Y + ((t & 1) * 2 + a) * kUAtom, c0 + 64 * a, t * TT, blk, b);
        bulk_commit();
        bulk_wait_read_all();
        if (t + 2 < nt) load_y(t + 2);
      }
      bulk_wait_all();
    }
  } else {
    const int grp = warp >> 2, ch = tid & 127;
    const bool live = c0 + ch < p.n;
    const int chan = blk * p.n + c0 + (live ? ch : 0);
    const uint32_t tlane = tmem + ((uint32_t)((warp & 3) * 32) << 16);
    const int t0g = grp * TG;
    const float rb = -kLog2e * __bfloat162float(p.rb[chan]), ib = -kLog2e * __bfloat162float(p.ib[chan]);
    const float decay2 = -8.0f * seq::softplus_acc(p.lam[chan]) * kLog2e;   // log2 a = decay2 * r
    float* carry = reinterpret_cast<float*>(smem + SM_C);
    const uint32_t my_carry = B_CARRY + 8 * grp, from = B_CARRY + 8 * ((grp + GROUPS - 1) % GROUPS);
    const float* carry_in = carry + ((grp + GROUPS - 1) % GROUPS) * 128 + ch;
    uint8_t* ycol = smem + SM_Y + (ch >> 6) * kUAtom + (ch & 7) * 2;
    const int ychunk = (ch & 63) >> 3;
    const uint8_t* ucol = smem + SM_U + ((c0 + ch) >> 6) * kUAtom + (ch & 7) * 2;   // this channel's column of a stage
    const int chunk = ((c0 + ch) & 63) >> 3;
    float S0 = 0.f;
    if (grp == 0 && live && seq::position0(p.offsets, p.offset, b) > 0) S0 = p.state[(int64_t)b * p.W + chan];
    for (int t = 0; t < nt; ++t) {
      const int x = t & 1, tok0 = t * TT + t0g;
      mbar_wait_bounded(B_D + 8 * x, (t >> 1) & 1, abort_flag, p.status, 1u << 21);
      fence_after_sync();
      uint32_t gr[TG], gi[TG];
      tmem_ld16(tlane + 128 * x + t0g, gr);
      tmem_ld16(tlane + 128 * x + 64 + t0g, gi);
      tmem_ld_wait();
      const uint8_t* us = ucol + x * p.atoms * kUAtom;
      float P[TG], s[TG];   // product of the decays and state from zero, up to each token
      float pr = 1.f, sr = 0.f;
#pragma unroll
      for (int i = 0; i < TG; ++i) {
        const float u = live ? __bfloat162float(*reinterpret_cast<const bf16*>(us + (t0g + i) * 128 + ((chunk ^ (i & 7)) << 4))) : 0.f;
        const float er = 1.f + ex2(fminf(fmaf(__uint_as_float(gr[i]), -kLog2e, rb), 60.f));
        const float ei = 1.f + ex2(fminf(fmaf(__uint_as_float(gi[i]), -kLog2e, ib), 60.f));
        const float q = rcp(er * ei);                       // both sigmoids from one reciprocal
        const float l2 = decay2 * (q * ei), a = ex2(l2);
        // 1 - a^2 = -expm1(z), z = 2 log a: by its series near zero, where the difference cancels
        const float z = l2 * (2.f / kLog2e);
        float om = fmaf(z, 1.f / 720.f, 1.f / 120.f);
        om = fmaf(z, om, 1.f / 24.f);
        om = fmaf(z, om, 1.f / 6.f);
        om = fmaf(z, om, 0.5f);
        om = -fmaf(z * z, om, z);
        om = z > -0.25f ? om : fmaf(-a, a, 1.f);
        float in = sqrt_approx(om) * (q * er) * u, aa = a;
        if (tok0 + i >= p.L) { in = 0.f; aa = 1.f; }        // past the end nothing happens
        sr = fmaf(aa, sr, in);
        pr *= aa;
        P[i] = pr;
        s[i] = sr;
      }
      fence_before_sync();
      mbar_arrive(B_EMPTY + 8 * x);                          // gates and u of this tile have been read
      if (grp > 0 || t > 0) {
        mbar_wait_bounded(from, (grp > 0 ? t : t - 1) & 1, abort_flag, p.status, 1u << 22);
        S0 = *carry_in;
      }
      const float end = fmaf(pr, S0, sr);
      carry[grp * 128 + ch] = end;
      mbar_arrive(my_carry);
      mbar_wait_bounded(B_Y + 8 * x, (t >> 1) & 1, abort_flag, p.status, 1u << 24);
      uint8_t* ys = ycol + x * 2 * kUAtom;
      auto at = [&](int i) { return reinterpret_cast<bf16*>(ys + (t0g + i) * 128 + ((ychunk ^ (i & 7)) << 4)); };   // t0g is a multiple of 8
      bf16 yv[TG];   // all read before the first is replaced
#pragma unroll
      for (int i = 0; i < TG; ++i) yv[i] = *at(i);
#pragma unroll
      for (int i = 0; i < TG; ++i)     // rows past the sequence and channels past the block are clipped by the store
        *at(i) = __float2bfloat16_rn(fmaf(P[i], S0, s[i]) * seq::gelu_tanh_t<bf16>(__bfloat162float(yv[i])));
      fence_proxy_async();
      mbar_arrive(B_OUT + 8 * x);
      if (live && grp == GROUPS - 1 && t == nt - 1) p.state[(int64_t)b * p.W + chan] = end;
    }
  }
  __syncwarp();
  fence_before_sync();
  __syncthreads();
  if (warp == NC / 32) {
    fence_after_sync();
    tmem_dealloc(tmem, 256);
  }
}

}  // namespace

int read_tc_status_rglru(unsigned int* out, int reset) {
  unsigned int v = 0;
  cudaError_t e = cudaMemcpyFromSymbol(&v, g_tc_status_rglru, sizeof(v));
  if (e != cudaSuccess) return (int)e;
  if (out) *out = v;
  if (reset && v != 0) {
    v = 0;
    e = cudaMemcpyToSymbol(g_tc_status_rglru, &v, sizeof(v));
  }
  return (int)e;
}

// w [blocks, 2, n, n]: r and i matrices, [out, in].  BASED_ERR_IMPL: sizes or alignment this kernel does not take.
int launch_rglru_tc(const void* u, const void* y, const void* w, const void* rb, const void* ib, const float* lam,
                    float* state, void* out, int B, int L, int W, int n, Strides2 su, Strides2 sy, Strides2 so,
                    const int32_t* offsets, int offset, cudaStream_t stream) {
  if (n % 16 != 0 || n > 256 || W % 8 != 0 || B > 65535) return BASED_ERR_IMPL;
  if (!aligned16(u) || !aligned16(w) || su.h % 8 != 0 || (B > 1 && su.b % 8 != 0) || su.h <= 0) return BASED_ERR_IMPL;
  Params p;
  const int blocks = W / n;
  p.slices = (n + 127) / 128;
  p.atoms = (n + 63) / 64;
  static tma::MapCache cache;
  auto get_map = [&](CUtensorMap* m, const void* base, uint64_t d0, uint64_t d1, uint64_t d2, uint64_t d3, int64_t s1, int64_t s2,
                     int64_t s3, int rows) -> int {
    const tma::MapKey key = tma::make_key(base, d0, d1, d2, d3, 0, s1, s2, s3, 0, 64, (uint32_t)rows, 0, 4);
    if (cache.find(key, m)) return 0;
    if (tma::encode_bf16_4d_sw128(m, base, d0, d1, d2, d3, s1, s2, s3, 64, (uint32_t)rows)) return 1;
    cache.put(key, *m);
    return 0;
  };
  for (const Strides2& st : {sy, so})
    if (st.h % 8 != 0 || st.h <= 0 || (B > 1 && (st.b % 8 != 0 || st.b <= 0))) return BASED_ERR_IMPL;
  if (!aligned16(y) || !aligned16(out)) return BASED_ERR_IMPL;
  const int64_t nn = (int64_t)n * n;
  if (get_map(&p.mw, w, n, n, 2, blocks, n, nn, 2 * nn, 128) ||
      get_map(&p.mu, u, W, L, 1, B, L == 1 ? 8 : su.h, 8, B == 1 ? 8 : su.b, TT) ||
      get_map(&p.my, y, n, L, blocks, B, L == 1 ? 8 : sy.h, n, B == 1 ? 8 : sy.b, TT) ||
      get_map(&p.mo, out, n, L, blocks, B, L == 1 ? 8 : so.h, n, B == 1 ? 8 : so.b, TT))
    return BASED_ERR_IMPL;
  p.rb = static_cast<const bf16*>(rb);
  p.ib = static_cast<const bf16*>(ib);
  p.lam = lam; p.state = state;
  p.offsets = offsets; p.offset = offset; p.L = L; p.W = W; p.n = n;
  const int smem = 2 * p.atoms * (int)(kWAtom + kUAtom) + 4 * (int)kUAtom + GROUPS * 128 * 4 + 8 * (11 + GROUPS) + 16;
  if (smem > 227 * 1024) return BASED_ERR_IMPL;
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
      e = cudaGetSymbolAddress(reinterpret_cast<void**>(&addr), g_tc_status_rglru);
      if (e != cudaSuccess) return (int)e;
      e = cudaFuncSetAttribute(rglru_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
      if (e != cudaSuccess) return (int)e;
      status[dev] = addr;
    }
    p.status = status[dev];
  }
  rglru_tc_kernel<<<dim3(blocks * p.slices, B), NT, smem, stream>>>(p);
  return (int)cudaGetLastError();
}

}  // namespace based
