// Causal softmax attention over a cache whose rows are keys and values at once, for prompts and long portions, on the
// sm_100a tensor cores: bf16 operands, fp32 scores, softmax and accumulation.
//   s[i, t] = (q_i . k_t) factor_t scale, t <= offset + i;   out_i = sum_t exp(s) k_t / (sink + sum_t exp(s)) * sigmoid(gate_i)
// One CTA owns 256 queries of one (batch, head) as two tiles of 128 rows that take turns on the tensor pipe:
//   warps 0-3 / 4-7   softmax of tile 0 / 1, one query row per thread: S (TMEM) -> P (bf16, in S's columns)
//   warp 8            TMA producer
//   warp 9            MMA issue: S_x(j+1) = Q_x K(j+1)^T right behind O_x += P_x(j) K(j), so that one tile's softmax runs
//                     under the other tile's products; P is handed over in two halves
// A tile of 128 keys is loaded once (64-column atoms, 128-byte swizzle) and is the K-major operand of S and the MN-major
// operand of O; its 128 factors come with it by an untiled bulk copy.  The accumulator is rescaled only when a row's
// maximum grew by more than 2^8 since the last rescale; the reader of S(j) may touch O because S(j) was issued behind
// P K (j-1) and its commit covers both.  A tile's Q is free when its last S has been computed: the gate tile is loaded into
// its place by TMA under the last softmax, replaced by the output, and stored from there by TMA (a thread owns a row, and
// rows are far apart in memory).
#include <initializer_list>
#include <mutex>

#include "seq_common.cuh"
#include "tcgen05.cuh"
#include "tma.cuh"

namespace based {

__device__ unsigned int g_tc_status_tied = 0;

namespace {

using namespace tc;

constexpr int TQ = 128, TK = 128;
constexpr int NT = 384;                // two softmax warpgroups; producer, MMA and two idle warps
// registers per thread: 168 at launch, 3 * 168 = 2 * 232 + 40 after the split
constexpr int kSoftmaxRegs = 232, kOtherRegs = 40;
constexpr uint32_t kAtom = 128 * 128;  // bytes
constexpr int kMaxStages = 6;
constexpr float kRescale = 8.0f;       // log2 units

struct Params {
  CUtensorMap mq, mk, mg, mo;    // q, gate and out [B][H][L][d], cache [B][G][T][d]
  const float* factor;
  int64_t fb, fh;
  int offset, L, group, d, atoms, stages, gated;
  float scale_log2e, sink;
  unsigned int* status;
};

__device__ __forceinline__ void bulk_load(uint32_t dst, const void* src, uint32_t bytes, uint32_t mbar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];\n" ::"r"(dst), "l"(src),
               "r"(bytes), "r"(mbar)
               : "memory");
}
__device__ __forceinline__ float ex2(float x) { float r; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x)); return r; }
__device__ __forceinline__ void mul2(uint32_t& a, uint32_t& b, float fa, float fb) {   // (a, b) *= (fa, fb) in one instruction
  asm("{\n\t.reg .b64 x, y;\n\tmov.b64 x, {%0, %1};\n\tmov.b64 y, {%2, %3};\n\tmul.rn.f32x2 x, x, y;\n\tmov.b64 {%0, %1}, x;\n\t}\n"
      : "+r"(a), "+r"(b) : "f"(fa), "f"(fb));
}

__device__ __forceinline__ uint64_t pair(float lo, float hi) { uint64_t r; asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi)); return r; }
__device__ __forceinline__ void split(uint64_t v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ uint64_t add2(uint64_t a, uint64_t b) { uint64_t r; asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b)); return r; }
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) { uint64_t r; asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c)); return r; }
__device__ __forceinline__ float max3(float a, float b, float c) { float r; asm("max.f32 %0, %1, %2, %3;" : "=f"(r) : "f"(a), "f"(b), "f"(c)); return r; }

__global__ void __launch_bounds__(NT, 1) tied_prefill_tc_kernel(const __grid_constant__ Params p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
  const uint32_t sb = smem_u32(smem);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.y, b = blockIdx.z, kh = h / p.group;
  const int q0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * (2 * TQ);   // longest rows first
  const int na = p.atoms;
  const uint32_t kTile = (uint32_t)na * kAtom;
  const uint32_t SM_K = 2u * kTile, SM_F = SM_K + (uint32_t)p.stages * kTile, SM_BAR = SM_F + (uint32_t)p.stages * TK * 4;
  // barriers: q, full[stages], empty[stages], s_full[2], p_full[2], o_full[2], gate[2], first half of P[2]
  const uint32_t B_Q = sb + SM_BAR, B_F = B_Q + 8, B_E = B_F + 8 * kMaxStages, B_S = B_E + 8 * kMaxStages, B_P = B_S + 16,
                 B_O = B_P + 16, B_G = B_O + 16, B_H = B_G + 16;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem + SM_BAR + 8 * (1 + 2 * kMaxStages + 10));
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  // keys tile x's last row sees, in tiles (a tile with no valid row at all is skipped)
  int ntile[2];
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    const int rows = min(TQ, p.L - q0 - x * TQ);
    ntile[x] = rows > 0 ? (p.offset + q0 + x * TQ + rows - 1) / TK + 1 : 0;
  }
  const int nkv = max(ntile[0], ntile[1]);

  if (tid == 0) {
    mbar_init(B_Q, 1);
    for (int i = 0; i < p.stages; ++i) { mbar_init(B_F + 8 * i, 1); mbar_init(B_E + 8 * i, 1); }
    for (int x = 0; x < 2; ++x) { mbar_init(B_S + 8 * x, 1); mbar_init(B_P + 8 * x, TQ); mbar_init(B_O + 8 * x, 1); mbar_init(B_G + 8 * x, 1); mbar_init(B_H + 8 * x, TQ); }
    *abort_flag = 0;
    fence_mbar_init();
    fence_proxy_async();
  }
  if (warp == 9) tmem_alloc(smem_u32(tmem_slot), 512);
  fence_before_sync();
  __syncthreads();
  fence_after_sync();
  const uint32_t tmem = *tmem_slot;
  const uint32_t TM_S[2] = {0u, 128u}, TM_O[2] = {256u, 384u};

  if (warp >= 8) {
    asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(kOtherRegs));
    if (warp == 8) {
    // ---------------- producer
    if (lane == 0) {
      const int nx = ntile[1] > 0 ? 2 : 1;
      tma::mbar_expect_tx(B_Q, (uint32_t)nx * kTile);
      for (int x = 0; x < nx; ++x)
        for (int a = 0; a < na; ++a) tma::load_4d(sb + x * kTile + a * kAtom, &p.mq, B_Q, 64 * a, q0 + x * TQ, h, b);
      const float* f = p.factor + b * p.fb + kh * p.fh;
      int st = 0, ph = 0;
      for (int j = 0; j < nkv; ++j) {
        if (j >= p.stages) mbar_wait_bounded<false>(B_E + 8 * st, ph ^ 1, abort_flag, p.status, 1u << 8);
        const uint32_t full = B_F + 8 * st;
        tma::mbar_expect_tx(full, kTile + TK * 4);
        for (int a = 0; a < na; ++a) tma::load_4d(sb + SM_K + st * kTile + a * kAtom, &p.mk, full, 64 * a, j * TK, kh, b);
        bulk_load(sb + SM_F + st * TK * 4, f + j * TK, TK * 4, full);
        if (++st == p.stages) { st = 0; ph ^= 1; }
      }
    }
    } else if (warp == 9) {
    // ---------------- MMA issue (converged warp, one elected lane)
    const uint32_t tmem_u = __shfl_sync(0xffffffffu, tmem, 0);
    const bool leader = elect_one_sync();
    const uint32_t idesc_s = make_idesc_bf16(128, TK, 0, 0), idesc_o = make_idesc_bf16(128, p.d, 0, 1);
    auto issue_s = [&](int x, int st) {
      for (int a = 0; a < na; ++a) {
        // a K step of 16 advances both start addresses by 32 bytes, 2 in descriptor units
        const uint64_t da = make_smem_desc_sw128(sb + x * kTile + a * kAtom, 16, 1024);
        const uint64_t db = make_smem_desc_sw128(sb + SM_K + st * kTile + a * kAtom, 16, 1024);
        const int ks = min(64, p.d - 64 * a) >> 4;
#pragma unroll
        for (int k = 0; k < 4; ++k)
          if (k < ks && leader) mma_ss(tmem_u + TM_S[x], da + 2 * k, db + 2 * k, idesc_s, (a > 0 || k > 0) ? 1u : 0u);
      }
      if (leader) mma_commit(B_S + 8 * x);
    };
    auto issue_o = [&](int x, int j, int st, int k0) {
      const uint64_t dv = make_smem_desc_sw128(sb + SM_K + st * kTile, kAtom, 1024);
#pragma unroll
      for (int kk = 0; kk < TK / 32; ++kk) {   // 16 keys are 2048 bytes
        const int k = k0 + kk;
        if (leader) mma_ts(tmem_u + TM_O[x], tmem_u + TM_S[x] + 8 * k, dv + 128 * k, idesc_o, (j > 0 || k > 0) ? 1u : 0u);
      }
    };
    mbar_wait_bounded(B_Q, 0, abort_flag, p.status, 1u << 9);
    int st = 0, next = 0, ph = 0;   // stages of tiles j and j + 1, phase of the latter
    for (int j = -1; j < nkv; ++j) {
      const bool more = j + 1 < nkv;
      if (more) {
        mbar_wait_bounded(B_F + 8 * next, ph, abort_flag, p.status, 1u << 10);
        fence_after_sync();
      }
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        if (j >= 0 && j < ntile[x]) {
          mbar_wait_bounded(B_H + 8 * x, j & 1, abort_flag, p.status, 1u << 16);
          fence_after_sync();
          issue_o(x, j, st, 0);
          mbar_wait_bounded(B_P + 8 * x, j & 1, abort_flag, p.status, 1u << 11);
          fence_after_sync();
          issue_o(x, j, st, 4);
          if (j == ntile[x] - 1 && leader) mma_commit(B_O + 8 * x);
        }
        if (more && j + 1 < ntile[x]) issue_s(x, next);
      }
      if (j >= 0 && leader) mma_commit(B_E + 8 * st);   // everything that reads tile j has been issued
      st = next;
      if (++next == p.stages) { next = 0; ph ^= 1; }
      __syncwarp();
    }
    }
  } else {
    asm volatile("setmaxnreg.inc.sync.aligned.u32 %0;" ::"n"(kSoftmaxRegs));
    // ---------------- softmax: one query row per thread
    const int x = warp >> 2, row = tid & 127;
    const int n = x == 0 ? ntile[0] : ntile[1];
    const uint32_t tlane = tmem + ((uint32_t)((warp & 3) * 32) << 16);
    const uint32_t ts = tlane + (x == 0 ? TM_S[0] : TM_S[1]), to = tlane + (x == 0 ? TM_O[0] : TM_O[1]);
    const uint32_t bs = B_S + 8 * x, bp = B_P + 8 * x;
    const int qi = q0 + x * TQ + row;           // index of this row's query in the call
    const int last = p.offset + qi;             // last key it sees
    float m = 0.f, sum = 0.f;                   // m: the maximum the exponentials are taken against (scaled, log2)
    int st = 0;
    for (int j = 0; j < n; ++j) {
      mbar_wait_bounded(bs, j & 1, abort_flag, p.status, 1u << 13);   // S(j) read tile j, so its factors have landed, too
      fence_after_sync();
      mbar_wait_bounded(B_F + 8 * st, (j / p.stages) & 1, abort_flag, p.status, 1u << 12);
      if (p.gated && j == n - 1 && row == 0) {
        tma::mbar_expect_tx(B_G + 8 * x, kTile);
        for (int a = 0; a < na; ++a) tma::load_4d(sb + x * kTile + a * kAtom, &p.mg, B_G + 8 * x, 64 * a, q0 + x * TQ, h, b);
      }
      __syncwarp();
      uint32_t r[4][32];
#pragma unroll
      for (int c = 0; c < 4; ++c) tmem_ld32(ts + 32 * c, r[c]);
      const float4* f4 = reinterpret_cast<const float4*>(smem + SM_F + st * TK * 4);
      if (++st == p.stages) st = 0;
      tmem_ld_wait();
      float m4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int c = 0; c < 4; ++c)
#pragma unroll
        for (int i = 0; i < 32; i += 4) {
          const float4 f = f4[8 * c + (i >> 2)];
          mul2(r[c][i], r[c][i + 1], f.x, f.y);
          mul2(r[c][i + 2], r[c][i + 3], f.z, f.w);
        }
      const int lim = last - j * TK;            // columns 0..lim are visible
      if (__any_sync(0xffffffffu, lim < TK - 1)) {
#pragma unroll
        for (int c = 0; c < 4; ++c)
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (32 * c + i > lim) r[c][i] = 0xff800000u;  // -inf
      }
#pragma unroll
      for (int c = 0; c < 4; ++c)
#pragma unroll
        for (int i = 0; i < 32; i += 2) m4[(i >> 1) & 3] = max3(m4[(i >> 1) & 3], __uint_as_float(r[c][i]), __uint_as_float(r[c][i + 1]));
      const float mt = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3])) * p.scale_log2e;
      const bool grow = mt > m + kRescale;
      if (j == 0) {                             // the sink is one more score of 0
        m = p.sink > 0.f ? fmaxf(mt, 0.f) : mt;
        sum = p.sink > 0.f ? p.sink * exp2f(-m) : 0.f;
      } else if (__any_sync(0xffffffffu, grow)) {
        const float mn = grow ? mt : m;
        const float corr = grow ? exp2f(m - mn) : 1.0f;
        m = mn;
        sum *= corr;
        for (int c = 0; c < p.d; c += 16) {
          uint32_t o[16];
          tmem_ld16(to + c, o);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * corr);
          tmem_st16(to + c, o);
        }
        tmem_st_wait();
      }
      uint64_t s2[4] = {0ull, 0ull, 0ull, 0ull};
      const uint64_t sc2 = pair(p.scale_log2e, p.scale_log2e), nm2 = pair(-m, -m);
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        uint32_t pk[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          float e0, e1;
          split(fma2(pair(__uint_as_float(r[c][2 * i]), __uint_as_float(r[c][2 * i + 1])), sc2, nm2), e0, e1);
          e0 = ex2(e0);
          e1 = ex2(e1);
          s2[i & 3] = add2(s2[i & 3], pair(e0, e1));
          pk[i] = pack_bf16(e0, e1);
        }
        tmem_st16(ts + 16 * c, pk);
        if (c == 1) {                           // the products of keys 0-63 may start
          tmem_st_wait();
          fence_before_sync();
          mbar_arrive(B_H + 8 * x);
        }
      }
      float sl, sh;
      split(add2(add2(s2[0], s2[1]), add2(s2[2], s2[3])), sl, sh);
      sum += sl + sh;
      tmem_st_wait();
      fence_before_sync();
      mbar_arrive(bp);
    }
    if (n > 0) {
      mbar_wait_bounded(B_O + 8 * x, 0, abort_flag, p.status, 1u << 14);
      fence_after_sync();
      if (p.gated) mbar_wait_bounded(B_G + 8 * x, 0, abort_flag, p.status, 1u << 15);
      const float f = 1.0f / sum;
      uint8_t* tile = smem + x * kTile;
      for (int c = 0; c < p.d; c += 16) {
        uint32_t t[16];
        tmem_ld16(to + c, t);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 16; i += 8) {
          __nv_bfloat16* at = reinterpret_cast<__nv_bfloat16*>(tile + (c >> 6) * kAtom + tma::sw128_offset(row, ((c & 63) + i) >> 3));
          float y[8], z[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) y[e] = __uint_as_float(t[i + e]) * f;
          if (p.gated) {
            seq::Pack<__nv_bfloat16, 8>::load(at, z);
#pragma unroll
            for (int e = 0; e < 8; ++e) y[e] *= seq::sigmoid_t<__nv_bfloat16>(z[e]);
          }
          seq::Pack<__nv_bfloat16, 8>::store(at, y);
        }
      }
      fence_proxy_async();
      if (x == 0) asm volatile("bar.sync 1, 128;" ::: "memory");   // this tile's four warps
      else asm volatile("bar.sync 2, 128;" ::: "memory");
      if (row == 0) {                           // rows past the call's tokens are clipped
        for (int a = 0; a < na; ++a) tma::store_4d(&p.mo, sb + x * kTile + a * kAtom, 64 * a, q0 + x * TQ, h, b);
        bulk_commit();
        bulk_wait_all();
      }
    }
  }
  __syncwarp();
  fence_before_sync();
  __syncthreads();
  if (warp == 9) {
    fence_after_sync();
    tmem_dealloc(tmem, 512);
  }
}

}  // namespace

int read_tc_status_tied(unsigned int* out, int reset) {
  unsigned int v = 0;
  cudaError_t e = cudaMemcpyFromSymbol(&v, g_tc_status_tied, sizeof(v));
  if (e != cudaSuccess) return (int)e;
  if (out) *out = v;
  if (reset && v != 0) {
    v = 0;
    e = cudaMemcpyToSymbol(g_tc_status_tied, &v, sizeof(v));
  }
  return (int)e;
}

// factor rows are read up to the next multiple of 128 keys.  BASED_ERR_IMPL: sizes or strides this kernel does not take.
int launch_tied_prefill_tc(const void* q, const void* cache, const float* factor, const void* gate, void* out, int B, int L,
                           int H, int G, int d, int64_t qb, int64_t ql, int64_t cb, int64_t cl, int64_t fb, int64_t fh,
                           int64_t gb, int64_t gl, int64_t ob, int64_t ol, int offset, float scale, float sink,
                           cudaStream_t stream) {
  if (d % 16 || d > 128 || B > 65535 || H > 65535) return BASED_ERR_IMPL;
  if (scale <= 0.f) return BASED_ERR_IMPL;   // the row maximum is taken before scaling
  const int T = offset + L;
  if (!aligned16(q) || !aligned16(cache) || !aligned16(factor) || !aligned16(out) || (gate && !aligned16(gate))) return BASED_ERR_IMPL;
  auto fix = [&](int64_t s, int extent) { return extent == 1 ? (int64_t)8 : s; };
  for (int64_t s : {fix(qb, B), fix(ql, L), fix(cb, B), fix(cl, T), fix(ob, B), fix(ol, L)})
    if (s % 8 != 0 || s <= 0) return BASED_ERR_IMPL;
  if (gate && (fix(gb, B) % 8 || fix(gb, B) <= 0 || fix(gl, L) % 8 || fix(gl, L) <= 0)) return BASED_ERR_IMPL;
  if ((G > 1 && fh % 4) || (B > 1 && fb % 4) || fh < (int64_t)(T + TK - 1) / TK * TK) return BASED_ERR_IMPL;
  Params p;
  p.atoms = (d + 63) / 64;
  const int tile = p.atoms * (int)kAtom;
  constexpr int kMaxSmem = 227 * 1024, kFixed = 1024 + 256;
  p.stages = (kMaxSmem - kFixed - 2 * tile) / (tile + TK * 4);
  if (p.stages > kMaxStages) p.stages = kMaxStages;
  static tma::MapCache cache_;
  auto get_map = [&](CUtensorMap* m, const void* base, int rows, int heads, int64_t sl, int64_t sbt) -> int {
    const tma::MapKey key = tma::make_key(base, d, rows, heads, B, 0, fix(sl, rows), fix(d, heads), fix(sbt, B), 0, 64, 128, 0, 4);
    if (cache_.find(key, m)) return 0;
    if (tma::encode_bf16_4d_sw128(m, base, d, rows, heads, B, fix(sl, rows), fix(d, heads), fix(sbt, B), 64, 128)) return 1;
    cache_.put(key, *m);
    return 0;
  };
  if (get_map(&p.mq, q, L, H, ql, qb) || get_map(&p.mk, cache, T, G, cl, cb)) return BASED_ERR_IMPL;
  p.gated = gate != nullptr;
  if (get_map(&p.mo, out, L, H, ol, ob) || (p.gated && get_map(&p.mg, gate, L, H, gl, gb))) return BASED_ERR_IMPL;
  p.factor = factor;
  p.fb = fb; p.fh = fh;
  p.offset = offset; p.L = L; p.group = H / G; p.d = d;
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
      e = cudaGetSymbolAddress(reinterpret_cast<void**>(&addr), g_tc_status_tied);
      if (e != cudaSuccess) return (int)e;
      e = cudaFuncSetAttribute(tied_prefill_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxSmem);
      if (e != cudaSuccess) return (int)e;
      status[dev] = addr;
    }
    p.status = status[dev];
  }
  const int smem = 2 * tile + p.stages * (tile + TK * 4) + kFixed;
  tied_prefill_tc_kernel<<<dim3((L + 2 * TQ - 1) / (2 * TQ), H, B), NT, smem, stream>>>(p);
  return (int)cudaGetLastError();
}

}  // namespace based
