// Causal softmax attention of the expanded latent-attention form on the sm_100a tensor cores, bf16 operands, fp32
// scores, softmax and accumulation:
//   s[i, t] = (q1_i . k1_t + q2_i . k2_t) * scale   (k1 per head, k2 shared by all heads), t <= offset + i
//   out_i   = sigmoid(gate_i) * sum_t softmax(s)[i, t] v_t
// One CTA owns 256 queries of one (batch, head) as two tiles of 128 rows that take turns on the tensor pipe:
//   warps 0-3 / 4-7   softmax of tile 0 / 1, one query row per thread: S (TMEM) -> P (bf16, in S's columns)
//   warp 8            TMA producer
//   warp 9            MMA issue: S_x(j+1) = Q_x K(j+1)^T right behind O_x += P_x(j) V(j), so that one tile's softmax
//                     runs under the other tile's products
// The shared-memory ring holds 16 KB atoms (128 rows x 64 columns, 128-byte swizzle).  A K tile takes one atom per 64
// key dimensions (the shared part has atoms of its own), a V tile one per 64 value columns; units are loaded in the
// order K0 V0 K1 V1 .. and released in the same order, so whatever fits in shared memory is prefetch depth.
// The accumulator is rescaled only when a row's maximum grew by more than 2^8 since the last rescale; the reader of
// S(j) may touch O because S(j) was issued behind P V (j-1) and its commit covers both.
#include <initializer_list>
#include <mutex>

#include "seq_common.cuh"
#include "tcgen05.cuh"
#include "tma.cuh"

namespace based {

__device__ unsigned int g_tc_status_latent = 0;

namespace {

using namespace tc;

constexpr int TQ = 128, TK = 128;
constexpr int NT = 320;
constexpr uint32_t kAtom = 128 * 128;  // bytes
constexpr int kUnits = 4;              // outstanding K (and V) tiles
constexpr float kRescale = 8.0f;       // log2 units

struct Params {
  CUtensorMap mq1, mq2, mk1, mk2, mv;
  const __nv_bfloat16* gate;
  __nv_bfloat16* out;
  int64_t gb, gl, ob, ol, oh;
  const int32_t* offsets;
  int offset, L, d1, d2, dv, a1, a2, av, ring, tmem_cols;
  float scale_log2e;
  unsigned int* status;
};

// the ring allocator both the producer and the MMA warp step through, in the same order
struct Ring {
  int at = 0;
  // first slot of a unit of n atoms; `contiguous` units never wrap (pad counts the skipped slots)
  __device__ __forceinline__ int place(int n, bool contiguous, int size, int& pad) {
    pad = 0;
    if (contiguous && at + n > size) { pad = size - at; at = 0; }
    const int s = at;
    at += n;
    if (at >= size) at -= size;
    return s;
  }
};

__global__ void __launch_bounds__(NT, 1) latent_prefill_tc_kernel(const __grid_constant__ Params p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
  const uint32_t sb = smem_u32(smem);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.y, b = blockIdx.z;
  const int q0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * (2 * TQ);   // longest rows first
  const int off = seq::position0(p.offsets, p.offset, b);
  const int na = p.a1 + p.a2;
  const uint32_t SM_RING = 2u * na * kAtom, SM_BAR = SM_RING + (uint32_t)p.ring * kAtom;
  const uint32_t bar = sb + SM_BAR;
  // barriers: q, k_full[4], k_empty[4], v_full[4], v_empty[4], s_full[2], p_full[2], o_full[2]
  const uint32_t B_Q = bar, B_KF = bar + 8, B_KE = B_KF + 8 * kUnits, B_VF = B_KE + 8 * kUnits, B_VE = B_VF + 8 * kUnits,
                 B_S = B_VE + 8 * kUnits, B_P = B_S + 16, B_O = B_P + 16;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem + SM_BAR + 8 * (1 + 4 * kUnits + 6));
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  // keys tile x's last row sees, in tiles (a tile with no valid row at all is skipped)
  int ntile[2];
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    const int rows = min(TQ, p.L - q0 - x * TQ);
    ntile[x] = rows > 0 ? (off + q0 + x * TQ + rows - 1) / TK + 1 : 0;
  }
  const int nkv = max(ntile[0], ntile[1]);

  if (tid == 0) {
    mbar_init(B_Q, 1);
    for (int i = 0; i < kUnits; ++i) {
      mbar_init(B_KF + 8 * i, 1); mbar_init(B_KE + 8 * i, 1); mbar_init(B_VF + 8 * i, 1); mbar_init(B_VE + 8 * i, 1);
    }
    for (int x = 0; x < 2; ++x) { mbar_init(B_S + 8 * x, 1); mbar_init(B_P + 8 * x, TQ); mbar_init(B_O + 8 * x, 1); }
    *abort_flag = 0;
    fence_mbar_init();
    fence_proxy_async();
  }
  if (warp == 9) tmem_alloc(smem_u32(tmem_slot), p.tmem_cols);
  fence_before_sync();
  __syncthreads();
  fence_after_sync();
  const uint32_t tmem = *tmem_slot;
  const uint32_t TM_S[2] = {0u, 128u}, TM_O[2] = {256u, 256u + (uint32_t)((p.dv + 31) & ~31)};

  if (warp == 8) {
    // ---------------- producer
    if (lane == 0) {
      const int nx = ntile[1] > 0 ? 2 : 1;
      tma::mbar_expect_tx(B_Q, (uint32_t)(nx * na) * kAtom);
      for (int x = 0; x < nx; ++x) {
        for (int a = 0; a < p.a1; ++a) tma::load_4d(sb + (x * na + a) * kAtom, &p.mq1, B_Q, 64 * a, q0 + x * TQ, h, b);
        for (int a = 0; a < p.a2; ++a) tma::load_4d(sb + (x * na + p.a1 + a) * kAtom, &p.mq2, B_Q, 64 * a, q0 + x * TQ, h, b);
      }
      Ring ring;
      int used = 0, oldest = 0;            // units are numbered 2j (K of tile j), 2j + 1 (V of tile j)
      int pads[2 * kUnits];                // slots each outstanding unit holds
      for (int u = 0; u < 2 * nkv; ++u) {
        const bool is_v = u & 1;
        const int j = u >> 1, n = is_v ? p.av : na;
        int pad;
        const int slot = ring.place(n, is_v, p.ring, pad);
        while (used + n + pad > p.ring || u - oldest >= 2 * kUnits) {
          const int jo = oldest >> 1;
          mbar_wait_bounded<false>(((oldest & 1) ? B_VE : B_KE) + 8 * (jo % kUnits), (jo / kUnits) & 1, abort_flag, p.status, 1u << 8);
          used -= pads[oldest % (2 * kUnits)];
          ++oldest;
        }
        used += n + pad;
        pads[u % (2 * kUnits)] = n + pad;
        const uint32_t full = (is_v ? B_VF : B_KF) + 8 * (j % kUnits);
        tma::mbar_expect_tx(full, (uint32_t)n * kAtom);
        for (int a = 0; a < n; ++a) {
          int s = slot + a;
          if (s >= p.ring) s -= p.ring;
          const uint32_t dst = sb + SM_RING + s * kAtom;
          if (is_v) tma::load_4d(dst, &p.mv, full, 64 * a, j * TK, h, b);
          else if (a < p.a1) tma::load_4d(dst, &p.mk1, full, 64 * a, j * TK, h, b);
          else tma::load_4d(dst, &p.mk2, full, 64 * (a - p.a1), j * TK, 0, b);
        }
      }
    }
  } else if (warp == 9) {
    // ---------------- MMA issue (converged warp, one elected lane)
    const uint32_t tmem_u = __shfl_sync(0xffffffffu, tmem, 0);
    const bool leader = elect_one_sync();
    const uint32_t idesc_s = make_idesc_bf16(128, TK, 0, 0), idesc_o = make_idesc_bf16(128, p.dv, 0, 1);
    Ring ring;
    int kslot[2] = {0, 0}, vslot[2] = {0, 0};  // by parity of the tile
    auto issue_s = [&](int x, int j) {
      uint32_t acc = 0;
      for (int a = 0; a < na; ++a) {
        int s = kslot[j & 1] + a;
        if (s >= p.ring) s -= p.ring;
        const uint32_t qa = sb + (x * na + a) * kAtom, ka = sb + SM_RING + s * kAtom;
        const int left = a < p.a1 ? p.d1 - 64 * a : p.d2 - 64 * (a - p.a1);
        const int ks = min(64, left) >> 4;
        for (int k = 0; k < ks; ++k) {
          const uint64_t da = make_smem_desc_sw128(qa + k * 32, 16, 1024), db = make_smem_desc_sw128(ka + k * 32, 16, 1024);
          if (leader) mma_ss(tmem_u + TM_S[x], da, db, idesc_s, acc);
          acc = 1;
        }
      }
      if (leader) mma_commit(B_S + 8 * x);
    };
    auto issue_pv = [&](int x, int j) {
      const uint32_t va = sb + SM_RING + vslot[j & 1] * kAtom;
#pragma unroll
      for (int k = 0; k < TK / 16; ++k) {
        const uint64_t dvd = make_smem_desc_sw128(va + k * 2048, kAtom, 1024);
        if (leader) mma_ts(tmem_u + TM_O[x], tmem_u + TM_S[x] + 8 * k, dvd, idesc_o, (j > 0 || k > 0) ? 1u : 0u);
      }
    };
    int pad;
    mbar_wait_bounded(B_Q, 0, abort_flag, p.status, 1u << 9);
    for (int j = -1; j < nkv; ++j) {
      // K(j+1) and V(j) are units in this order: V(j) was placed before K(j+1)
      if (j >= 0) {
        vslot[j & 1] = ring.place(p.av, true, p.ring, pad);
        mbar_wait_bounded(B_VF + 8 * (j % kUnits), (j / kUnits) & 1, abort_flag, p.status, 1u << 10);
      }
      const bool more = j + 1 < nkv;
      if (more) kslot[(j + 1) & 1] = ring.place(na, false, p.ring, pad);
      bool k_ready = false;
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        if (j >= 0 && j < ntile[x]) {
          mbar_wait_bounded(B_P + 8 * x, j & 1, abort_flag, p.status, 1u << 11);
          fence_after_sync();
          issue_pv(x, j);
          if (j == ntile[x] - 1 && leader) mma_commit(B_O + 8 * x);
        }
        if (more && j + 1 < ntile[x]) {
          if (!k_ready) {
            mbar_wait_bounded(B_KF + 8 * ((j + 1) % kUnits), ((j + 1) / kUnits) & 1, abort_flag, p.status, 1u << 12);
            fence_after_sync();
            k_ready = true;
          }
          issue_s(x, j + 1);
        }
      }
      // everything that reads V(j) and K(j+1) has been issued
      if (j >= 0 && leader) mma_commit(B_VE + 8 * (j % kUnits));
      if (more && leader) mma_commit(B_KE + 8 * ((j + 1) % kUnits));
      __syncwarp();
    }
  } else {
    // ---------------- softmax: one query row per thread
    const int x = warp >> 2, row = tid & 127;
    const int n = x == 0 ? ntile[0] : ntile[1];
    const uint32_t tlane = tmem + ((uint32_t)((warp & 3) * 32) << 16);
    const uint32_t ts = tlane + (x == 0 ? TM_S[0] : TM_S[1]), to = tlane + (x == 0 ? TM_O[0] : TM_O[1]);
    const uint32_t bs = B_S + 8 * x, bp = B_P + 8 * x;
    const int qi = q0 + x * TQ + row;           // index of this row's query in the call
    const int last = off + qi;                  // last key it sees
    float m = -INFINITY, sum = 0.f;             // m: the maximum the exponentials are taken against (scaled, log2)
    for (int j = 0; j < n; ++j) {
      mbar_wait_bounded(bs, j & 1, abort_flag, p.status, 1u << 13);
      fence_after_sync();
      uint32_t r[4][32];
#pragma unroll
      for (int c = 0; c < 4; ++c) tmem_ld32(ts + 32 * c, r[c]);
      tmem_ld_wait();
      const int lim = last - j * TK;            // columns 0..lim are visible
      if (__any_sync(0xffffffffu, lim < TK - 1)) {
#pragma unroll
        for (int c = 0; c < 4; ++c)
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (32 * c + i > lim) r[c][i] = 0xff800000u;  // -inf
      }
      float m4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int c = 0; c < 4; ++c)
#pragma unroll
        for (int i = 0; i < 32; ++i) m4[i & 3] = fmaxf(m4[i & 3], __uint_as_float(r[c][i]));
      const float mt = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3])) * p.scale_log2e;
      bool grow = mt > m + kRescale;
      if (j == 0) {
        m = mt;
      } else if (__any_sync(0xffffffffu, grow)) {
        const float mn = grow ? mt : m;
        const float corr = grow ? exp2f(m - mn) : 1.0f;
        m = mn;
        sum *= corr;
        for (int c = 0; c < p.dv; c += 16) {
          uint32_t o[16];
          tmem_ld16(to + c, o);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * corr);
          tmem_st16(to + c, o);
        }
        tmem_st_wait();
      }
      float s4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        uint32_t pk[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          float e0, e1;
          asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(e0) : "f"(fmaf(__uint_as_float(r[c][2 * i]), p.scale_log2e, -m)));
          asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(e1) : "f"(fmaf(__uint_as_float(r[c][2 * i + 1]), p.scale_log2e, -m)));
          s4[i & 3] += e0 + e1;
          pk[i] = pack_bf16(e0, e1);
        }
        tmem_st16(ts + 16 * c, pk);
      }
      sum += (s4[0] + s4[1]) + (s4[2] + s4[3]);
      tmem_st_wait();
      fence_before_sync();
      mbar_arrive(bp);
    }
    if (n > 0) {
      mbar_wait_bounded(B_O + 8 * x, 0, abort_flag, p.status, 1u << 14);
      fence_after_sync();
      float f = 1.0f / sum;
      const bool live = qi < p.L;
      if (p.gate && live) f *= seq::sigmoid_acc(__bfloat162float(p.gate[b * p.gb + qi * p.gl + h]));
      __nv_bfloat16* o = p.out + b * p.ob + (int64_t)qi * p.ol + h * p.oh;
      for (int c = 0; c < p.dv; c += 16) {
        uint32_t t[16];
        tmem_ld16(to + c, t);
        tmem_ld_wait();
        if (live) {
          uint32_t w[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) w[i] = pack_bf16(__uint_as_float(t[2 * i]) * f, __uint_as_float(t[2 * i + 1]) * f);
          *reinterpret_cast<uint4*>(o + c) = make_uint4(w[0], w[1], w[2], w[3]);
          *reinterpret_cast<uint4*>(o + c + 8) = make_uint4(w[4], w[5], w[6], w[7]);
        }
      }
    }
  }
  __syncwarp();
  fence_before_sync();
  __syncthreads();
  if (warp == 9) {
    fence_after_sync();
    tmem_dealloc(tmem, p.tmem_cols);
  }
}

}  // namespace

int read_tc_status_latent(unsigned int* out, int reset) {
  unsigned int v = 0;
  cudaError_t e = cudaMemcpyFromSymbol(&v, g_tc_status_latent, sizeof(v));
  if (e != cudaSuccess) return (int)e;
  if (out) *out = v;
  if (reset && v != 0) {
    v = 0;
    e = cudaMemcpyToSymbol(g_tc_status_latent, &v, sizeof(v));
  }
  return (int)e;
}

// k2 is shared by all heads (its head stride is not used).  BASED_ERR_IMPL: sizes or strides this kernel does not take.
int launch_latent_prefill_tc(const void* q1, const void* q2, const void* k1, const void* k2, const void* v,
                             const void* gate, void* out, int B, int L, int T, int H, int d1, int d2, int dv, Strides3 sq1,
                             Strides3 sq2, Strides3 sk1, Strides3 sk2, Strides3 sv, Strides3 so, int64_t gb, int64_t gl,
                             const int32_t* offsets, int offset, float scale, cudaStream_t stream) {
  if (d1 % 16 || d2 % 16 || dv % 16 || d1 <= 0 || d2 <= 0 || dv > 128) return BASED_ERR_IMPL;
  if (scale <= 0.f) return BASED_ERR_IMPL;   // the row maximum is taken before scaling
  if (!aligned16(q1) || !aligned16(q2) || !aligned16(k1) || !aligned16(k2) || !aligned16(v) || !aligned16(out)) return BASED_ERR_IMPL;
  auto fix = [&](int64_t s, int extent) { return extent == 1 ? (int64_t)8 : s; };
  const int64_t all[] = {fix(sq1.b, B), fix(sq1.h, H), fix(sq1.l, L), fix(sq2.b, B), fix(sq2.h, H), fix(sq2.l, L),
                         fix(sk1.b, B), fix(sk1.h, H), fix(sk1.l, T), fix(sk2.b, B), fix(sk2.l, T), fix(sv.b, B),
                         fix(sv.h, H), fix(sv.l, T), fix(so.b, B), fix(so.h, H), fix(so.l, L)};
  for (int64_t s : all)
    if (s % 8 != 0 || s <= 0) return BASED_ERR_IMPL;
  if (B > 65535 || H > 65535) return BASED_ERR_IMPL;
  Params p;
  p.a1 = (d1 + 63) / 64; p.a2 = (d2 + 63) / 64; p.av = (dv + 63) / 64;
  const int na = p.a1 + p.a2;
  constexpr int kMaxSmem = 227 * 1024, kFixed = 1024 + 512;
  p.ring = (kMaxSmem - kFixed - 2 * na * (int)kAtom) / (int)kAtom;
  // K(j+1) and V(j) are needed together, and a V tile may skip a slot
  if (p.ring < na + 2 * p.av) return BASED_ERR_IMPL;
  if (p.ring > 2 * (na + p.av) + p.av) p.ring = 2 * (na + p.av) + p.av;
  const int ocols = (dv + 31) & ~31;
  p.tmem_cols = 512;
  if (256 + 2 * ocols > 512) return BASED_ERR_IMPL;
  static tma::MapCache cache;
  auto get_map = [&](CUtensorMap* m, const void* base, int cols, int rows, int heads, Strides3 s) -> int {
    const tma::MapKey key = tma::make_key(base, cols, rows, heads, B, 0, fix(s.l, rows), fix(s.h, heads), fix(s.b, B), 0, 64, 128, 0, 4);
    if (cache.find(key, m)) return 0;
    if (tma::encode_bf16_4d_sw128(m, base, cols, rows, heads, B, fix(s.l, rows), fix(s.h, heads), fix(s.b, B), 64, 128)) return 1;
    cache.put(key, *m);
    return 0;
  };
  if (get_map(&p.mq1, q1, d1, L, H, sq1) || get_map(&p.mq2, q2, d2, L, H, sq2) || get_map(&p.mk1, k1, d1, T, H, sk1) ||
      get_map(&p.mk2, k2, d2, T, 1, sk2) || get_map(&p.mv, v, dv, T, H, sv))
    return BASED_ERR_IMPL;
  p.gate = static_cast<const __nv_bfloat16*>(gate);
  p.out = static_cast<__nv_bfloat16*>(out);
  p.gb = gb; p.gl = gl; p.ob = so.b; p.ol = so.l; p.oh = so.h;
  p.offsets = offsets; p.offset = offset; p.L = L; p.d1 = d1; p.d2 = d2; p.dv = dv;
  p.scale_log2e = scale * 1.4426950408889634f;
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
      e = cudaGetSymbolAddress(reinterpret_cast<void**>(&addr), g_tc_status_latent);
      if (e != cudaSuccess) return (int)e;
      e = cudaFuncSetAttribute(latent_prefill_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxSmem);
      if (e != cudaSuccess) return (int)e;
      status[dev] = addr;
    }
    p.status = status[dev];
  }
  const int smem = 2 * na * (int)kAtom + p.ring * (int)kAtom + kFixed;
  latent_prefill_tc_kernel<<<dim3((L + 2 * TQ - 1) / (2 * TQ), H, B), NT, smem, stream>>>(p);
  return (int)cudaGetLastError();
}

}  // namespace based
