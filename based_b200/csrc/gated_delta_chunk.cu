// Gated delta rule over whole prompts and portions in chunks of 64 tokens, bf16 operands with fp32 results throughout
// the recurrence.  With G_i the running sum of log g inside a chunk and S0 the state before it (khat, qhat unit vectors):
//   u_i = beta_i (v_i - e^{G_i} S0^T khat_i) - sum_{j<i} A_ij u_j,   A_ij = beta_i e^{G_i - G_j} khat_i . khat_j
//   o_i = e^{G_i} S0^T qhat_i + sum_{j<=i} P_ij u_j,                 P_ij = e^{G_i - G_j} qhat_i . khat_j
//   S   = e^{G_C} S0 + sum_j e^{G_C - G_j} khat_j u_j^T
// Everything is separable over the value columns, so a warp owns 16 of them and keeps S^T [16, d] in registers for the
// whole sequence, as mma accumulators; an accumulator tile is also the A operand of the next product, so
// S^T -> (K S0)^T -> u^T -> S^T never leaves registers and warps meet only in the output norm.
//
// 32-bit without 32-bit operands: q and k enter as the bf16 values the convolution stored, their norms and all decays
// are fp32 factors applied to fp32 sums; in everything that enters the recurrence an fp32 matrix (S, u, A, T, the
// residual) is used as a bf16 pair hi + lo (16 mantissa bits), products of two pairs as hi hi + hi lo + lo hi.  The
// read-out S0^T q + P u, which nothing feeds back, multiplies bf16 operands once, like P V of an attention.
//
// The triangular system is solved by 16-token blocks: u_b = T_b (y_b - sum_{c<b} A_bc u_c) with T_b = (I + A_bb)^-1.
//
// One CTA per (head, batch, slice of the value columns), 16 warps:
//   warps 0-7   consumers (16 value columns each; surplus ones idle)
//   warps 8-15  helpers: load q, k, v of chunk c+2, take norms and gates, build A, P and T_b (mma.sync), and turn the
//               consumers' read-out of chunk c into the normed, gated output
// Two buffers; `ready` hands a prepared chunk to the consumers, `done` hands the read-out and the buffer back.
#include <initializer_list>
#include <mutex>
#include <type_traits>

#include "seq_common.cuh"
#include "tcgen05.cuh"

namespace based {

__device__ unsigned int g_tc_status_delta = 0;

namespace {

using namespace tc;
using bf16 = __nv_bfloat16;

constexpr int C = 64;               // tokens per chunk
constexpr int LT = C + 8;           // row stride of the [64, 64] operand tiles
constexpr int LI = 20;              // row stride of the diagonal blocks, stored transposed
constexpr int kConsumers = 8, kHelpers = 8;
constexpr int NT = 32 * (kConsumers + kHelpers), HT = 32 * kHelpers;
constexpr float kUnitEps = 1e-6f, kLog2e = 1.4426950408889634f;

struct Params {
  const bf16 *q, *k, *v, *z, *norm_w;
  const float *a, *b, *A_log, *dt_bias;
  float *state, *raw;               // raw [B, L, H, dv] fp32: read-out for a separate norm launch (slices), or null
  bf16* out;
  const int32_t* offsets;
  int offset, B, L, H, Hk, dv, vs;  // vs: value columns of this CTA's slice
  Strides2 sq, sk, sv, sz, sg, so;
  float eps;
  unsigned int* status;
};

struct Layout {                     // byte offsets in shared memory
  int ldk, ldv, K, Q, V, R, inv, gates, z, w, bars, total, tile_k, tile_v, region, ldo;
  __host__ __device__ Layout(int d, int vs) {
    ldk = d + 8; ldv = vs + 8; ldo = vs + 20;
    tile_k = C * ldk * 2; tile_v = C * ldv * 2;
    const int mats = 3 * C * LT * 2, stage = C * ldo * 4;
    region = mats > stage ? mats : stage;
    K = 0; Q = K + 2 * tile_k; V = Q + 2 * tile_k; R = V + 2 * tile_v;
    inv = R + 2 * region;
    gates = inv + 4 * 16 * LI * 4;
    z = gates + 3 * 9 * C * 4;
    w = z + HT * vs / 16 * 8;
    bars = w + ((vs * 4 + 15) & ~15);
    total = bars + 64;
  }
};
// gates of one chunk, C floats each (logarithms to base 2); chunk c's sit in slot c mod 3
enum { G_CUM = 0, G_BETA, G_RK, G_RQ, G_EGK, G_EGQ, G_W, G_COL, G_TOT, G_N };

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// x, y -> packed hi and lo halves: x = hi + lo to 16 mantissa bits
__device__ __forceinline__ void split(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(x, y);
  lo = pack_bf16(x - seq::bf16_lo(hi), y - seq::bf16_hi(hi));
}
// two adjacent 8-column accumulator tiles -> A operand of a 16-wide K step, hi and lo
__device__ __forceinline__ void split_a(const float (&t0)[4], const float (&t1)[4], uint32_t (&hi)[4], uint32_t (&lo)[4]) {
  split(t0[0], t0[1], hi[0], lo[0]);
  split(t0[2], t0[3], hi[1], lo[1]);
  split(t1[0], t1[1], hi[2], lo[2]);
  split(t1[2], t1[3], hi[3], lo[3]);
}
__device__ __forceinline__ float ex2(float x) { float r; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x)); return r; }
__device__ __forceinline__ void bar_sync(int id, int n) { asm volatile("bar.sync %0, %1;\n" ::"r"(id), "r"(n) : "memory"); }
template <int R> __device__ __forceinline__ void reg_inc() { asm volatile("setmaxnreg.inc.sync.aligned.u32 %0;\n" ::"n"(R)); }
template <int R> __device__ __forceinline__ void reg_dec() { asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;\n" ::"n"(R)); }

template <int DK>  // d = 16 DK
__global__ void __launch_bounds__(NT, 1) delta_chunk_kernel(const Params p) {
  constexpr int d = 16 * DK;
  extern __shared__ __align__(16) uint8_t sm[];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.x, b = blockIdx.y, v0 = blockIdx.z * p.vs;
  const int hk = h / (p.H / p.Hk);
  const Layout lay(d, p.vs);
  const uint32_t sb = smem_u32(sm);
  const uint32_t READY = sb + lay.bars, DONE = READY + 16;
  volatile int* abort_flag = reinterpret_cast<volatile int*>(sm + lay.bars + 32);
  const int nc = (p.L + C - 1) / C;
  const int active = (p.vs + 15) / 16;      // consumer warps with work
  if (tid == 0) {
    for (int i = 0; i < 2; ++i) { mbar_init(READY + 8 * i, HT); mbar_init(DONE + 8 * i, 32 * active); }
    *abort_flag = 0;
    fence_mbar_init();
  }
  __syncthreads();

  if (warp >= kConsumers) {
    // ------------------------------------------------------------ helpers
    reg_dec<80>();
    const int ht = tid - 32 * kConsumers, hw = warp - kConsumers;
    float* inv = reinterpret_cast<float*>(sm + lay.inv);
    const float A = expf(p.A_log[h]), dt = p.dt_bias[h];
    const int g = lane >> 2, t4 = lane & 3;

    const bf16 *kp = p.k + b * p.sk.b + (int64_t)hk * d, *qp = p.q + b * p.sq.b + (int64_t)hk * d,
               *vp = p.v + b * p.sv.b + (int64_t)h * p.dv + v0;
    auto gates_of = [&](int c) { return reinterpret_cast<float*>(sm + lay.gates) + (c % 3) * G_N * C; };
    // decays and step sizes of chunk c, two tokens per lane of one warp; tokens past the end neither decay nor write
    auto gates = [&](int c) {
      float* gt = gates_of(c);
      float lg[2] = {0.f, 0.f}, be[2] = {0.f, 0.f};
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int l = c * C + 2 * lane + e;
        if (l < p.L) {
          const int64_t gi = b * p.sg.b + (int64_t)l * p.sg.h + h;
          lg[e] = -A * kLog2e * seq::softplus_acc(p.a[gi] + dt);
          be[e] = seq::sigmoid_acc(p.b[gi]);
        }
      }
      float s = lg[0] + lg[1];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float t = __shfl_up_sync(0xffffffffu, s, o);
        if (lane >= o) s += t;
      }
      gt[G_CUM * C + 2 * lane] = s - lg[1];
      gt[G_CUM * C + 2 * lane + 1] = s;
      gt[G_BETA * C + 2 * lane] = be[0];
      gt[G_BETA * C + 2 * lane + 1] = be[1];
      if (lane == 31) gt[G_TOT * C] = s;
    };
    // q, k, v of chunk c into its buffer, and those of the chunk after it towards L2
    auto load = [&](int c) {
      const int buf = c & 1, base = c * C, n = min(C, p.L - base);
      const uint32_t kt = sb + lay.K + buf * lay.tile_k, qt = sb + lay.Q + buf * lay.tile_k, vt = sb + lay.V + buf * lay.tile_v;
      constexpr int RS = HT / (d / 8);   // rows per pass (HT is a multiple of d / 8 for d = 32, 64, 128; d = 96 leaves threads idle)
      const int r0 = ht / (d / 8), cc = ht % (d / 8);
      if (r0 < RS) {
        const bf16 *ks = kp + (int64_t)(base + r0) * p.sk.h + cc * 8, *qs = qp + (int64_t)(base + r0) * p.sq.h + cc * 8;
        uint32_t dst = r0 * lay.ldk * 2 + cc * 16;
#pragma unroll
        for (int i = r0; i < C; i += RS) {
          const bool ok = i < n;
          cp_async16(kt + dst, ok ? ks : kp, ok);
          cp_async16(qt + dst, ok ? qs : qp, ok);
          ks += RS * p.sk.h;
          qs += RS * p.sq.h;
          dst += RS * lay.ldk * 2;
        }
      }
      {
        const int i = ht >> 2;   // four threads per row
        const bool ok = i < n;
        const bf16* src = vp + (int64_t)(base + (ok ? i : 0)) * p.sv.h;
        for (int cc = ht & 3; cc < p.vs / 8; cc += 4) cp_async16(vt + i * lay.ldv * 2 + cc * 16, src + cc * 8, ok);
        const int64_t next = base + C + i;
        if (next < p.L) {
          for (int x = 32 * (ht & 3); x < d; x += 128) {   // 64-byte pieces
            asm volatile("prefetch.global.L2 [%0];" ::"l"(kp + next * p.sk.h + x));
            asm volatile("prefetch.global.L2 [%0];" ::"l"(qp + next * p.sq.h + x));
          }
          for (int x = 32 * (ht & 3); x < p.vs; x += 128) asm volatile("prefetch.global.L2 [%0];" ::"l"(vp + next * p.sv.h + x));
        }
      }
      cp_async_commit();
    };
    auto prepare = [&](int c) {
      const int buf = c & 1;
      float* gt = gates_of(c);
      const uint32_t kt = sb + lay.K + buf * lay.tile_k, qt = sb + lay.Q + buf * lay.tile_k;
      cp_async_wait_1();   // only the gate values of the next read-out may still be on their way
      bar_sync(1, HT);
      {  // squared norms of the 64 k rows and the 64 q rows, two threads per row
        const int row = ht >> 1, i = row & (C - 1);
        const bool is_q = row >= C;
        const uint8_t* src = sm + (is_q ? lay.Q : lay.K) + buf * lay.tile_k + i * lay.ldk * 2 + (ht & 1) * d;
        float ss = 0.f;
#pragma unroll
        for (int cc = 0; cc < d / 16; ++cc) {
          float x[8];
          seq::Pack<bf16, 8>::load(reinterpret_cast<const bf16*>(src) + 8 * cc, x);
#pragma unroll
          for (int e = 0; e < 8; ++e) ss = fmaf(x[e], x[e], ss);
        }
        ss += __shfl_xor_sync(0xffffffffu, ss, 1);
        if ((ht & 1) == 0) {
          const float r = rsqrtf(ss + kUnitEps), G = gt[G_CUM * C + i];
          if (is_q) {
            const float rq = r * rsqrtf((float)d);
            gt[G_RQ * C + i] = rq;
            gt[G_EGQ * C + i] = ex2(G) * rq;
          } else {
            gt[G_RK * C + i] = r;
            gt[G_EGK * C + i] = ex2(G) * r;
            gt[G_W * C + i] = ex2(gt[G_TOT * C] - G) * r;
            gt[G_COL * C + i] = ex2(gt[G_CUM * C + (i | 15)] - G) * r;   // decay from here to the end of the 16-block
          }
        }
      }
      bar_sync(1, HT);
      // 16 x 16 blocks of K K^T and Q K^T on and below the diagonal, both products of a block by one warp; the diagonal
      // ones first.  Off the diagonal e^{G_i - G_j} splits at the end of j's block into two factors of at most 1.
      bf16* Th = reinterpret_cast<bf16*>(sm + lay.R + buf * lay.region);
      bf16 *Tl = Th + C * LT, *Ph = Tl + C * LT;
      for (int t = hw; t < 10; t += kHelpers) {
        const int bi = t < 4 ? t : t == 4 ? 1 : t < 7 ? 2 : 3, bj = t < 4 ? t : t == 4 ? 0 : t < 7 ? t - 5 : t - 7;
        float kk2[2][4] = {}, qk2[2][4] = {};
        const uint32_t ra = ((bi * 16 + (lane & 15)) * lay.ldk + (lane >> 4) * 8) * 2;
        const uint32_t ba = kt + ((bj * 16 + (lane & 7) + (lane >> 4) * 8) * lay.ldk + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
        for (int kk = 0; kk < DK; ++kk) {
          uint32_t fk[4], fq[4], fb[4];
          ldsm4(fb, ba + kk * 32);
          ldsm4(fk, kt + ra + kk * 32);
          ldsm4(fq, qt + ra + kk * 32);
          mma(kk2[0], fk, fb[0], fb[1]);
          mma(kk2[1], fk, fb[2], fb[3]);
          mma(qk2[0], fq, fb[0], fb[1]);
          mma(qk2[1], fq, fb[2], fb[3]);
        }
        const bool diag = bi == bj;
        const float end = gt[G_CUM * C + bj * 16 + 15];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int ii = g + 8 * half, i = bi * 16 + ii;
          const float Gi = gt[G_CUM * C + i];
          float fk = gt[G_BETA * C + i] * gt[G_RK * C + i], fq = gt[G_RQ * C + i];
          if (!diag) {
            const float ei = ex2(Gi - end);
            fk *= -ei;
            fq *= ei;
          }
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            const int jj = nt * 8 + 2 * t4, j = bj * 16 + jj;
            float a0 = kk2[nt][2 * half] * fk, a1 = kk2[nt][2 * half + 1] * fk, p0 = qk2[nt][2 * half] * fq, p1 = qk2[nt][2 * half + 1] * fq;
            if (diag) {
              const float2 gj = *reinterpret_cast<const float2*>(gt + G_CUM * C + j), rk = *reinterpret_cast<const float2*>(gt + G_RK * C + j);
              const float e0 = jj <= ii ? ex2(Gi - gj.x) * rk.x : 0.f, e1 = jj + 1 <= ii ? ex2(Gi - gj.y) * rk.y : 0.f;
              inv[(bi * 16 + jj) * LI + ii] = jj < ii ? a0 * e0 : 0.f;
              inv[(bi * 16 + jj + 1) * LI + ii] = jj + 1 < ii ? a1 * e1 : 0.f;
              p0 *= e0;
              p1 *= e1;
            } else {
              const float2 cj = *reinterpret_cast<const float2*>(gt + G_COL * C + j);
              uint32_t hi, lo;
              split(a0 * cj.x, a1 * cj.y, hi, lo);
              *reinterpret_cast<uint32_t*>(Th + i * LT + j) = hi;
              *reinterpret_cast<uint32_t*>(Tl + i * LT + j) = lo;
              p0 *= cj.x;
              p1 *= cj.y;
            }
            *reinterpret_cast<uint32_t*>(Ph + i * LT + j) = pack_bf16(p0, p1);
          }
        }
      }
      if (hw == kHelpers - 1 && c + 1 < nc) gates(c + 1);
      bar_sync(1, HT);
      if (hw < 4 && lane < 16) {  // one column of one diagonal block's inverse per thread
        float t[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) t[i] = i == lane ? 1.f : 0.f;
#pragma unroll
        for (int k = 0; k < 15; ++k) {
          float col[16];   // column k of the block, from its diagonal's 4-group on
#pragma unroll
          for (int i4 = k / 4 * 4; i4 < 16; i4 += 4) {
            const float4 x = *reinterpret_cast<const float4*>(inv + (hw * 16 + k) * LI + i4);
            col[i4] = x.x; col[i4 + 1] = x.y; col[i4 + 2] = x.z; col[i4 + 3] = x.w;
          }
#pragma unroll
          for (int i = k + 1; i < 16; ++i) t[i] = fmaf(-col[i], t[k], t[i]);
        }
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const bf16 hi = __float2bfloat16_rn(t[i]);
          Th[(hw * 16 + i) * LT + hw * 16 + lane] = hi;
          Tl[(hw * 16 + i) * LT + hw * 16 + lane] = __float2bfloat16_rn(t[i] - __bfloat162float(hi));
        }
      }
      mbar_arrive(READY + 8 * buf);
    };

    // 4 threads per token of a chunk, every 4th group of 4 values
    const int fi = ht >> 2, fpart = ht & 3, groups = p.vs / 4;
    constexpr int FG = 8;      // groups per thread at 128 columns
    // z values of the next read-out, 8 bytes per group, read back by the thread that copied them
    const uint32_t zs = sb + lay.z + ht * 8;
    const uint2* zr = reinterpret_cast<const uint2*>(sm + lay.z) + ht;
    auto fetch_z = [&](int c) {
      const int l = c * C + fi;
      if (!p.raw && l < p.L) {
        const bf16* zp = p.z + b * p.sz.b + (int64_t)l * p.sz.h + (int64_t)h * p.dv;
#pragma unroll
        for (int r = 0; r < FG; ++r)
          if (fpart + 4 * r < groups)
            asm volatile("cp.async.ca.shared.global [%0], [%1], 8;\n" ::"r"(zs + r * HT * 8), "l"(zp + 4 * (fpart + 4 * r)) : "memory");
      }
      cp_async_commit();
    };
    auto finish = [&](int c) {  // read-out of chunk c -> output
      const int buf = c & 1, l = c * C + fi;
      const float* st = reinterpret_cast<const float*>(sm + lay.R + buf * lay.region) + fi * lay.ldo;
      if (p.raw) {
        if (l < p.L) {
          float* dst = p.raw + (((int64_t)b * p.L + l) * p.H + h) * p.dv + v0;
          for (int e = fpart; e < groups; e += 4)
            *reinterpret_cast<float4*>(dst + 4 * e) = *reinterpret_cast<const float4*>(st + 4 * e);
        }
        return;
      }
      const float* wn = reinterpret_cast<const float*>(sm + lay.w);
      float ss = 0.f;
      for (int e = fpart; e < groups; e += 4) {
        const float4 x = *reinterpret_cast<const float4*>(st + 4 * e);
        ss += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
      }
      ss += __shfl_xor_sync(0xffffffffu, ss, 1);
      ss += __shfl_xor_sync(0xffffffffu, ss, 2);
      if (l >= p.L) return;
      const float rstd = rsqrtf(ss / (float)p.dv + p.eps);
      bf16* op = p.out + b * p.so.b + (int64_t)l * p.so.h + (int64_t)h * p.dv;
      auto some = [&](int r0, auto count) {   // groups r0 .. r0 + count - 1 of this thread, without branches in between
        constexpr int N = decltype(count)::value;
        float4 x[N], w[N];
        uint2 z[N];
#pragma unroll
        for (int r = 0; r < N; ++r) {
          const int e = fpart + 4 * (r0 + r);
          x[r] = *reinterpret_cast<const float4*>(st + 4 * e);
          w[r] = *reinterpret_cast<const float4*>(wn + 4 * e);
          z[r] = zr[(r0 + r) * HT];
        }
#pragma unroll
        for (int r = 0; r < N; ++r) {
          const float o[4] = {x[r].x * rstd * w[r].x * seq::silu_t<bf16>(seq::bf16_lo(z[r].x)),
                              x[r].y * rstd * w[r].y * seq::silu_t<bf16>(seq::bf16_hi(z[r].x)),
                              x[r].z * rstd * w[r].z * seq::silu_t<bf16>(seq::bf16_lo(z[r].y)),
                              x[r].w * rstd * w[r].w * seq::silu_t<bf16>(seq::bf16_hi(z[r].y))};
          seq::Pack<bf16, 4>::store(op + 4 * (fpart + 4 * (r0 + r)), o);
        }
      };
      const int mine = p.vs / 16;
      int r0 = 0;
      for (; r0 + 4 <= mine; r0 += 4) some(r0, std::integral_constant<int, 4>{});
      for (; r0 < mine; ++r0) some(r0, std::integral_constant<int, 1>{});
    };

    // Copy groups in order: tiles(0), z(0), [tiles(1),] then per chunk tiles(c + 2), z(c + 1): whoever waits for a group
    // leaves one younger group in flight.
    if (!p.raw)
      for (int e = ht; e < p.vs; e += HT) reinterpret_cast<float*>(sm + lay.w)[e] = __bfloat162float(p.norm_w[e]);
    if (hw == kHelpers - 1) gates(0);
    load(0);
    fetch_z(0);
    prepare(0);
    if (nc > 1) {
      load(1);
      cp_async_commit();   // an empty group, so that the wait below is for the tiles
      prepare(1);
    }
    for (int c = 0; c < nc; ++c) {
      mbar_wait_bounded(DONE + 8 * (c & 1), (c >> 1) & 1, abort_flag, p.status, 1u << 16);
      if (c + 2 < nc) load(c + 2);   // lands while the read-out is finished
      else cp_async_commit();
      cp_async_wait_1();             // z(c)
      finish(c);
      if (c + 1 < nc) fetch_z(c + 1);
      if (c + 2 < nc) {
        bar_sync(1, HT);   // every helper has read the stage before the next chunk's matrices overwrite it
        prepare(c + 2);
      }
    }
  } else {
    // ------------------------------------------------------------ consumers
    reg_inc<168>();
    if (warp < active) {
      const int g = lane >> 2, t4 = lane & 3;
      float s[2 * DK][4];   // S^T tiles: rows = value columns v0 + 16 warp + {g, g + 8}, columns = key dims 8 n + 2 t4 + {0, 1}
      const int64_t sbase = ((int64_t)b * p.H + h) * d * p.dv + v0 + 16 * warp + g;
      const bool fresh = seq::position0(p.offsets, p.offset, b) == 0;
#pragma unroll
      for (int n = 0; n < 2 * DK; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e)
          s[n][e] = fresh ? 0.f : p.state[sbase + (int64_t)(8 * n + 2 * t4 + (e & 1)) * p.dv + (e >> 1) * 8];
      // lane parts of the ldmatrix addresses (bytes)
      const uint32_t b_lane = (((lane & 7) + (lane >> 4) * 8) * lay.ldk + ((lane >> 3) & 1) * 8) * 2;   // [n 16][k 16], K / Q
      const uint32_t t_lane = (((lane & 7) + (lane >> 4) * 8) * LT + ((lane >> 3) & 1) * 8) * 2;        // the same in T / P
      const uint32_t k_lane = ((lane & 15) * lay.ldk + (lane >> 4) * 8) * 2;                            // transposed: [k 16][n 16]
      const uint32_t v_lane = ((lane & 15) * lay.ldv + (lane >> 4) * 8 + 16 * warp) * 2;                // transposed: [tokens 16][cols 16]
      for (int c = 0; c < nc; ++c) {
        const int buf = c & 1;
        const float* gt = reinterpret_cast<const float*>(sm + lay.gates) + (c % 3) * G_N * C;
        const uint32_t kt = sb + lay.K + buf * lay.tile_k, qt = sb + lay.Q + buf * lay.tile_k, vt = sb + lay.V + buf * lay.tile_v;
        const uint32_t th = sb + lay.R + buf * lay.region + t_lane, tl = th + C * LT * 2, ph = tl + C * LT * 2;
        mbar_wait_bounded(READY + 8 * buf, (c >> 1) & 1, abort_flag, p.status, 1u << 17);
        float x[8][4], o[8][4];   // [16 value columns, 64 tokens]: S0^T k, then the residual, then u; S0^T q, then the read-out
#pragma unroll
        for (int n = 0; n < 8; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) { x[n][e] = 0.f; o[n][e] = 0.f; }
#pragma unroll
        for (int kk = 0; kk < DK; ++kk) {
          uint32_t ah[4], al[4];
          split_a(s[2 * kk], s[2 * kk + 1], ah, al);
#pragma unroll
          for (int np = 0; np < 4; ++np) {
            uint32_t fb[4];
            ldsm4(fb, kt + b_lane + (np * 16 * lay.ldk + kk * 16) * 2);
            mma(x[2 * np], ah, fb[0], fb[1]);
            mma(x[2 * np + 1], ah, fb[2], fb[3]);
            mma(x[2 * np], al, fb[0], fb[1]);
            mma(x[2 * np + 1], al, fb[2], fb[3]);
            ldsm4(fb, qt + b_lane + (np * 16 * lay.ldk + kk * 16) * 2);
            mma(o[2 * np], ah, fb[0], fb[1]);
            mma(o[2 * np + 1], ah, fb[2], fb[3]);
          }
        }
        // y = beta (v - e^G S0^T khat); decayed read-out of S0
#pragma unroll
        for (int np = 0; np < 4; ++np) {
          uint32_t fv[4];   // (tokens 0-7 | 8-15) x (columns g | g + 8)
          ldsm4t(fv, vt + v_lane + np * 16 * lay.ldv * 2);
#pragma unroll
          for (int q = 0; q < 2; ++q) {
            const int n = 2 * np + q, tok = 8 * n + 2 * t4;
            const float2 be = *reinterpret_cast<const float2*>(gt + G_BETA * C + tok);
            const float2 ek = *reinterpret_cast<const float2*>(gt + G_EGK * C + tok);
            const float2 eq = *reinterpret_cast<const float2*>(gt + G_EGQ * C + tok);
            const uint32_t lo = fv[q], hi = fv[q + 2];
            x[n][0] = be.x * (seq::bf16_lo(lo) - ek.x * x[n][0]);
            x[n][1] = be.y * (seq::bf16_hi(lo) - ek.y * x[n][1]);
            x[n][2] = be.x * (seq::bf16_lo(hi) - ek.x * x[n][2]);
            x[n][3] = be.y * (seq::bf16_hi(hi) - ek.y * x[n][3]);
            o[n][0] *= eq.x; o[n][1] *= eq.y; o[n][2] *= eq.x; o[n][3] *= eq.y;
          }
        }
        // S <- e^{G_C} S + sum_j (w_j u_j) k_j: decayed here, each block's sum added as soon as its u is known, so that
        // these products fill the gaps of the block-by-block solution
        const float gc = ex2(gt[G_TOT * C]);
#pragma unroll
        for (int n = 0; n < 2 * DK; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[n][e] *= gc;
        // blocks of 16 tokens: u_b = T_b (residual), then its part in the later residuals and in the read-out
#pragma unroll
        for (int bb = 0; bb < 4; ++bb) {
          uint32_t fh[4], fl[4], mh[4], ml[4];
          split_a(x[2 * bb], x[2 * bb + 1], fh, fl);
          ldsm4(mh, th + (bb * 16 * LT + bb * 16) * 2);
          ldsm4(ml, tl + (bb * 16 * LT + bb * 16) * 2);
#pragma unroll
          for (int q = 0; q < 2; ++q) {
            float u[4] = {0.f, 0.f, 0.f, 0.f};
            mma(u, fl, mh[2 * q], mh[2 * q + 1]);
            mma(u, fh, ml[2 * q], ml[2 * q + 1]);
            mma(u, fh, mh[2 * q], mh[2 * q + 1]);
#pragma unroll
            for (int e = 0; e < 4; ++e) x[2 * bb + q][e] = u[e];
          }
          split_a(x[2 * bb], x[2 * bb + 1], fh, fl);
#pragma unroll
          for (int np = bb; np < 4; ++np) {
            if (np > bb) {
              ldsm4(mh, th + (np * 16 * LT + bb * 16) * 2);
              ldsm4(ml, tl + (np * 16 * LT + bb * 16) * 2);
              mma(x[2 * np], fl, mh[0], mh[1]);
              mma(x[2 * np + 1], fl, mh[2], mh[3]);
              mma(x[2 * np], fh, ml[0], ml[1]);
              mma(x[2 * np + 1], fh, ml[2], ml[3]);
              mma(x[2 * np], fh, mh[0], mh[1]);
              mma(x[2 * np + 1], fh, mh[2], mh[3]);
            }
            ldsm4(mh, ph + (np * 16 * LT + bb * 16) * 2);
            mma(o[2 * np], fh, mh[0], mh[1]);
            mma(o[2 * np + 1], fh, mh[2], mh[3]);
          }
#pragma unroll
          for (int q = 0; q < 2; ++q) {
            const float2 w = *reinterpret_cast<const float2*>(gt + G_W * C + 16 * bb + 8 * q + 2 * t4);
            x[2 * bb + q][0] *= w.x; x[2 * bb + q][1] *= w.y; x[2 * bb + q][2] *= w.x; x[2 * bb + q][3] *= w.y;
          }
          split_a(x[2 * bb], x[2 * bb + 1], fh, fl);
#pragma unroll
          for (int np = 0; np < DK; ++np) {
            uint32_t fb[4];
            ldsm4t(fb, kt + k_lane + (bb * 16 * lay.ldk + np * 16) * 2);
            mma(s[2 * np], fl, fb[0], fb[1]);
            mma(s[2 * np + 1], fl, fb[2], fb[3]);
            mma(s[2 * np], fh, fb[0], fb[1]);
            mma(s[2 * np + 1], fh, fb[2], fb[3]);
          }
        }
        bar_sync(2, 32 * active);   // every consumer is through with T and P: the stage may overwrite them
        {
          float* st = reinterpret_cast<float*>(sm + lay.R + buf * lay.region) + 16 * warp + g;
#pragma unroll
          for (int n = 0; n < 8; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) st[(8 * n + 2 * t4 + (e & 1)) * lay.ldo + (e >> 1) * 8] = o[n][e];
        }
        mbar_arrive(DONE + 8 * buf);
      }
#pragma unroll
      for (int n = 0; n < 2 * DK; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) p.state[sbase + (int64_t)(8 * n + 2 * t4 + (e & 1)) * p.dv + (e >> 1) * 8] = s[n][e];
    }
  }
}

// out = raw / rms(raw) * norm_w * silu(z), one warp per (token, head)
__global__ void __launch_bounds__(128) delta_finish_kernel(const Params p) {
  const int64_t row = (int64_t)blockIdx.x * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (row >= (int64_t)p.B * p.L * p.H) return;
  const int h = row % p.H;
  const int64_t t = row / p.H;
  const int l = t % p.L, b = t / p.L;
  const float* x = p.raw + row * p.dv;
  float ss = 0.f;
  for (int c = 4 * lane; c < p.dv; c += 128) {
    const float4 v = *reinterpret_cast<const float4*>(x + c);
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  const float rstd = rsqrtf(warp_sum(ss) / (float)p.dv + p.eps);
  const bf16* z = p.z + b * p.sz.b + l * p.sz.h + (int64_t)h * p.dv;
  bf16* out = p.out + b * p.so.b + l * p.so.h + (int64_t)h * p.dv;
  for (int c = 4 * lane; c < p.dv; c += 128) {
    const float4 v = *reinterpret_cast<const float4*>(x + c);
    const float xv[4] = {v.x, v.y, v.z, v.w};
    float zv[4], w[4], o[4];
    seq::Pack<bf16, 4>::load(z + c, zv);
    seq::Pack<bf16, 4>::load(p.norm_w + c, w);
#pragma unroll
    for (int r = 0; r < 4; ++r) o[r] = xv[r] * rstd * w[r] * seq::silu_t<bf16>(zv[r]);
    seq::Pack<bf16, 4>::store(out + c, o);
  }
}

constexpr int kMaxSmem = 227 * 1024;

template <int DK>
int launch_dk(const Params& p, int slices, cudaStream_t st) {
  const Layout lay(16 * DK, p.vs);
  if (lay.total > kMaxSmem) return BASED_ERR_IMPL;
  const cudaError_t e = cudaFuncSetAttribute(delta_chunk_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxSmem);
  if (e != cudaSuccess) return (int)e;
  delta_chunk_kernel<DK><<<dim3(p.H, p.B, slices), NT, lay.total, st>>>(p);
  return (int)cudaGetLastError();
}

bool sizes_ok(int d, int dv) { return (d == 32 || d == 64 || d == 96 || d == 128) && dv % 16 == 0 && dv <= 1024; }

// slices of the value columns: as many as keep the SMs busy, none narrower than 32 columns
int slices_of(int B, int H, int dv) {
  int n = (dv + 127) / 128;
  while (dv % (16 * n)) ++n;
  while (2 * n * B * H <= 148 && dv / (2 * n) >= 32 && dv % (32 * n) == 0) n *= 2;
  return n;
}

}  // namespace

int read_tc_status_delta(unsigned int* out, int reset) {
  unsigned int v = 0;
  cudaError_t e = cudaMemcpyFromSymbol(&v, g_tc_status_delta, sizeof(v));
  if (e != cudaSuccess) return (int)e;
  if (out) *out = v;
  if (reset && v != 0) {
    v = 0;
    e = cudaMemcpyToSymbol(g_tc_status_delta, &v, sizeof(v));
  }
  return (int)e;
}

size_t delta_chunk_scratch_bytes(int B, int L, int H, int d, int dv) {
  if (!sizes_ok(d, dv) || slices_of(B, H, dv) == 1) return 0;
  return (size_t)B * L * H * dv * sizeof(float);
}

// BASED_ERR_IMPL: sizes, strides or alignment this kernel does not take.
int launch_delta_chunk(const void* q, const void* k, const void* v, const void* z, const float* a, const float* b,
                       const float* A_log, const float* dt_bias, const void* norm_w, float* state, void* out, void* scratch,
                       size_t scratch_bytes, int B, int L, int H, int Hk, int d, int dv, Strides2 sq, Strides2 sk,
                       Strides2 sv, Strides2 sz, Strides2 sg, Strides2 so, const int32_t* offsets, int offset, float eps,
                       cudaStream_t stream) {
  if (!sizes_ok(d, dv) || B > 65535) return BASED_ERR_IMPL;
  if (!aligned16(q) || !aligned16(k) || !aligned16(v) || !aligned16(z) || !aligned16(out) || !aligned16(norm_w)) return BASED_ERR_IMPL;
  for (const Strides2& s : {sq, sk, sv, sz, so})
    if ((B > 1 && s.b % 8) || s.h % 8) return BASED_ERR_IMPL;
  const int slices = slices_of(B, H, dv);
  Params p{static_cast<const bf16*>(q), static_cast<const bf16*>(k), static_cast<const bf16*>(v), static_cast<const bf16*>(z),
           static_cast<const bf16*>(norm_w), a, b, A_log, dt_bias, state, nullptr, static_cast<bf16*>(out), offsets, offset,
           B, L, H, Hk, dv, dv / slices, sq, sk, sv, sz, sg, so, eps, nullptr};
  if (slices > 1) {
    if (!scratch || scratch_bytes < delta_chunk_scratch_bytes(B, L, H, d, dv) || !aligned16(scratch)) return BASED_ERR_SCRATCH;
    p.raw = static_cast<float*>(scratch);
  }
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
      e = cudaGetSymbolAddress(reinterpret_cast<void**>(&addr), g_tc_status_delta);
      if (e != cudaSuccess) return (int)e;
      status[dev] = addr;
    }
    p.status = status[dev];
  }
  int rc;
  if (d == 32) rc = launch_dk<2>(p, slices, stream);
  else if (d == 64) rc = launch_dk<4>(p, slices, stream);
  else if (d == 96) rc = launch_dk<6>(p, slices, stream);
  else rc = launch_dk<8>(p, slices, stream);
  if (rc != 0 || slices == 1) return rc;
  const int64_t rows = (int64_t)B * L * H;
  delta_finish_kernel<<<(unsigned)((rows + 3) / 4), 128, 0, stream>>>(p);
  return (int)cudaGetLastError();
}

}  // namespace based
