// The two elementwise / row-wise steps that sit between the mixers and the GEMMs of a block:
//
//  * residual add + RMSNorm in one pass: z = x + residual; residual_out = z; out = z * rstd(z) * w + b.
//    Replaces the Triton kernel behind RMSNorm.forward / rms_norm_fn as Block.forward and
//    GPTModel.forward call it with prenorm=True (based/ops/triton/layer_norm.py:926-953, semantics
//    restated in rms_norm_ref :74-125; call sites based/models/block.py:134-163 and
//    based/models/gpt.py:696-733).
//  * gated activation of the MLP: out = y * act(gate) with (y, gate) the two halves of fc1's output.
//    Replaces `y, gate = y.chunk(2, dim=-1); y = swiglu(gate, y)` / F.glu in GatedMlp.forward
//    (based/models/mlp.py:141-154), where the reference uses flash-attn's jiterator swiglu.
//
//  * the norm step of a PARALLEL block (x <- x + m * (mixer(norm1(x)) + mlp(norm2(x)))): the previous block's scaled
//    branch sum is added to the fp32 residual stream and the new stream is normed once and scaled by TWO weights
//    (the two norms of one x share their root mean square).  With token ids instead of a branch the row is
//    norm(embedding[token]), so a model's first step is the same launch.
//
//  * the norm step of a POST-norm block (x <- x + norm(sublayer(x))): the sublayer's output is normed, added to the fp32
//    stream, and the new stream is handed on in the activations' dtype, plain or with a norm of its own (a model's last).
//    stream_embed starts such a stream: scaled token vector plus position vector.
//  * norm_gate: norm(x) * w * sigmoid(gate).  token_gate: gelu(z) times a slice of the token's own vector.
//
// All are HBM-bound; 16-byte vector accesses, fp32 arithmetic, one read of every input.
#include "seq_common.cuh"

namespace based {
namespace {

template <typename T>
struct V16;  // 16 bytes of T <-> floats
template <>
struct V16<float> {
  static constexpr int N = 4;
  static __device__ __forceinline__ void unpack(const uint4& v, float (&x)[4]) {
    x[0] = __uint_as_float(v.x); x[1] = __uint_as_float(v.y); x[2] = __uint_as_float(v.z); x[3] = __uint_as_float(v.w);
  }
  static __device__ __forceinline__ void load(const float* p, float (&x)[4]) {
    unpack(*reinterpret_cast<const uint4*>(p), x);
  }
  static __device__ __forceinline__ void store(float* p, const float (&x)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1], x[2], x[3]);
  }
};
template <>
struct V16<__nv_bfloat16> {
  static constexpr int N = 8;
  static __device__ __forceinline__ void unpack(const uint4& v, float (&x)[8]) {
    const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      x[2 * i] = __uint_as_float(w[i] << 16);
      x[2 * i + 1] = __uint_as_float(w[i] & 0xFFFF0000u);
    }
  }
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&x)[8]) {
    unpack(*reinterpret_cast<const uint4*>(p), x);
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&x)[8]) {
    uint4 v;
    uint32_t* w = reinterpret_cast<uint32_t*>(&v);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const __nv_bfloat162 h = __floats2bfloat162_rn(x[2 * i], x[2 * i + 1]);
      w[i] = *reinterpret_cast<const uint32_t*>(&h);
    }
    *reinterpret_cast<uint4*>(p) = v;
  }
};

// 8 consecutive values of a tensor of runtime dtype (two 16-byte loads when it is fp32)
__device__ __forceinline__ void load8(const void* base, int bf16, int64_t idx, float (&x)[8]) {
  if (bf16) {
    V16<__nv_bfloat16>::load(static_cast<const __nv_bfloat16*>(base) + idx, x);
  } else {
    float a[4], b[4];
    V16<float>::load(static_cast<const float*>(base) + idx, a);
    V16<float>::load(static_cast<const float*>(base) + idx + 4, b);
#pragma unroll
    for (int i = 0; i < 4; ++i) { x[i] = a[i]; x[4 + i] = b[i]; }
  }
}
__device__ __forceinline__ void store8(void* base, int bf16, int64_t idx, const float (&x)[8]) {
  if (bf16) {
    V16<__nv_bfloat16>::store(static_cast<__nv_bfloat16*>(base) + idx, x);
  } else {
    const float a[4] = {x[0], x[1], x[2], x[3]}, b[4] = {x[4], x[5], x[6], x[7]};
    V16<float>::store(static_cast<float*>(base) + idx, a);
    V16<float>::store(static_cast<float*>(base) + idx + 4, b);
  }
}

struct NormParams {
  const void *x, *residual, *weight, *bias;
  void *out, *residual_out;
  int64_t M, sx, sr, so, sro;  // rows and row strides (elements)
  int D, io_bf16, res_bf16, w_bf16, round_input;
  float eps;
};

constexpr int NORM_THREADS = 128;

// One row per block; thread t owns the 8-value groups t, t + 128, ... (VPT of them, in registers
// between the reduction and the scaling, so the row is read once).
template <int VPT>
__global__ void __launch_bounds__(NORM_THREADS) add_rmsnorm_kernel(const NormParams p) {
  const int64_t row = blockIdx.x;
  const int ngroups = p.D >> 3;
  float z[VPT][8];
  float ss = 0.f;
#pragma unroll
  for (int v = 0; v < VPT; ++v) {
    const int g = threadIdx.x + v * NORM_THREADS;
    if (g < ngroups) {
      load8(p.x, p.io_bf16, row * p.sx + 8 * g, z[v]);
      if (p.residual) {
        float r[8];
        load8(p.residual, p.res_bf16, row * p.sr + 8 * g, r);
#pragma unroll
        for (int i = 0; i < 8; ++i) z[v][i] += r[i];
      }
      if (p.residual_out) {
        store8(p.residual_out, p.res_bf16, row * p.sro + 8 * g, z[v]);
        if (p.res_bf16) {  // the norm sees the residual stream as it is stored
#pragma unroll
          for (int i = 0; i < 8; ++i) z[v][i] = __bfloat162float(__float2bfloat16_rn(z[v][i]));
        }
      }
      if (p.round_input && p.io_bf16) {  // the norm sees z cast to the activation dtype
#pragma unroll
        for (int i = 0; i < 8; ++i) z[v][i] = __bfloat162float(__float2bfloat16_rn(z[v][i]));
      }
#pragma unroll
      for (int i = 0; i < 8; ++i) ss = fmaf(z[v][i], z[v][i], ss);
    }
  }
  __shared__ float part[NORM_THREADS / 32];
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xFFFFFFFFu, ss, o);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int w = 0; w < NORM_THREADS / 32; ++w) tot += part[w];
  const float rstd = rsqrtf(tot / (float)p.D + p.eps);
#pragma unroll
  for (int v = 0; v < VPT; ++v) {
    const int g = threadIdx.x + v * NORM_THREADS;
    if (g < ngroups) {
      float w[8], o[8];
      load8(p.weight, p.w_bf16, 8 * g, w);
#pragma unroll
      for (int i = 0; i < 8; ++i) o[i] = z[v][i] * rstd * w[i];
      if (p.bias) {
        load8(p.bias, p.w_bf16, 8 * g, w);
#pragma unroll
        for (int i = 0; i < 8; ++i) o[i] += w[i];
      }
      store8(p.out, p.io_bf16, row * p.so + 8 * g, o);
    }
  }
}

__device__ __forceinline__ float block_sum(float v) {
  __shared__ float part[NORM_THREADS / 32];
  __syncthreads();  // part may still be read by a previous call
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int w = 0; w < NORM_THREADS / 32; ++w) tot += part[w];
  return tot;
}
// Plain RMSNorm of rows of any width and alignment, one value per access.
template <typename T>
__global__ void __launch_bounds__(NORM_THREADS) rmsnorm_scalar_kernel(const T* x, const T* w, T* out, int D, int64_t sx,
                                                                      int64_t so, float eps) {
  x += blockIdx.x * sx;
  out += blockIdx.x * so;
  float ss = 0.f;
  for (int c = threadIdx.x; c < D; c += NORM_THREADS) { const float z = to_float<T>(x[c]); ss = fmaf(z, z, ss); }
  const float rstd = rsqrtf(block_sum(ss) / (float)D + eps);
  for (int c = threadIdx.x; c < D; c += NORM_THREADS) out[c] = from_float<T>(to_float<T>(x[c]) * rstd * to_float<T>(w[c]));
}

// ---- parallel block: residual stream update and one or two norms of the result
struct StreamParams {
  const int64_t* tokens;                  // [M] with table [V, D] and table_norm [D]: the row is norm(table[token])
  const void *table, *table_norm, *branch;
  float* residual;                        // [M, D] fp32, read (unless tokens) and written in place
  const void *w1, *w2;                    // [D] each; w2 / out2 may be null
  void *out1, *out2;
  int64_t M, V, sb;                       // sb: row stride of branch; residual and outputs are contiguous
  int D;
  float mult, eps;
};

// One row per block; N values per access (8, or 1 for any D), VPT accesses per thread kept in registers.
template <typename T, int N, int VPT>
__global__ void __launch_bounds__(NORM_THREADS) stream_norm_kernel(const StreamParams p) {
  using seq::Pack;
  const int64_t row = blockIdx.x;
  const int groups = p.D / N;
  float* res = p.residual + row * p.D;
  float z[VPT][N];
  auto load_res = [&](int g, float (&v)[N]) {
    if constexpr (N == 8) load8(res, 0, 8 * g, v);
    else v[0] = res[g];
  };
  auto store_res = [&](int g, const float (&v)[N]) {
    if constexpr (N == 8) store8(res, 0, 8 * g, v);
    else res[g] = v[0];
  };
  const int64_t tok = p.tokens ? p.tokens[row] : 0;
  const bool known = tok >= 0 && tok < p.V;   // an id outside the table reads as a zero row
  const T* src = p.tokens ? static_cast<const T*>(p.table) + (known ? tok : 0) * p.D
                          : static_cast<const T*>(p.branch) + row * p.sb;
  float ss = 0.f;
#pragma unroll
  for (int v = 0; v < VPT; ++v) {
    const int g = threadIdx.x + v * NORM_THREADS;
    if (g < groups) {
      float b[N];
      if (p.tokens || p.branch) Pack<T, N>::load(src + (int64_t)g * N, b);
      if (!p.tokens) load_res(g, z[v]);
#pragma unroll
      for (int i = 0; i < N; ++i) {
        if (p.tokens) z[v][i] = known ? b[i] : 0.f;
        else if (p.branch) z[v][i] = fmaf(p.mult, b[i], z[v][i]);
        ss = fmaf(z[v][i], z[v][i], ss);
      }
      if (!p.tokens && p.branch) store_res(g, z[v]);
    }
  }
  float tot = block_sum(ss);
  if (p.tokens) {
    const float rstd = rsqrtf(tot / (float)p.D + p.eps);
    ss = 0.f;
#pragma unroll
    for (int v = 0; v < VPT; ++v) {
      const int g = threadIdx.x + v * NORM_THREADS;
      if (g < groups) {
        float w[N];
        Pack<T, N>::load(static_cast<const T*>(p.table_norm) + (int64_t)g * N, w);
#pragma unroll
        for (int i = 0; i < N; ++i) {
          z[v][i] *= rstd * w[i];
          ss = fmaf(z[v][i], z[v][i], ss);
        }
        store_res(g, z[v]);
      }
    }
    tot = block_sum(ss);
  }
  const float rstd = rsqrtf(tot / (float)p.D + p.eps);
#pragma unroll
  for (int v = 0; v < VPT; ++v) {
    const int g = threadIdx.x + v * NORM_THREADS;
    if (g < groups) {
      float w[N], o[N];
      Pack<T, N>::load(static_cast<const T*>(p.w1) + (int64_t)g * N, w);
#pragma unroll
      for (int i = 0; i < N; ++i) o[i] = z[v][i] * rstd * w[i];
      Pack<T, N>::store(static_cast<T*>(p.out1) + row * p.D + (int64_t)g * N, o);
      if (p.out2) {
        Pack<T, N>::load(static_cast<const T*>(p.w2) + (int64_t)g * N, w);
#pragma unroll
        for (int i = 0; i < N; ++i) o[i] = z[v][i] * rstd * w[i];
        Pack<T, N>::store(static_cast<T*>(p.out2) + row * p.D + (int64_t)g * N, o);
      }
    }
  }
}

// ---- post-norm block
struct PostNormParams {
  const void *branch, *w;      // [M, D] and [D]
  float* residual;             // [M, D] fp32, updated in place
  const void* w_out;           // [D] or null: out = norm(residual) * w_out, else out = residual
  void* out;                   // [M, D] in T; null: nothing but the stream is written
  int64_t sb;
  int D;
  float eps;
};

template <typename T, int N, int VPT>
__global__ void __launch_bounds__(NORM_THREADS) stream_post_norm_kernel(const PostNormParams p) {
  using seq::Pack;
  const int64_t row = blockIdx.x;
  const int groups = p.D / N;
  float* res = p.residual + row * p.D;
  const T* br = static_cast<const T*>(p.branch) + row * p.sb;
  float z[VPT][N], r[VPT][N];
  float ss = 0.f;
#pragma unroll
  for (int v = 0; v < VPT; ++v) {
    const int g = threadIdx.x + v * NORM_THREADS;
    if (g < groups) {
      Pack<T, N>::load(br + (int64_t)g * N, z[v]);
      Pack<float, N>::load(res + (int64_t)g * N, r[v]);
#pragma unroll
      for (int i = 0; i < N; ++i) ss = fmaf(z[v][i], z[v][i], ss);
    }
  }
  float rstd = rsqrtf(block_sum(ss) / (float)p.D + p.eps);
  ss = 0.f;
#pragma unroll
  for (int v = 0; v < VPT; ++v) {
    const int g = threadIdx.x + v * NORM_THREADS;
    if (g < groups) {
      float w[N];
      Pack<T, N>::load(static_cast<const T*>(p.w) + (int64_t)g * N, w);
#pragma unroll
      for (int i = 0; i < N; ++i) {
        r[v][i] = fmaf(z[v][i] * rstd, w[i], r[v][i]);
        ss = fmaf(r[v][i], r[v][i], ss);
      }
      Pack<float, N>::store(res + (int64_t)g * N, r[v]);
    }
  }
  if (!p.out) return;
  rstd = p.w_out ? rsqrtf(block_sum(ss) / (float)p.D + p.eps) : 1.0f;
#pragma unroll
  for (int v = 0; v < VPT; ++v) {
    const int g = threadIdx.x + v * NORM_THREADS;
    if (g < groups) {
      if (p.w_out) {
        float w[N];
        Pack<T, N>::load(static_cast<const T*>(p.w_out) + (int64_t)g * N, w);
#pragma unroll
        for (int i = 0; i < N; ++i) r[v][i] *= rstd * w[i];
      }
      Pack<T, N>::store(static_cast<T*>(p.out) + row * p.D + (int64_t)g * N, r[v]);
    }
  }
}

struct EmbedParams {
  const int64_t* tokens;        // [B, L]
  const void *table, *pos;      // [V, D], [P, D]
  float* residual;              // [B, L, D] fp32
  void* out;                    // the same in T, or null
  const int32_t* offsets;
  int64_t V, P;
  int offset, L, D;
  float scale;
};

template <typename T, int N>
__global__ void __launch_bounds__(NORM_THREADS) stream_embed_kernel(const EmbedParams p) {
  using seq::Pack;
  const int64_t row = (int64_t)blockIdx.y * p.L + blockIdx.x;
  const int64_t tok = p.tokens[row], at = (int64_t)seq::position0(p.offsets, p.offset, blockIdx.y) + blockIdx.x;
  const bool known = tok >= 0 && tok < p.V, placed = at >= 0 && at < p.P;   // ids and positions outside a table add nothing
  const T* e = static_cast<const T*>(p.table) + (known ? tok : 0) * p.D;
  const T* q = static_cast<const T*>(p.pos) + (placed ? at : 0) * p.D;
  for (int g = threadIdx.x; g < p.D / N; g += NORM_THREADS) {
    float a[N], b[N];
    Pack<T, N>::load(e + (int64_t)g * N, a);
    Pack<T, N>::load(q + (int64_t)g * N, b);
#pragma unroll
    for (int i = 0; i < N; ++i) a[i] = fmaf(known ? a[i] : 0.f, p.scale, placed ? b[i] : 0.f);
    Pack<float, N>::store(p.residual + row * p.D + (int64_t)g * N, a);
    if (p.out) Pack<T, N>::store(static_cast<T*>(p.out) + row * p.D + (int64_t)g * N, a);
  }
}

struct NormGateParams {
  const void *x, *w, *gate;     // [M, D] (rows sx apart), [D], [M, D] (rows sg apart)
  void* out;                    // rows so apart
  int64_t sx, sg, so;
  int D;
  float eps;
};

template <typename T, int N, int VPT>
__global__ void __launch_bounds__(NORM_THREADS) norm_gate_kernel(const NormGateParams p) {
  using seq::Pack;
  const int64_t row = blockIdx.x;
  const int groups = p.D / N;
  const T *x = static_cast<const T*>(p.x) + row * p.sx, *gate = static_cast<const T*>(p.gate) + row * p.sg;
  float z[VPT][N], h[VPT][N];
  float ss = 0.f;
#pragma unroll
  for (int v = 0; v < VPT; ++v) {
    const int g = threadIdx.x + v * NORM_THREADS;
    if (g < groups) {
      Pack<T, N>::load(x + (int64_t)g * N, z[v]);
      Pack<T, N>::load(gate + (int64_t)g * N, h[v]);
#pragma unroll
      for (int i = 0; i < N; ++i) ss = fmaf(z[v][i], z[v][i], ss);
    }
  }
  const float rstd = rsqrtf(block_sum(ss) / (float)p.D + p.eps);
#pragma unroll
  for (int v = 0; v < VPT; ++v) {
    const int g = threadIdx.x + v * NORM_THREADS;
    if (g < groups) {
      float w[N];
      Pack<T, N>::load(static_cast<const T*>(p.w) + (int64_t)g * N, w);
#pragma unroll
      for (int i = 0; i < N; ++i) z[v][i] *= rstd * w[i] * seq::sigmoid_t<T>(h[v][i]);
      Pack<T, N>::store(static_cast<T*>(p.out) + row * p.so + (int64_t)g * N, z[v]);
    }
  }
}

struct TokenGateParams {
  const void *z, *table;        // [M, n] (rows sz apart); table rows of st elements, the slice starts at `column`
  const int64_t* tokens;        // [M]
  void* out;                    // [M, n] contiguous
  int64_t M, V, sz, st, column;
  int n;
};

template <typename T, int N>
__global__ void __launch_bounds__(256) token_gate_kernel(const TokenGateParams p) {
  using seq::Pack;
  const int per = p.n / N;
  const int64_t i = (int64_t)blockIdx.x * 256 + threadIdx.x;
  if (i >= p.M * per) return;
  const int64_t row = i / per;
  const int c = (int)(i - row * per) * N;
  const int64_t tok = p.tokens[row];
  const bool known = tok >= 0 && tok < p.V;
  float z[N], e[N];
  Pack<T, N>::load(static_cast<const T*>(p.z) + row * p.sz + c, z);
  Pack<T, N>::load(static_cast<const T*>(p.table) + (known ? tok : 0) * p.st + p.column + c, e);
#pragma unroll
  for (int k = 0; k < N; ++k) z[k] = known ? seq::gelu_tanh_t<T>(z[k]) * e[k] : 0.f;
  Pack<T, N>::store(static_cast<T*>(p.out) + row * p.n + c, z);
}

struct ActParams {
  const void *y, *gate;
  void* out;
  int64_t M, sy, sg, so;
  int F, act;
};

__device__ __forceinline__ float act_fn(float g, int act) {
  const float s = __fdividef(1.0f, 1.0f + __expf(-g));  // sigmoid
  return act == 0 ? g * s : s;                            // 0: silu, 1: sigmoid
}

// One row per block; thread t owns the 16-byte vectors t, t + 128, ... of the row (VPT of them): a
// warp's accesses are contiguous, all loads of a thread are issued before any arithmetic.
template <typename T, int VPT>
__global__ void __launch_bounds__(NORM_THREADS) gated_act_kernel(const ActParams p) {
  constexpr int N = V16<T>::N;
  const int nvec = p.F / N;
  const int64_t row = blockIdx.x;
  const T* y = static_cast<const T*>(p.y) + row * p.sy;
  const T* gate = static_cast<const T*>(p.gate) + row * p.sg;
  T* out = static_cast<T*>(p.out) + row * p.so;
  uint4 a[VPT], g[VPT];
#pragma unroll
  for (int v = 0; v < VPT; ++v) {
    const int c = threadIdx.x + v * NORM_THREADS;
    if (c < nvec) {
      a[v] = *reinterpret_cast<const uint4*>(y + c * N);
      g[v] = *reinterpret_cast<const uint4*>(gate + c * N);
    }
  }
#pragma unroll
  for (int v = 0; v < VPT; ++v) {
    const int c = threadIdx.x + v * NORM_THREADS;
    if (c < nvec) {
      float x[N], h[N];
      V16<T>::unpack(a[v], x);
      V16<T>::unpack(g[v], h);
#pragma unroll
      for (int e = 0; e < N; ++e) x[e] *= act_fn(h[e], p.act);
      V16<T>::store(out + c * N, x);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(NORM_THREADS) gated_act_scalar_kernel(const ActParams p) {
  const int64_t row = blockIdx.x;
  for (int c = threadIdx.x; c < p.F; c += NORM_THREADS) {
    const float g = to_float<T>(static_cast<const T*>(p.gate)[row * p.sg + c]);
    static_cast<T*>(p.out)[row * p.so + c] =
        from_float<T>(to_float<T>(static_cast<const T*>(p.y)[row * p.sy + c]) * act_fn(g, p.act));
  }
}

template <typename T>
int launch_stream_norm_t(const StreamParams& p, cudaStream_t stream) {
  const unsigned grid = (unsigned)p.M;
  const bool vec = p.D % 8 == 0 && aligned16(p.table) && aligned16(p.table_norm) && aligned16(p.branch) &&
                   aligned16(p.residual) && aligned16(p.w1) && aligned16(p.w2) && aligned16(p.out1) &&
                   aligned16(p.out2) && p.sb % 8 == 0;
  const int vpt = (p.D / (vec ? 8 : 1) + NORM_THREADS - 1) / NORM_THREADS;
  if (vec) {
    if (vpt <= 1) stream_norm_kernel<T, 8, 1><<<grid, NORM_THREADS, 0, stream>>>(p);
    else if (vpt <= 2) stream_norm_kernel<T, 8, 2><<<grid, NORM_THREADS, 0, stream>>>(p);
    else if (vpt <= 4) stream_norm_kernel<T, 8, 4><<<grid, NORM_THREADS, 0, stream>>>(p);
    else if (vpt <= 8) stream_norm_kernel<T, 8, 8><<<grid, NORM_THREADS, 0, stream>>>(p);
    else return BASED_ERR_SHAPE;   // rows up to 8192 wide
  } else {
    if (vpt <= 4) stream_norm_kernel<T, 1, 4><<<grid, NORM_THREADS, 0, stream>>>(p);
    else if (vpt <= 32) stream_norm_kernel<T, 1, 32><<<grid, NORM_THREADS, 0, stream>>>(p);
    else return BASED_ERR_SHAPE;   // rows up to 4096 wide
  }
  return (int)cudaGetLastError();
}

template <typename T>
int launch_post_norm_t(const PostNormParams& p, int64_t M, cudaStream_t stream) {
  const bool vec = p.D % 8 == 0 && p.sb % 8 == 0 && aligned16(p.branch) && aligned16(p.w) && aligned16(p.residual) &&
                   aligned16(p.w_out) && aligned16(p.out);
  const int vpt = (p.D / (vec ? 8 : 1) + NORM_THREADS - 1) / NORM_THREADS;
  const unsigned grid = (unsigned)M;
  if (vec) {
    if (vpt <= 1) stream_post_norm_kernel<T, 8, 1><<<grid, NORM_THREADS, 0, stream>>>(p);
    else if (vpt <= 2) stream_post_norm_kernel<T, 8, 2><<<grid, NORM_THREADS, 0, stream>>>(p);
    else if (vpt <= 4) stream_post_norm_kernel<T, 8, 4><<<grid, NORM_THREADS, 0, stream>>>(p);
    else if (vpt <= 8) stream_post_norm_kernel<T, 8, 8><<<grid, NORM_THREADS, 0, stream>>>(p);
    else return BASED_ERR_SHAPE;   // rows up to 8192 wide
  } else {
    if (vpt <= 4) stream_post_norm_kernel<T, 1, 4><<<grid, NORM_THREADS, 0, stream>>>(p);
    else if (vpt <= 32) stream_post_norm_kernel<T, 1, 32><<<grid, NORM_THREADS, 0, stream>>>(p);
    else return BASED_ERR_SHAPE;   // rows up to 4096 wide
  }
  return (int)cudaGetLastError();
}

template <typename T>
int launch_embed_t(const EmbedParams& p, int B, cudaStream_t stream) {
  const dim3 grid((unsigned)p.L, (unsigned)B);
  if (p.D % 8 == 0 && aligned16(p.table) && aligned16(p.pos) && aligned16(p.residual) && aligned16(p.out))
    stream_embed_kernel<T, 8><<<grid, NORM_THREADS, 0, stream>>>(p);
  else
    stream_embed_kernel<T, 1><<<grid, NORM_THREADS, 0, stream>>>(p);
  return (int)cudaGetLastError();
}

template <typename T>
int launch_norm_gate_t(const NormGateParams& p, int64_t M, cudaStream_t stream) {
  const bool vec = p.D % 8 == 0 && p.sx % 8 == 0 && p.sg % 8 == 0 && p.so % 8 == 0 && aligned16(p.x) && aligned16(p.w) &&
                   aligned16(p.gate) && aligned16(p.out);
  const int vpt = (p.D / (vec ? 8 : 1) + NORM_THREADS - 1) / NORM_THREADS;
  const unsigned grid = (unsigned)M;
  if (vec) {
    if (vpt <= 1) norm_gate_kernel<T, 8, 1><<<grid, NORM_THREADS, 0, stream>>>(p);
    else if (vpt <= 2) norm_gate_kernel<T, 8, 2><<<grid, NORM_THREADS, 0, stream>>>(p);
    else if (vpt <= 4) norm_gate_kernel<T, 8, 4><<<grid, NORM_THREADS, 0, stream>>>(p);
    else if (vpt <= 8) norm_gate_kernel<T, 8, 8><<<grid, NORM_THREADS, 0, stream>>>(p);
    else return BASED_ERR_SHAPE;
  } else {
    if (vpt <= 4) norm_gate_kernel<T, 1, 4><<<grid, NORM_THREADS, 0, stream>>>(p);
    else if (vpt <= 32) norm_gate_kernel<T, 1, 32><<<grid, NORM_THREADS, 0, stream>>>(p);
    else return BASED_ERR_SHAPE;
  }
  return (int)cudaGetLastError();
}

template <typename T>
int launch_token_gate_t(const TokenGateParams& p, cudaStream_t stream) {
  const bool vec = p.n % 8 == 0 && p.sz % 8 == 0 && p.st % 8 == 0 && p.column % 8 == 0 && aligned16(p.z) && aligned16(p.table) &&
                   aligned16(p.out);
  const int64_t work = p.M * (p.n / (vec ? 8 : 1)), blocks = (work + 255) / 256;
  if (blocks > 2147483647LL) return BASED_ERR_TOO_LARGE;
  if (vec) token_gate_kernel<T, 8><<<(unsigned)blocks, 256, 0, stream>>>(p);
  else token_gate_kernel<T, 1><<<(unsigned)blocks, 256, 0, stream>>>(p);
  return (int)cudaGetLastError();
}

}  // namespace

int launch_stream_post_norm(const void* branch, int64_t sb, const void* w, float* residual, const void* w_out, void* out,
                            int64_t M, int D, float eps, int io_dtype, cudaStream_t stream) {
  if (M > 2147483647LL) return BASED_ERR_TOO_LARGE;
  const PostNormParams p{branch, w, residual, w_out, out, sb, D, eps};
  return io_dtype == BASED_BF16 ? launch_post_norm_t<__nv_bfloat16>(p, M, stream) : launch_post_norm_t<float>(p, M, stream);
}

int launch_stream_embed(const int64_t* tokens, const void* table, int64_t V, float scale, const void* pos, int64_t P,
                        float* residual, void* out, int B, int L, int D, const int32_t* offsets, int offset, int io_dtype,
                        cudaStream_t stream) {
  if (B > 65535) return BASED_ERR_TOO_LARGE;
  const EmbedParams p{tokens, table, pos, residual, out, offsets, V, P, offset, L, D, scale};
  return io_dtype == BASED_BF16 ? launch_embed_t<__nv_bfloat16>(p, B, stream) : launch_embed_t<float>(p, B, stream);
}

int launch_norm_gate(const void* x, int64_t sx, const void* w, const void* gate, int64_t sg, void* out, int64_t so, int64_t M,
                     int D, float eps, int io_dtype, cudaStream_t stream) {
  if (M > 2147483647LL) return BASED_ERR_TOO_LARGE;
  const NormGateParams p{x, w, gate, out, sx, sg, so, D, eps};
  return io_dtype == BASED_BF16 ? launch_norm_gate_t<__nv_bfloat16>(p, M, stream) : launch_norm_gate_t<float>(p, M, stream);
}

int launch_token_gate(const void* z, int64_t sz, const int64_t* tokens, const void* table, int64_t V, int64_t st,
                      int64_t column, void* out, int64_t M, int n, int io_dtype, cudaStream_t stream) {
  const TokenGateParams p{z, table, tokens, out, M, V, sz, st, column, n};
  return io_dtype == BASED_BF16 ? launch_token_gate_t<__nv_bfloat16>(p, stream) : launch_token_gate_t<float>(p, stream);
}

int launch_stream_norm(const int64_t* tokens, const void* table, const void* table_norm, int64_t V, const void* branch,
                       int64_t branch_stride, float mult, float* residual, const void* w1, const void* w2, void* out1,
                       void* out2, int64_t M, int D, float eps, int io_dtype, cudaStream_t stream) {
  if (M > 2147483647LL) return BASED_ERR_TOO_LARGE;
  const StreamParams p{tokens, table, table_norm, branch, residual, w1, w2, out1, out2, M, V, branch_stride, D, mult, eps};
  return io_dtype == BASED_BF16 ? launch_stream_norm_t<__nv_bfloat16>(p, stream) : launch_stream_norm_t<float>(p, stream);
}

int launch_add_rmsnorm(const void* x, const void* residual, const void* weight, const void* bias, void* out,
                       void* residual_out, int64_t M, int D, int64_t sx, int64_t sr, int64_t so, int64_t sro, float eps,
                       int io_dtype, int res_dtype, int w_dtype, int round_input, cudaStream_t stream) {
  if (D % 8 != 0 || D > 8 * NORM_THREADS * 8) return BASED_ERR_SHAPE;
  if (!aligned16(x) || !aligned16(out) || !aligned16(weight) || (residual && !aligned16(residual)) ||
      (residual_out && !aligned16(residual_out)) || (bias && !aligned16(bias)))
    return BASED_ERR_ALIGN;
  if (sx % 8 || so % 8 || (residual && sr % 8) || (residual_out && sro % 8)) return BASED_ERR_ALIGN;
  if (M > 2147483647LL) return BASED_ERR_TOO_LARGE;
  NormParams p{x, residual, weight, bias, out, residual_out, M, sx, sr, so, sro, D,
               io_dtype == BASED_BF16, res_dtype == BASED_BF16, w_dtype == BASED_BF16, round_input != 0, eps};
  const int groups = D / 8, vpt = (groups + NORM_THREADS - 1) / NORM_THREADS;
  const unsigned grid = (unsigned)M;
  if (vpt <= 1) add_rmsnorm_kernel<1><<<grid, NORM_THREADS, 0, stream>>>(p);
  else if (vpt <= 2) add_rmsnorm_kernel<2><<<grid, NORM_THREADS, 0, stream>>>(p);
  else if (vpt <= 4) add_rmsnorm_kernel<4><<<grid, NORM_THREADS, 0, stream>>>(p);
  else add_rmsnorm_kernel<8><<<grid, NORM_THREADS, 0, stream>>>(p);
  return (int)cudaGetLastError();
}

int launch_rmsnorm(const void* x, const void* w, void* out, int64_t M, int D, int64_t sx, int64_t so, float eps,
                   int io_dtype, cudaStream_t stream) {
  const int rc = launch_add_rmsnorm(x, nullptr, w, nullptr, out, nullptr, M, D, sx, 0, so, 0, eps, io_dtype, io_dtype,
                                    io_dtype, 0, stream);
  if (rc != BASED_ERR_SHAPE && rc != BASED_ERR_ALIGN) return rc;
  if (io_dtype == BASED_BF16)
    rmsnorm_scalar_kernel<__nv_bfloat16><<<(unsigned)M, NORM_THREADS, 0, stream>>>(
        static_cast<const __nv_bfloat16*>(x), static_cast<const __nv_bfloat16*>(w), static_cast<__nv_bfloat16*>(out), D, sx,
        so, eps);
  else
    rmsnorm_scalar_kernel<float><<<(unsigned)M, NORM_THREADS, 0, stream>>>(
        static_cast<const float*>(x), static_cast<const float*>(w), static_cast<float*>(out), D, sx, so, eps);
  return (int)cudaGetLastError();
}

int launch_gated_act(const void* y, const void* gate, void* out, int64_t M, int F, int64_t sy, int64_t sg, int64_t so,
                     int act, int io_dtype, cudaStream_t stream) {
  const int N = io_dtype == BASED_BF16 ? 8 : 4;
  if (M > 2147483647LL) return BASED_ERR_TOO_LARGE;
  const int nvec = F / N, vpt = (nvec + NORM_THREADS - 1) / NORM_THREADS;
  ActParams p{y, gate, out, M, sy, sg, so, F, act};
  const unsigned grid = (unsigned)M;
  if (F % N != 0 || vpt > 16 || !aligned16(y) || !aligned16(gate) || !aligned16(out) || sy % N || sg % N || so % N) {
    if (io_dtype == BASED_BF16) gated_act_scalar_kernel<__nv_bfloat16><<<grid, NORM_THREADS, 0, stream>>>(p);
    else gated_act_scalar_kernel<float><<<grid, NORM_THREADS, 0, stream>>>(p);
    return (int)cudaGetLastError();
  }
#define BASED_LAUNCH_ACT(T)                                                                      \
  do {                                                                                           \
    if (vpt <= 1) gated_act_kernel<T, 1><<<grid, NORM_THREADS, 0, stream>>>(p);                  \
    else if (vpt <= 2) gated_act_kernel<T, 2><<<grid, NORM_THREADS, 0, stream>>>(p);             \
    else if (vpt <= 4) gated_act_kernel<T, 4><<<grid, NORM_THREADS, 0, stream>>>(p);             \
    else if (vpt <= 8) gated_act_kernel<T, 8><<<grid, NORM_THREADS, 0, stream>>>(p);             \
    else gated_act_kernel<T, 16><<<grid, NORM_THREADS, 0, stream>>>(p);                          \
  } while (0)
  if (io_dtype == BASED_BF16) BASED_LAUNCH_ACT(__nv_bfloat16);
  else BASED_LAUNCH_ACT(float);
#undef BASED_LAUNCH_ACT
  return (int)cudaGetLastError();
}

}  // namespace based
