// Depthwise causal convolution over time with a carried state, for tokens that continue a sequence at any position:
//   y[b, l, c] = act( sum_j w[c, j] x[b, l - (taps-1) + j, c] (+ bias[c]) ),  act = identity or silu
// Inputs before this call's first token come from a ring: the input of position p sits in slot p mod taps of
// ring [B, taps, C]; positions before 0 are zero.  A step at position p writes the one slot that none of its readers
// look at (they need positions p-1 .. p-taps+1), so a single-token call reads and updates the ring in one launch, and
// several blocks may write the same slot with the same value.  Longer calls update the ring in a second launch.
//
// HBM-bound: one read of x and one write of y.  A thread owns TT consecutive tokens of one 16-byte vector of
// channels, so the taps-1 rows it shares with its neighbour are the only re-reads (L1 / L2 hits).
#include <initializer_list>

#include "seq_common.cuh"

namespace based {
namespace {

using namespace seq;

struct ConvP {
  const void *x, *w, *bias;
  void *y, *ring;
  const int32_t* offsets;
  int offset, B, L, C, taps, silu;
  Strides2 sx, sy;  // .b batch, .h token
};

constexpr int kThreads = 128;

template <typename T>
__device__ __forceinline__ void unpack16(const uint4& v, float (&x)[Wide<T>::N]) {
  const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    if constexpr (sizeof(T) == 2) { x[2 * i] = bf16_lo(w[i]); x[2 * i + 1] = bf16_hi(w[i]); }
    else x[i] = __uint_as_float(w[i]);
  }
}

template <typename T, int N, int TT>
__global__ void __launch_bounds__(kThreads) short_conv_kernel(const ConvP p) {
  const int c = (blockIdx.x * kThreads + threadIdx.x) * N;
  const int l0 = blockIdx.y * TT, b = blockIdx.z;
  if (c >= p.C) return;
  const int taps = p.taps;
  const int pos0 = position0(p.offsets, p.offset, b);
  const T* x = static_cast<const T*>(p.x) + b * p.sx.b + c;
  T* ring = p.ring ? static_cast<T*>(p.ring) + (int64_t)b * taps * p.C + c : nullptr;
  auto fetch = [&](int l, float (&v)[N]) {  // input of token l of this call (l < 0: earlier tokens of the sequence)
    if (l >= 0) {
      Pack<T, N>::load(x + (int64_t)l * p.sx.h, v);
    } else if (ring && pos0 + l >= 0) {
      Pack<T, N>::load(ring + (int64_t)((pos0 + l) % taps) * p.C, v);
    } else {
#pragma unroll
      for (int i = 0; i < N; ++i) v[i] = 0.f;
    }
  };
  float acc[TT][N];
#pragma unroll
  for (int t = 0; t < TT; ++t)
#pragma unroll
    for (int i = 0; i < N; ++i) acc[t][i] = p.bias ? to_float<T>(static_cast<const T*>(p.bias)[c + i]) : 0.f;
  const T* w = static_cast<const T*>(p.w) + (int64_t)c * taps;
  for (int t = 0; t < TT; ++t) {
    if (l0 + t >= p.L) break;
    for (int j = 0; j < taps; ++j) {
      float v[N];
      fetch(l0 + t - (taps - 1) + j, v);
#pragma unroll
      for (int i = 0; i < N; ++i) acc[t][i] = fmaf(to_float<T>(w[i * taps + j]), v[i], acc[t][i]);
    }
  }
  T* y = static_cast<T*>(p.y) + b * p.sy.b + c;
#pragma unroll
  for (int t = 0; t < TT; ++t) {
    if (l0 + t >= p.L) break;
    if (p.silu) {
#pragma unroll
      for (int i = 0; i < N; ++i) acc[t][i] = silu_t<T>(acc[t][i]);
    }
    Pack<T, N>::store(y + (int64_t)(l0 + t) * p.sy.h, acc[t]);
  }
  if (p.L == 1 && ring) {  // single-token call: the slot nobody reads
    float v[N];
    Pack<T, N>::load(x, v);
    Pack<T, N>::store(ring + (int64_t)(pos0 % taps) * p.C, v);
  }
}

// The same for 16-byte vectors of channels and a compile-time number of taps: rows stay packed in registers until they
// are used, so that a thread's loads are all in flight together, and the taps of its channels are TAPS 16-byte loads.
template <typename T, int TT, int TAPS>
__global__ void __launch_bounds__(kThreads, 5) short_conv_vec_kernel(const ConvP p) {
  constexpr int N = Wide<T>::N;
  const int c = (blockIdx.x * kThreads + threadIdx.x) * N;
  const int l0 = blockIdx.y * TT, b = blockIdx.z;
  if (c >= p.C) return;
  const int pos0 = position0(p.offsets, p.offset, b);
  const T* x = static_cast<const T*>(p.x) + b * p.sx.b + c;
  T* ring = p.ring ? static_cast<T*>(p.ring) + (int64_t)b * TAPS * p.C + c : nullptr;
  uint4 rows[TT + TAPS - 1];
#pragma unroll
  for (int r = 0; r < TT + TAPS - 1; ++r) {
    const int l = l0 + r - (TAPS - 1);
    rows[r] = make_uint4(0, 0, 0, 0);
    if (l >= 0) {
      if (l < p.L) rows[r] = *reinterpret_cast<const uint4*>(x + (int64_t)l * p.sx.h);
    } else if (ring && pos0 + l >= 0) {
      rows[r] = *reinterpret_cast<const uint4*>(ring + (int64_t)((pos0 + l) % TAPS) * p.C);
    }
  }
  float w[N][TAPS], bias[N], win[TAPS][N];
  {
    float flat[N * TAPS];
    const uint4* src = reinterpret_cast<const uint4*>(static_cast<const T*>(p.w) + (int64_t)c * TAPS);
#pragma unroll
    for (int q = 0; q < TAPS; ++q) {
      float v[N];
      unpack16<T>(__ldg(src + q), v);
#pragma unroll
      for (int i = 0; i < N; ++i) flat[q * N + i] = v[i];
    }
#pragma unroll
    for (int i = 0; i < N; ++i)
#pragma unroll
      for (int j = 0; j < TAPS; ++j) w[i][j] = flat[i * TAPS + j];
  }
#pragma unroll
  for (int i = 0; i < N; ++i) bias[i] = 0.f;
  if (p.bias) Pack<T, N>::load(static_cast<const T*>(p.bias) + c, bias);
#pragma unroll
  for (int r = 0; r < TAPS - 1; ++r) unpack16<T>(rows[r], win[r]);
  T* y = static_cast<T*>(p.y) + b * p.sy.b + c;
#pragma unroll
  for (int t = 0; t < TT; ++t) {
    unpack16<T>(rows[t + TAPS - 1], win[(t + TAPS - 1) % TAPS]);
    if (l0 + t < p.L) {
      float acc[N];
#pragma unroll
      for (int i = 0; i < N; ++i) {
        acc[i] = bias[i];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) acc[i] = fmaf(w[i][j], win[(t + j) % TAPS][i], acc[i]);
        if (p.silu) acc[i] = silu_t<T>(acc[i]);
      }
      Pack<T, N>::store(y + (int64_t)(l0 + t) * p.sy.h, acc);
    }
  }
  if (p.L == 1 && ring) *reinterpret_cast<uint4*>(ring + (int64_t)(pos0 % TAPS) * p.C) = rows[TAPS - 1];
}

// the last min(L, taps) inputs of the call into their slots
template <typename T>
__global__ void __launch_bounds__(kThreads) ring_update_kernel(const ConvP p) {
  const int c = blockIdx.x * kThreads + threadIdx.x, b = blockIdx.z;
  if (c >= p.C) return;
  const int pos0 = position0(p.offsets, p.offset, b);
  const int l = p.L - 1 - (int)blockIdx.y;
  if (l < 0) return;
  static_cast<T*>(p.ring)[((int64_t)b * p.taps + (pos0 + l) % p.taps) * p.C + c] =
      static_cast<const T*>(p.x)[b * p.sx.b + (int64_t)l * p.sx.h + c];
}

template <typename T, int TT>
bool launch_vec(const ConvP& p, cudaStream_t st) {
  constexpr int N = Wide<T>::N;
  const dim3 grid((p.C / N + kThreads - 1) / kThreads, (p.L + TT - 1) / TT, p.B);
  switch (p.taps) {
    case 2: short_conv_vec_kernel<T, TT, 2><<<grid, kThreads, 0, st>>>(p); return true;
    case 3: short_conv_vec_kernel<T, TT, 3><<<grid, kThreads, 0, st>>>(p); return true;
    case 4: short_conv_vec_kernel<T, TT, 4><<<grid, kThreads, 0, st>>>(p); return true;
    default: return false;
  }
}

template <typename T, int N, int TT>
void launch_taps(const ConvP& p, cudaStream_t st) {
  const dim3 grid((p.C / N + kThreads - 1) / kThreads, (p.L + TT - 1) / TT, p.B);
  short_conv_kernel<T, N, TT><<<grid, kThreads, 0, st>>>(p);
}

template <typename T>
int launch_t(const ConvP& p, cudaStream_t st) {
  constexpr int N = Wide<T>::N;
  const bool vec = p.C % N == 0 && can_pack<T>(N, p.x, {p.sx.b, p.sx.h}) && can_pack<T>(N, p.y, {p.sy.b, p.sy.h}) &&
                   can_pack<T>(N, p.ring, {});
  const int tt = p.L == 1 ? 1 : 4;
  if ((p.L + tt - 1) / tt > 65535 || p.B > 65535) return BASED_ERR_TOO_LARGE;
  if (vec && aligned16(p.w) && aligned16(p.bias) && (p.L == 1 ? launch_vec<T, 1>(p, st) : launch_vec<T, 4>(p, st))) {
  } else if (vec) {
    if (p.L == 1) launch_taps<T, N, 1>(p, st);
    else launch_taps<T, N, 4>(p, st);
  } else {
    if (p.L == 1) launch_taps<T, 1, 1>(p, st);
    else launch_taps<T, 1, 4>(p, st);
  }
  if (p.ring && p.L > 1)
    ring_update_kernel<T><<<dim3((p.C + kThreads - 1) / kThreads, p.L < p.taps ? p.L : p.taps, p.B), kThreads, 0, st>>>(p);
  return (int)cudaGetLastError();
}

}  // namespace

int launch_short_conv(const void* x, void* y, void* ring, const void* w, const void* bias, int B, int L, int C, int taps,
                      Strides2 sx, Strides2 sy, const int32_t* offsets, int offset, int silu, int io_dtype,
                      cudaStream_t stream) {
  const ConvP p{x, w, bias, y, ring, offsets, offset, B, L, C, taps, silu, sx, sy};
  return io_dtype == BASED_BF16 ? launch_t<__nv_bfloat16>(p, stream) : launch_t<float>(p, stream);
}

}  // namespace based
