// Helpers shared by the kernels of the stateful mixers (short convolution, gated delta rule, gated linear recurrent
// unit, latent attention): vector access in the activations' dtype and the scalar functions the recurrences use.
#pragma once

#include "common.cuh"

namespace based {
namespace seq {

// N consecutive values of T <-> floats; one 16-byte access when N * sizeof(T) == 16, element-wise for N == 1.
template <typename T, int N>
struct Pack;
template <typename T>
struct Pack<T, 1> {
  static __device__ __forceinline__ void load(const T* p, float (&x)[1]) { x[0] = to_float<T>(*p); }
  static __device__ __forceinline__ void store(T* p, const float (&x)[1]) { *p = from_float<T>(x[0]); }
};
template <>
struct Pack<float, 4> {
  static __device__ __forceinline__ void load(const float* p, float (&x)[4]) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    x[0] = v.x; x[1] = v.y; x[2] = v.z; x[3] = v.w;
  }
  static __device__ __forceinline__ void store(float* p, const float (&x)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1], x[2], x[3]);
  }
};
template <>
struct Pack<float, 8> {  // two accesses
  static __device__ __forceinline__ void load(const float* p, float (&x)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    x[0] = a.x; x[1] = a.y; x[2] = a.z; x[3] = a.w; x[4] = b.x; x[5] = b.y; x[6] = b.z; x[7] = b.w;
  }
  static __device__ __forceinline__ void store(float* p, const float (&x)[8]) {
    *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1], x[2], x[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(x[4], x[5], x[6], x[7]);
  }
};
__device__ __forceinline__ uint32_t bf16x2_bits(float lo, float hi) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&h);
}
__device__ __forceinline__ float bf16_lo(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float bf16_hi(uint32_t w) { return __uint_as_float(w & 0xFFFF0000u); }
template <>
struct Pack<__nv_bfloat16, 4> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&x)[4]) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    x[0] = bf16_lo(v.x); x[1] = bf16_hi(v.x); x[2] = bf16_lo(v.y); x[3] = bf16_hi(v.y);
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&x)[4]) {
    *reinterpret_cast<uint2*>(p) = make_uint2(bf16x2_bits(x[0], x[1]), bf16x2_bits(x[2], x[3]));
  }
};
template <>
struct Pack<__nv_bfloat16, 8> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&x)[8]) {
    const uint4 v = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) { x[2 * i] = bf16_lo(w[i]); x[2 * i + 1] = bf16_hi(w[i]); }
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&x)[8]) {
    *reinterpret_cast<uint4*>(p) = make_uint4(bf16x2_bits(x[0], x[1]), bf16x2_bits(x[2], x[3]), bf16x2_bits(x[4], x[5]),
                                             bf16x2_bits(x[6], x[7]));
  }
};
// widest pack of T with one 16-byte access
template <typename T> struct Wide { static constexpr int N = 16 / sizeof(T); };

// a vector load of N elements of T at base is allowed for every multiple-of-N index and these strides
template <typename T>
inline bool can_pack(int n, const void* base, std::initializer_list<int64_t> strides) {
  if (base && (reinterpret_cast<uintptr_t>(base) % (n * sizeof(T)))) return false;
  for (int64_t s : strides)
    if (s % n) return false;
  return true;
}

// Activation functions of the activations' dtype T: hardware approximations where the result is rounded to bf16,
// the accurate library functions in fp32.
template <typename T> __device__ __forceinline__ float sigmoid_t(float x) { return __fdividef(1.0f, 1.0f + __expf(-x)); }
template <> __device__ __forceinline__ float sigmoid_t<float>(float x) { return 1.0f / (1.0f + expf(-x)); }
template <typename T> __device__ __forceinline__ float silu_t(float x) { return x * sigmoid_t<T>(x); }

// gelu with the tanh form: 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))) = z * sigmoid(2 * the argument)
template <typename T>
__device__ __forceinline__ float gelu_tanh_t(float z) {
  const float a = 0.7978845608028654f * fmaf(0.044715f * z * z, z, z);
  return z * sigmoid_t<T>(2.0f * a);
}

// Functions of the recurrences: always accurate fp32, whatever the activations' dtype.
__device__ __forceinline__ float sigmoid_acc(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float softplus_acc(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }

// First position of a call's tokens for batch row b: the device array when there is one, else the scalar.
__device__ __forceinline__ int position0(const int32_t* offsets, int offset, int b) { return offsets ? offsets[b] : offset; }

}  // namespace seq
}  // namespace based
