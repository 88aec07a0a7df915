// Element types of the kernels that are compiled for several of them: conversions, 16-byte chunks, dot products.
#pragma once
#include <cuda_bf16.h>

#include "common.cuh"

namespace djv {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__half v) { return __half2float(v); }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }

template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ __half from_f<__half>(float v) { return __float2half_rn(v); }
template <>
__device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }

// Number of elements in a 16-byte chunk.
template <typename T>
struct Chunk {
  static constexpr int N = 16 / (int)sizeof(T);
};

// bf16 pair packed in a word -> two floats (a bf16 is the upper half of the float with the same value)
__device__ __forceinline__ float2 b2f(uint32_t u) {
  return make_float2(__uint_as_float(u << 16), __uint_as_float(u & 0xffff0000u));
}

// unpacks a 16-byte chunk into Chunk<T>::N floats
template <typename T>
__device__ __forceinline__ void unpack_chunk(const uint4 &v, float *f);
template <>
__device__ __forceinline__ void unpack_chunk<float>(const uint4 &v, float *f) {
  f[0] = __uint_as_float(v.x);
  f[1] = __uint_as_float(v.y);
  f[2] = __uint_as_float(v.z);
  f[3] = __uint_as_float(v.w);
}
template <>
__device__ __forceinline__ void unpack_chunk<__half>(const uint4 &v, float *f) {
  const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 t = h2f(w[i]);
    f[2 * i] = t.x;
    f[2 * i + 1] = t.y;
  }
}
template <>
__device__ __forceinline__ void unpack_chunk<bf16>(const uint4 &v, float *f) {
  const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 t = b2f(w[i]);
    f[2 * i] = t.x;
    f[2 * i + 1] = t.y;
  }
}

// dot product of two 16-byte chunks, fp32 accumulate in element order
template <typename T>
__device__ __forceinline__ float dot_chunk(const uint4 &a, const uint4 &b, float acc) {
  float x[Chunk<T>::N], y[Chunk<T>::N];
  unpack_chunk<T>(a, x);
  unpack_chunk<T>(b, y);
#pragma unroll
  for (int i = 0; i < Chunk<T>::N; ++i) acc = fmaf(x[i], y[i], acc);
  return acc;
}

// two floats -> packed bf16 pair (lo in the lower half)
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t *>(&h);
}

inline size_t dtype_bytes(int dtype) { return dtype == DJV_DTYPE_F32 ? 4 : 2; }

// sigmoid(z) written so that neither tail overflows
__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
// log(sigmoid(z)) = min(z, 0) - log(1 + exp(-|z|))
__device__ __forceinline__ float log_sigmoid_f(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

}  // namespace djv
