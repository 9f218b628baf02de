// Element access for kernels that run in any of the three activation types (fp16, bf16, fp32): one scalar at a time,
// arithmetic in fp32.  The 16-byte helpers of common.cuh cover the 16-bit types only.
#pragma once
#include "common.cuh"

namespace blitz {

template <typename T>
__device__ __forceinline__ float ldf(const T* p) { return to_f<T>(*p); }
template <>
__device__ __forceinline__ float ldf<float>(const float* p) { return *p; }

template <typename T>
__device__ __forceinline__ void stf(T* p, float v);
template <>
__device__ __forceinline__ void stf<float>(float* p, float v) { *p = v; }
template <>
__device__ __forceinline__ void stf<__nv_bfloat16>(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
template <>
__device__ __forceinline__ void stf<__half>(__half* p, float v) { *p = __float2half_rn(v); }

// Two neighbouring elements (the address is a multiple of two elements).
template <typename T>
__device__ __forceinline__ float2 ldf2(const T* p) { return cvt2<T>(*reinterpret_cast<const uint32_t*>(p)); }
template <>
__device__ __forceinline__ float2 ldf2<float>(const float* p) { return *reinterpret_cast<const float2*>(p); }
template <typename T>
__device__ __forceinline__ void stf2(T* p, float a, float b) { *reinterpret_cast<uint32_t*>(p) = pk2<T>(a, b); }
template <>
__device__ __forceinline__ void stf2<float>(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }

// Four neighbouring elements (the address is a multiple of four elements).
template <typename T>
__device__ __forceinline__ float4 ldf4(const T* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = cvt2<T>(u.x), b = cvt2<T>(u.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
template <>
__device__ __forceinline__ float4 ldf4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <typename T>
__device__ __forceinline__ void stf4(T* p, const float4& v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pk2<T>(v.x, v.y), pk2<T>(v.z, v.w));
}
template <>
__device__ __forceinline__ void stf4<float>(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }

// Eight neighbouring elements (the address is a multiple of eight elements).
template <typename T>
__device__ __forceinline__ void ldf8(const T* p, float (&f)[8]) { unpack8<T>(*reinterpret_cast<const uint4*>(p), f); }
template <>
__device__ __forceinline__ void ldf8<float>(const float* p, float (&f)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}

template <typename T>
__device__ __forceinline__ void stf8(T* p, const float (&f)[8]) { *reinterpret_cast<uint4*>(p) = pack8<T>(f); }
template <>
__device__ __forceinline__ void stf8<float>(float* p, const float (&f)[8]) {
  reinterpret_cast<float4*>(p)[0] = make_float4(f[0], f[1], f[2], f[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(f[4], f[5], f[6], f[7]);
}

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float silu_acc(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// log(sigmoid(z)), exact for large |z|
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float gelu_tanh_f(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

// Sequence row that token t belongs to: the r with tok_indptr[r] <= t < tok_indptr[r + 1].
__device__ __forceinline__ int row_of_token(const int32_t* __restrict__ tok_indptr, int rows, int t) {
  int lo = 0, hi = rows - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (tok_indptr[mid] <= t) lo = mid; else hi = mid - 1;
  }
  return lo;
}

#define BLITZ_DISPATCH_DTYPE3(dtype, ...)           \
  do {                                              \
    if ((dtype) == 2) {                             \
      using T = float;                              \
      __VA_ARGS__;                                  \
    } else if ((dtype) == 1) {                      \
      using T = __nv_bfloat16;                      \
      __VA_ARGS__;                                  \
    } else {                                        \
      using T = __half;                             \
      __VA_ARGS__;                                  \
    }                                               \
  } while (0)

}  // namespace blitz
