// Shared device helpers for the memory-bound kernels: 16-byte vector views of
// 16-bit element types, warp/block reductions.
#pragma once
#include <cuda_runtime.h>
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <stdint.h>
#include <type_traits>
#include "status.h"

namespace blitz {

template <typename T>
struct Vec8 {  // eight 16-bit elements = 16 bytes
  uint4 raw;
};

template <typename T>
__device__ __forceinline__ float2 cvt2(uint32_t u);
template <>
__device__ __forceinline__ float2 cvt2<__nv_bfloat16>(uint32_t u) {
  return __bfloat1622float2(*reinterpret_cast<__nv_bfloat162*>(&u));
}
template <>
__device__ __forceinline__ float2 cvt2<__half>(uint32_t u) {
  return __half22float2(*reinterpret_cast<__half2*>(&u));
}
template <typename T>
__device__ __forceinline__ uint32_t pk2(float a, float b);
template <>
__device__ __forceinline__ uint32_t pk2<__nv_bfloat16>(float a, float b) {
  __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&v);
}
template <>
__device__ __forceinline__ uint32_t pk2<__half>(float a, float b) {
  __half2 v = __floats2half2_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&v);
}

template <typename T>
__device__ __forceinline__ void unpack8(const uint4& v, float (&f)[8]) {
  float2 a = cvt2<T>(v.x), b = cvt2<T>(v.y), c = cvt2<T>(v.z), d = cvt2<T>(v.w);
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y; f[4] = c.x; f[5] = c.y; f[6] = d.x; f[7] = d.y;
}
template <typename T>
__device__ __forceinline__ uint4 pack8(const float (&f)[8]) {
  return make_uint4(pk2<T>(f[0], f[1]), pk2<T>(f[2], f[3]), pk2<T>(f[4], f[5]), pk2<T>(f[6], f[7]));
}

template <typename T>
__device__ __forceinline__ float to_f(T v);
template <>
__device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <>
__device__ __forceinline__ float to_f<__half>(__half v) { return __half2float(v); }

// Streaming 16-byte load: read-only path, no L1 allocation.
__device__ __forceinline__ uint4 ld_nc16(const void* p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];"
               : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w)
               : "l"(p));
  return v;
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}

// Block-wide sum; `red` must hold 33 floats.  Every thread gets the result.
__device__ __forceinline__ float block_sum(float v, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  if (warp == 0) {
    float x = lane < nw ? red[lane] : 0.f;
    x = warp_sum(x);
    if (lane == 0) red[32] = x;
  }
  __syncthreads();
  return red[32];
}
// The same for two numbers with a single barrier; `red` must not be in use by anything before that barrier.
__device__ __forceinline__ float2 block_sum2(float a, float b, float2 (&red)[32]) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  a = warp_sum(a);
  b = warp_sum(b);
  if (lane == 0) red[warp] = make_float2(a, b);
  __syncthreads();
  float2 s = red[0];
  for (int w = 1; w < nw; ++w) {
    s.x += red[w].x;
    s.y += red[w].y;
  }
  return s;
}
__device__ __forceinline__ float block_max(float v, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  v = warp_max(v);
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  if (warp == 0) {
    float x = lane < nw ? red[lane] : -INFINITY;
    x = warp_max(x);
    if (lane == 0) red[32] = x;
  }
  __syncthreads();
  return red[32];
}

#define BLITZ_DISPATCH_DTYPE(dtype, ...)            \
  do {                                              \
    if ((dtype) == 1) {                             \
      using T = __nv_bfloat16;                      \
      __VA_ARGS__;                                  \
    } else {                                        \
      using T = __half;                             \
      __VA_ARGS__;                                  \
    }                                               \
  } while (0)

}  // namespace blitz
