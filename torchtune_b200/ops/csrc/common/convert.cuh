// Conversions between fp32 and a kernel's tensor type, and the four-element accesses built on them.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace ttb {

__device__ __forceinline__ float as_float(float v) { return v; }
__device__ __forceinline__ float as_float(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T float_as(float v) {
  if constexpr (sizeof(T) == 4) return v;
  else return __float2bfloat16_rn(v);
}

__device__ __forceinline__ void load4(const float* p, float (&f)[4]) {
  const float4 v = *reinterpret_cast<const float4*>(p);
  f[0] = v.x, f[1] = v.y, f[2] = v.z, f[3] = v.w;
}
__device__ __forceinline__ void load4(const __nv_bfloat16* p, float (&f)[4]) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  f[0] = a.x, f[1] = a.y, f[2] = b.x, f[3] = b.y;
}
__device__ __forceinline__ void store4(float* p, const float (&f)[4]) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float (&f)[4]) {
  uint2 u;
  *reinterpret_cast<__nv_bfloat162*>(&u.x) = __floats2bfloat162_rn(f[0], f[1]);
  *reinterpret_cast<__nv_bfloat162*>(&u.y) = __floats2bfloat162_rn(f[2], f[3]);
  *reinterpret_cast<uint2*>(p) = u;
}
__device__ __forceinline__ void unpack_bf16x8(const uint4& u, float (&f)[8]) {
  const __nv_bfloat162* b = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 t = __bfloat1622float2(b[i]);
    f[2 * i] = t.x, f[2 * i + 1] = t.y;
  }
}
__device__ __forceinline__ uint4 pack_bf16x8(const float (&f)[8]) {
  uint4 u;
  __nv_bfloat162* b = reinterpret_cast<__nv_bfloat162*>(&u);
#pragma unroll
  for (int i = 0; i < 4; ++i) b[i] = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
  return u;
}

// Lanes 4m ... 4m + 3 hold four 16-byte pieces each; piece j of lane 4m + i becomes piece i of lane 4m + j.  A warp whose lanes hold rows so
// turns 16-byte accesses to 32 rows into 64-byte accesses to eight.  All lanes take part.
__device__ __forceinline__ void transpose_quads(uint4 (&v)[4]) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int bit = 1; bit <= 2; bit <<= 1) {
    const bool upper = lane & bit;
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const int a = bit == 1 ? 2 * k : k, b = a + bit;
      uint4 t = upper ? v[a] : v[b];
      t.x = __shfl_xor_sync(0xffffffffu, t.x, bit);
      t.y = __shfl_xor_sync(0xffffffffu, t.y, bit);
      t.z = __shfl_xor_sync(0xffffffffu, t.z, bit);
      t.w = __shfl_xor_sync(0xffffffffu, t.w, bit);
      if (upper) v[a] = t;
      else v[b] = t;
    }
  }
}

// 1 / (1 + e^-z): the fast exponential where the result is rounded to bf16 anyway, the full-precision one for fp32 tensors
template <typename T>
__device__ __forceinline__ float logistic(float z) {
  if constexpr (sizeof(T) == 4) return 1.f / (1.f + expf(-z));
  else return 1.f / (1.f + __expf(-z));
}

// Sums of two values over all threads of a CTA; every thread gets them.
template <int THREADS>
__device__ __forceinline__ float2 cta_sum2(float a, float b, float2* scratch) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    a += __shfl_xor_sync(0xffffffffu, a, o);
    b += __shfl_xor_sync(0xffffffffu, b, o);
  }
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
  if (l == 0) scratch[w] = make_float2(a, b);
  __syncthreads();
  float2 t = make_float2(0.f, 0.f);
#pragma unroll
  for (int i = 0; i < THREADS / 32; ++i) {
    const float2 v = scratch[i];
    t.x += v.x, t.y += v.y;
  }
  return t;
}

// Sum over all threads of a CTA; every thread gets it.
template <int THREADS>
__device__ __forceinline__ float cta_sum(float v, float* scratch) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
  __syncthreads();
  if (l == 0) scratch[w] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < THREADS / 32; ++i) t += scratch[i];
  return t;
}

}  // namespace ttb
