// RMS norms around a 32-bit residual stream.
//
//   rms_norm_stream:   h = norm(x; w)                                     x fp32 -> h bf16 / fp32
//   residual_norm:     x' = x + mult * norm(y; w_post)                    y bf16 / fp32 (a sublayer's output)
//                      h  = norm(x'; w_next)                              optional
//
// with norm(z; w) = z / sqrt(mean(z^2) + eps) * (offset + w): offset 0 is a plain gain, 1 a gain stored around zero.  Both norms
// and the residual sum are fp32.  residual_norm is the step between two sublayers of a block whose sublayers are normed on both
// sides: the sublayer's output is read once, the stream is read and written once and the next sublayer's input leaves with it.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "common/tmap.h"

namespace ttb {
namespace resnorm {

template <typename T>
struct Vec4;  // four consecutive elements as fp32
template <>
struct Vec4<float> {
  static __device__ __forceinline__ void load(const float* p, float (&f)[4]) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    f[0] = v.x, f[1] = v.y, f[2] = v.z, f[3] = v.w;
  }
  static __device__ __forceinline__ void store(float* p, const float (&f)[4]) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }
  static __device__ __forceinline__ float one(const float* p) { return *p; }
  static __device__ __forceinline__ void put(float* p, float v) { *p = v; }
};
template <>
struct Vec4<__nv_bfloat16> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&f)[4]) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    f[0] = a.x, f[1] = a.y, f[2] = b.x, f[3] = b.y;
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&f)[4]) {
    uint2 u;
    *reinterpret_cast<__nv_bfloat162*>(&u.x) = __floats2bfloat162_rn(f[0], f[1]);
    *reinterpret_cast<__nv_bfloat162*>(&u.y) = __floats2bfloat162_rn(f[2], f[3]);
    *reinterpret_cast<uint2*>(p) = u;
  }
  static __device__ __forceinline__ float one(const __nv_bfloat16* p) { return __bfloat162float(*p); }
  static __device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
};

template <int THREADS>
__device__ __forceinline__ float block_sum(float v, float* scratch) {
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

// One CTA per row; V > 0: D % 4 == 0 and D <= 4 * THREADS * V, the row lives in registers between the passes.  V == 0: any D, the
// row is re-read (rare widths).
template <typename Ty, typename Th, int THREADS, int V>
__global__ void __launch_bounds__(THREADS)
residual_norm_kernel(const float* __restrict__ x, const Ty* __restrict__ y, const Ty* __restrict__ w_post, float* __restrict__ x_out,
                     const Ty* __restrict__ w_next, Th* __restrict__ h, int D, float eps, float mult, float offset) {
  __shared__ float scratch[THREADS / 32];
  const long long base = static_cast<long long>(blockIdx.x) * D;
  const float inv_d = 1.f / static_cast<float>(D);
  if constexpr (V > 0) {
    float xv[V][4];
#pragma unroll
    for (int k = 0; k < V; ++k) {
      const int i = (threadIdx.x + k * THREADS) * 4;
      if (i < D) Vec4<float>::load(x + base + i, xv[k]);
      else xv[k][0] = xv[k][1] = xv[k][2] = xv[k][3] = 0.f;
    }
    if (y != nullptr) {
      float yv[V][4];
      float ss = 0.f;
#pragma unroll
      for (int k = 0; k < V; ++k) {
        const int i = (threadIdx.x + k * THREADS) * 4;
        if (i < D) Vec4<Ty>::load(y + base + i, yv[k]);
        else yv[k][0] = yv[k][1] = yv[k][2] = yv[k][3] = 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) ss += yv[k][j] * yv[k][j];
      }
      const float rs = 1.f / sqrtf(block_sum<THREADS>(ss, scratch) * inv_d + eps);
#pragma unroll
      for (int k = 0; k < V; ++k) {
        const int i = (threadIdx.x + k * THREADS) * 4;
        if (i >= D) continue;
        float g[4];
        Vec4<Ty>::load(w_post + i, g);
#pragma unroll
        for (int j = 0; j < 4; ++j) xv[k][j] += mult * (yv[k][j] * rs * (offset + g[j]));
        Vec4<float>::store(x_out + base + i, xv[k]);
      }
    }
    if (h == nullptr) return;
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < V; ++k)
#pragma unroll
      for (int j = 0; j < 4; ++j) ss += xv[k][j] * xv[k][j];
    const float rs = 1.f / sqrtf(block_sum<THREADS>(ss, scratch) * inv_d + eps);
#pragma unroll
    for (int k = 0; k < V; ++k) {
      const int i = (threadIdx.x + k * THREADS) * 4;
      if (i >= D) continue;
      float g[4], o[4];
      Vec4<Ty>::load(w_next + i, g);
#pragma unroll
      for (int j = 0; j < 4; ++j) o[j] = xv[k][j] * rs * (offset + g[j]);
      Vec4<Th>::store(h + base + i, o);
    }
  } else {
    const float* xs = x + base;
    if (y != nullptr) {
      float ss = 0.f;
      for (int i = threadIdx.x; i < D; i += THREADS) {
        const float v = Vec4<Ty>::one(y + base + i);
        ss += v * v;
      }
      const float rs = 1.f / sqrtf(block_sum<THREADS>(ss, scratch) * inv_d + eps);
      for (int i = threadIdx.x; i < D; i += THREADS)
        x_out[base + i] = xs[i] + mult * (Vec4<Ty>::one(y + base + i) * rs * (offset + Vec4<Ty>::one(w_post + i)));
      xs = x_out + base;  // every element is read back by the thread that wrote it
    }
    if (h == nullptr) return;
    float ss = 0.f;
    for (int i = threadIdx.x; i < D; i += THREADS) ss += xs[i] * xs[i];
    const float rs = 1.f / sqrtf(block_sum<THREADS>(ss, scratch) * inv_d + eps);
    for (int i = threadIdx.x; i < D; i += THREADS) Vec4<Th>::put(h + base + i, xs[i] * rs * (offset + Vec4<Ty>::one(w_next + i)));
  }
}

template <typename Ty, typename Th>
static int launch(const float* x, const void* y, const void* w_post, float* x_out, const void* w_next, void* h, int rows, int D, float eps, float mult,
                  float offset, cudaStream_t st) {
  auto yp = static_cast<const Ty*>(y);
  auto wp = static_cast<const Ty*>(w_post);
  auto wn = static_cast<const Ty*>(w_next);
  auto hp = static_cast<Th*>(h);
  const bool aligned = D % 4 == 0 && !((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(w_post) |
                                        reinterpret_cast<uintptr_t>(x_out) | reinterpret_cast<uintptr_t>(w_next) | reinterpret_cast<uintptr_t>(h)) & 15);
  TTB_COUNT_LAUNCH(1);
#define TTB_RESNORM(THREADS, V) residual_norm_kernel<Ty, Th, THREADS, V><<<rows, THREADS, 0, st>>>(x, yp, wp, x_out, wn, hp, D, eps, mult, offset)
  if (!aligned || D > 16384) TTB_RESNORM(256, 0);
  else if (D <= 512) TTB_RESNORM(128, 1);
  else if (D <= 1024) TTB_RESNORM(256, 1);
  else if (D <= 2048) TTB_RESNORM(256, 2);
  else if (D <= 4096) TTB_RESNORM(256, 4);
  else if (D <= 8192) TTB_RESNORM(512, 4);
  else TTB_RESNORM(512, 8);
#undef TTB_RESNORM
  return cudaGetLastError() == cudaSuccess ? kOk : kErrDriver;
}

}  // namespace resnorm
}  // namespace ttb

// x [rows, D] fp32; y [rows, D] and the gains of type `wide` ? fp32 : bf16.  y == nullptr: h = norm(x; w_next) only.  h == nullptr:
// the residual step only.  h is fp32 if `wide`, else bf16.  x_out may alias x.
extern "C" int ttb_residual_norm(const float* x, const void* y, const void* w_post, float* x_out, const void* w_next, void* h, int rows, int D, float eps,
                                 float mult, float offset, int wide, void* stream) {
  using namespace ttb;
  if (rows <= 0 || D <= 0 || (y == nullptr && h == nullptr) || (y != nullptr && (w_post == nullptr || x_out == nullptr)) || (h != nullptr && w_next == nullptr))
    return kErrBadShape;
  auto st = static_cast<cudaStream_t>(stream);
  return wide ? resnorm::launch<float, float>(x, y, w_post, x_out, w_next, h, rows, D, eps, mult, offset, st)
              : resnorm::launch<__nv_bfloat16, __nv_bfloat16>(x, y, w_post, x_out, w_next, h, rows, D, eps, mult, offset, st);
}
