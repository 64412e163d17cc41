// The step between the input projections and attention over key ranges, one launch per layer for bf16 and fp32 tensors: norms over the whole
// query and key projections, a query temperature that grows with the position, and the write of the token's key and value into the cache.
#include "common/convert.cuh"
#include "common/tmap.h"

TTB_DEFINE_VIOLATION_COUNTER(span)

namespace ttb {
namespace span {

struct PrepareParams {
  void* q;              // [rows, ld_q], scaled in place
  const void *k, *v;    // [rows, ld_k | ld_v]
  long long ld_q, ld_k, ld_v;
  const void *q_gain, *k_gain;  // [q_width] / [k_width], or both nullptr: no norm
  void *keys, *values;  // [b, slots, k_width | v_width]
  const int* pos;       // [rows] positions, or nullptr (slot)
  const int* slot;      // device: slot of the first token, or nullptr
  int slot_host;
  int s, slots, q_width, k_width, v_width, every;
  float eps, coef;      // temperature 1 + coef * ln(floor((pos + 1) / every) + 1)
};

static constexpr int kThreads = 256;

template <typename T, int W>
struct Pack;  // W consecutive elements as fp32
template <typename T>
struct Pack<T, 1> {
  static __device__ __forceinline__ void load(const T* p, float (&f)[1]) { f[0] = as_float(*p); }
  static __device__ __forceinline__ void store(T* p, const float (&f)[1]) { *p = float_as<T>(f[0]); }
};
template <>
struct Pack<__nv_bfloat16, 8> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&f)[8]) { unpack_bf16x8(*reinterpret_cast<const uint4*>(p), f); }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&f)[8]) { *reinterpret_cast<uint4*>(p) = pack_bf16x8(f); }
};

template <typename T, int W>
__device__ __forceinline__ float squares(const T* p, int n) {
  float ss = 0.f;
  for (int i = threadIdx.x * W; i < n; i += kThreads * W) {
    float f[W];
    Pack<T, W>::load(p + i, f);
#pragma unroll
    for (int j = 0; j < W; ++j) ss += f[j] * f[j];
  }
  return ss;
}

template <typename T, int W>
__device__ __forceinline__ void scaled(T* dst, const T* src, const T* gain, int n, float by) {
  for (int i = threadIdx.x * W; i < n; i += kThreads * W) {
    float f[W], g[W];
    Pack<T, W>::load(src + i, f);
    if (gain != nullptr) Pack<T, W>::load(gain + i, g);
#pragma unroll
    for (int j = 0; j < W; ++j) f[j] = f[j] * by * (gain != nullptr ? g[j] : 1.f);
    Pack<T, W>::store(dst + i, f);
  }
}

template <typename T, int W>
__global__ void __launch_bounds__(kThreads) span_prepare_kernel(const PrepareParams p) {
  __shared__ float scratch[kThreads / 32];
  const long long row = blockIdx.x;
  const int bi = static_cast<int>(row / p.s), i = static_cast<int>(row % p.s);
  const int slot = (p.slot != nullptr ? *p.slot : p.slot_host) + i;
  T* q = static_cast<T*>(p.q) + row * p.ld_q;
  const T* k = static_cast<const T*>(p.k) + row * p.ld_k;
  const T* v = static_cast<const T*>(p.v) + row * p.ld_v;
  const T* q_gain = static_cast<const T*>(p.q_gain);
  const T* k_gain = static_cast<const T*>(p.k_gain);
  float by_q = 1.f, by_k = 1.f;
  if (q_gain != nullptr) {
    const float sq = squares<T, W>(q, p.q_width), sk = squares<T, W>(k, p.k_width);
    by_q = 1.f / sqrtf(cta_sum<kThreads>(sq, scratch) / static_cast<float>(p.q_width) + p.eps);
    by_k = 1.f / sqrtf(cta_sum<kThreads>(sk, scratch) / static_cast<float>(p.k_width) + p.eps);
  }
  if (p.coef != 0.f) {
    const int pos = max(p.pos != nullptr ? p.pos[row] : slot, 0);
    by_q *= 1.f + p.coef * logf(static_cast<float>((pos + 1) / p.every + 1));
  }
  if (q_gain != nullptr || p.coef != 0.f) scaled<T, W>(q, q, q_gain, p.q_width, by_q);
  if (slot < 0 || slot >= p.slots) {
    if (threadIdx.x == 0) TTB_NOTE_VIOLATION(span);
    return;
  }
  const long long at = static_cast<long long>(bi) * p.slots + slot;
  scaled<T, W>(static_cast<T*>(p.keys) + at * p.k_width, k, k_gain, p.k_width, by_k);
  scaled<T, W>(static_cast<T*>(p.values) + at * p.v_width, v, static_cast<const T*>(nullptr), p.v_width, 1.f);
}

}  // namespace span
}  // namespace ttb

// `wide`: fp32 tensors, else bf16.
extern "C" int ttb_span_prepare(void* q, long long ld_q, const void* k, long long ld_k, const void* v, long long ld_v, const void* q_gain, const void* k_gain, void* keys, void* values,
                                const int* pos, const int* slot, int slot_host, int rows, int s, int slots, int q_width, int k_width, int v_width, float eps, float coef, int every,
                                int wide, void* stream) {
  using namespace ttb;
  using namespace ttb::span;
  if (rows <= 0 || s <= 0 || rows % s || slots <= 0 || q_width <= 0 || k_width <= 0 || v_width <= 0 || every <= 0 || (q_gain == nullptr) != (k_gain == nullptr)) return kErrBadShape;
  PrepareParams p{q, k, v, ld_q, ld_k, ld_v, q_gain, k_gain, keys, values, pos, slot, slot_host, s, slots, q_width, k_width, v_width, every, eps, coef};
  const uintptr_t at = reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v) | reinterpret_cast<uintptr_t>(q_gain) |
                       reinterpret_cast<uintptr_t>(k_gain) | reinterpret_cast<uintptr_t>(keys) | reinterpret_cast<uintptr_t>(values);
  const bool vec = !wide && !(at & 15) && !((ld_q | ld_k | ld_v | q_width | k_width | v_width) & 7);
  auto st = static_cast<cudaStream_t>(stream);
  TTB_COUNT_LAUNCH(1);
  if (wide) span_prepare_kernel<float, 1><<<rows, kThreads, 0, st>>>(p);
  else if (vec) span_prepare_kernel<__nv_bfloat16, 8><<<rows, kThreads, 0, st>>>(p);
  else span_prepare_kernel<__nv_bfloat16, 1><<<rows, kThreads, 0, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? kOk : kErrDriver;
}
