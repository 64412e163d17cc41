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
struct Pack;  // W consecutive elements
template <typename T>
struct Pack<T, 1> {
  using Raw = T;
  static __device__ __forceinline__ Raw zero() { return float_as<T>(0.f); }
  static __device__ __forceinline__ void unpack(const Raw& r, float (&f)[1]) { f[0] = as_float(r); }
  static __device__ __forceinline__ Raw pack(const float (&f)[1]) { return float_as<T>(f[0]); }
};
template <>
struct Pack<__nv_bfloat16, 8> {
  using Raw = uint4;
  static __device__ __forceinline__ Raw zero() { return make_uint4(0u, 0u, 0u, 0u); }
  static __device__ __forceinline__ void unpack(const Raw& r, float (&f)[8]) { unpack_bf16x8(r, f); }
  static __device__ __forceinline__ Raw pack(const float (&f)[8]) { return pack_bf16x8(f); }
};

// A thread's pieces of a row: the first HELD of them wait in registers between the sum of squares and the scaling, the rest (of a very
// wide row) are read again.
template <typename T, int W, int HELD>
struct Row {
  using P = Pack<T, W>;
  using Raw = typename P::Raw;
  Raw r[HELD];
  static __device__ __forceinline__ int at(int k) { return (threadIdx.x + k * kThreads) * W; }
  static __device__ __forceinline__ const Raw& raw(const T* p) { return *reinterpret_cast<const Raw*>(p); }
  static __device__ __forceinline__ float squares_of(const Raw& v) {
    float f[W], ss = 0.f;
    P::unpack(v, f);
#pragma unroll
    for (int j = 0; j < W; ++j) ss += f[j] * f[j];
    return ss;
  }
  static __device__ __forceinline__ Raw scaled(const Raw& v, const T* gain, float by) {
    float f[W], g[W];
    P::unpack(v, f);
    if (gain != nullptr) P::unpack(raw(gain), g);
#pragma unroll
    for (int j = 0; j < W; ++j) f[j] = f[j] * by * (gain != nullptr ? g[j] : 1.f);
    return P::pack(f);
  }
  __device__ __forceinline__ void load(const T* p, int n) {
#pragma unroll
    for (int k = 0; k < HELD; ++k) r[k] = at(k) < n ? raw(p + at(k)) : P::zero();
  }
  __device__ __forceinline__ float squares(const T* p, int n) const {
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < HELD; ++k) ss += squares_of(r[k]);
    for (int i = at(HELD); i < n; i += kThreads * W) ss += squares_of(raw(p + i));
    return ss;
  }
  __device__ __forceinline__ void store(T* dst, const T* p, const T* gain, int n, float by) const {
#pragma unroll
    for (int k = 0; k < HELD; ++k)
      if (at(k) < n) *reinterpret_cast<Raw*>(dst + at(k)) = scaled(r[k], gain != nullptr ? gain + at(k) : nullptr, by);
    for (int i = at(HELD); i < n; i += kThreads * W) *reinterpret_cast<Raw*>(dst + i) = scaled(raw(p + i), gain != nullptr ? gain + i : nullptr, by);
  }
};

template <typename T, int W>
__global__ void __launch_bounds__(kThreads) span_prepare_kernel(const PrepareParams p) {
  __shared__ float2 scratch[kThreads / 32];
  const long long row = blockIdx.x;
  const int bi = static_cast<int>(row / p.s), i = static_cast<int>(row % p.s);
  T* q = static_cast<T*>(p.q) + row * p.ld_q;
  const T* k = static_cast<const T*>(p.k) + row * p.ld_k;
  const T* v = static_cast<const T*>(p.v) + row * p.ld_v;
  const T* q_gain = static_cast<const T*>(p.q_gain);
  const T* k_gain = static_cast<const T*>(p.k_gain);
  Row<T, W, 2> rq;
  Row<T, W, 1> rk, rv;
  rq.load(q, p.q_width);
  rk.load(k, p.k_width);
  rv.load(v, p.v_width);
  const int slot = (p.slot != nullptr ? *p.slot : p.slot_host) + i;
  float by_q = 1.f, by_k = 1.f;
  if (q_gain != nullptr) {
    const float2 ss = cta_sum2<kThreads>(rq.squares(q, p.q_width), rk.squares(k, p.k_width), scratch);
    by_q = 1.f / sqrtf(ss.x / static_cast<float>(p.q_width) + p.eps);
    by_k = 1.f / sqrtf(ss.y / static_cast<float>(p.k_width) + p.eps);
  }
  if (p.coef != 0.f) {
    const int pos = max(p.pos != nullptr ? p.pos[row] : slot, 0);
    by_q *= 1.f + p.coef * logf(static_cast<float>((pos + 1) / p.every + 1));
  }
  if (q_gain != nullptr || p.coef != 0.f) rq.store(q, q, q_gain, p.q_width, by_q);
  if (slot < 0 || slot >= p.slots) {
    if (threadIdx.x == 0) TTB_NOTE_VIOLATION(span);
    return;
  }
  const long long at = static_cast<long long>(bi) * p.slots + slot;
  rk.store(static_cast<T*>(p.keys) + at * p.k_width, k, k_gain, p.k_width, by_k);
  rv.store(static_cast<T*>(p.values) + at * p.v_width, v, nullptr, p.v_width, 1.f);
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
