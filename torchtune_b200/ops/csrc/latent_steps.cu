// The steps around latent attention, for bf16 and fp32 tensors:
//
//   latent_prepare     one launch per layer after the input projections: norm of the latent, rotation of the shared key part and of
//                      the queries' rotated parts, and the write of the latent row into the cache
//   latent_absorb      q_lat[r, h, :] = W_uk[h]^T q[r, h, :]            (few rows: weight-streaming)
//   latent_combine     split-key partials of the decode kernel -> latent outputs
//   latent_value       out[r, h, :] = (W_uv[h] o_lat[r, h, :]) * sigmoid(gate)
//   latent_attention_any   attention for every size and for fp32 (no tensor cores); queries or heads as rows
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "common/tmap.h"

TTB_DEFINE_VIOLATION_COUNTER(latent)

namespace ttb {
namespace latent {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) {
  return v;
}
template <>
__device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) {
  return __float2bfloat16_rn(v);
}
template <typename T>
__device__ __forceinline__ float sigmoid_as(float z) {
  if constexpr (sizeof(T) == 4) return 1.f / (1.f + expf(-z));
  else return 1.f / (1.f + __expf(-z));
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// ------------------------------------------------------------------------------- prepare
struct PrepareParams {
  const void* kv;        // [rows, ld_kv]: `rank` latent columns, then `rot` key columns; nullptr: the layer reads another layer's cache
  long long ld_kv;
  const void* kv_gain;   // [rank]
  void* q;               // [rows, ld_q]: head h at column h * (dim + rot), laid out [dim | rot]
  long long ld_q;
  void* q_out;           // nullptr: the rotated part is written in place; else [rows, heads, rank + rot], columns rank...
  void* cache;           // [b, slots, rank + rot]
  const float* table;    // [table_len, rot_dims / 2, 2] (cos, sin)
  const int* pos;        // [rows] positions, or nullptr (slot)
  const int* slot;       // device: slot of the first token, or nullptr
  int slot_host;
  int s, slots, heads, dim, rot, rot_dims, rank, table_len;
  float eps;
  int vec;               // bf16 rows that can be read and written 16 bytes at a time
};

__device__ __forceinline__ void unpack8(const uint4& u, float (&f)[8]) {
  const __nv_bfloat162* b = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 t = __bfloat1622float2(b[i]);
    f[2 * i] = t.x, f[2 * i + 1] = t.y;
  }
}
__device__ __forceinline__ uint4 pack8(const float (&f)[8]) {
  uint4 u;
  __nv_bfloat162* b = reinterpret_cast<__nv_bfloat162*>(&u);
#pragma unroll
  for (int i = 0; i < 4; ++i) b[i] = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
  return u;
}
// four pairs turned by the angles whose (cos, sin) start at t
__device__ __forceinline__ uint4 turn8(const uint4& u, const float* t) {
  float f[8], o[8];
  unpack8(u, f);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    o[2 * i] = f[2 * i] * t[2 * i] - f[2 * i + 1] * t[2 * i + 1];
    o[2 * i + 1] = f[2 * i + 1] * t[2 * i] + f[2 * i] * t[2 * i + 1];
  }
  return pack8(o);
}

// One token, 128 threads: the latent (at most 1024 values) stays in registers between its sum of squares and the scaling, and the
// queries' rotated parts are fetched before the reduction.
__device__ __forceinline__ void prepare_row_vec8(const PrepareParams& p, const float* cs, float* scratch, long long row, int bi, int slot) {
  const int per_head = p.rot >> 3, turned = p.rot_dims >> 3, total = p.heads * per_head;
  uint4* q = reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(p.q) + row * p.ld_q);
  const int q_pitch = (p.dim + p.rot) >> 3, q_off = p.dim >> 3, o_pitch = (p.rank + p.rot) >> 3, o_off = p.rank >> 3;
  uint4* out = p.q_out != nullptr ? reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(p.q_out) + row * p.heads * (p.rank + p.rot)) : nullptr;
  int h0 = 0, c0 = 0;
  uint4 first = make_uint4(0u, 0u, 0u, 0u);
  if (static_cast<int>(threadIdx.x) < total) {
    h0 = threadIdx.x / per_head, c0 = threadIdx.x - h0 * per_head;
    first = q[h0 * q_pitch + q_off + c0];
  }
  if (p.kv != nullptr) {
    const uint4* src = reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(p.kv) + row * p.ld_kv);
    const int i = threadIdx.x, n = p.rank >> 3;
    float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (i < n) unpack8(src[i], f);
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += f[j] * f[j];
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = ss;
    __syncthreads();
    const float rs = 1.f / sqrtf((scratch[0] + scratch[1] + scratch[2] + scratch[3]) / static_cast<float>(p.rank) + p.eps);
    if (slot >= 0 && slot < p.slots) {
      uint4* dst = reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(p.cache) + (static_cast<long long>(bi) * p.slots + slot) * (p.rank + p.rot));
      if (i < n) {
        float g[8];
        unpack8(reinterpret_cast<const uint4*>(p.kv_gain)[i], g);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] = f[j] * rs * g[j];
        dst[i] = pack8(f);
      }
      for (int k = threadIdx.x; k < per_head; k += 128) dst[n + k] = k < turned ? turn8(src[n + k], cs + k * 8) : src[n + k];
    } else if (threadIdx.x == 0) {
      TTB_NOTE_VIOLATION(latent);
    }
  }
  for (int w = threadIdx.x; w < total; w += 128) {
    const int h = w == static_cast<int>(threadIdx.x) ? h0 : w / per_head;
    const int c = w == static_cast<int>(threadIdx.x) ? c0 : w - h * per_head;
    const uint4 u = w == static_cast<int>(threadIdx.x) ? first : q[h * q_pitch + q_off + c];
    if (out != nullptr) out[h * o_pitch + o_off + c] = c < turned ? turn8(u, cs + c * 8) : u;
    else if (c < turned) q[h * q_pitch + q_off + c] = turn8(u, cs + c * 8);
  }
}

template <typename T>
__global__ void __launch_bounds__(128) latent_prepare_kernel(PrepareParams p) {
  __shared__ float scratch[4];
  extern __shared__ float cs[];  // rot_dims values: cos, sin of this token
  const long long row = blockIdx.x;
  const int bi = static_cast<int>(row / p.s), i = static_cast<int>(row % p.s);
  const int slot = (p.slot != nullptr ? *p.slot : p.slot_host) + i;
  int pos = p.pos != nullptr ? p.pos[row] : slot;
  if (pos < 0 || pos >= p.table_len) {
    if (threadIdx.x == 0) TTB_NOTE_VIOLATION(latent);
    pos = 0;
  }
  for (int k = threadIdx.x; k < p.rot_dims; k += blockDim.x) cs[k] = p.table[static_cast<long long>(pos) * p.rot_dims + k];
  __syncthreads();
  const int half = p.rot_dims / 2;

  if constexpr (sizeof(T) == 2) {
    if (p.vec) {
      prepare_row_vec8(p, cs, scratch, row, bi, slot);
      return;
    }
  }
  if (p.kv != nullptr) {
    const T* src = static_cast<const T*>(p.kv) + row * p.ld_kv;
    const T* gain = static_cast<const T*>(p.kv_gain);
    float ss = 0.f;
    for (int k = threadIdx.x; k < p.rank; k += blockDim.x) {
      const float v = to_f(src[k]);
      ss += v * v;
    }
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = ss;
    __syncthreads();
    const float rs = 1.f / sqrtf((scratch[0] + scratch[1] + scratch[2] + scratch[3]) / static_cast<float>(p.rank) + p.eps);
    if (slot >= 0 && slot < p.slots) {
      T* dst = static_cast<T*>(p.cache) + (static_cast<long long>(bi) * p.slots + slot) * (p.rank + p.rot);
      for (int k = threadIdx.x; k < p.rank; k += blockDim.x) dst[k] = from_f<T>(to_f(src[k]) * rs * to_f(gain[k]));
      src += p.rank, dst += p.rank;
      for (int k = threadIdx.x; k < half; k += blockDim.x) {
        const float u = to_f(src[2 * k]), v = to_f(src[2 * k + 1]), c = cs[2 * k], sn = cs[2 * k + 1];
        dst[2 * k] = from_f<T>(u * c - v * sn);
        dst[2 * k + 1] = from_f<T>(v * c + u * sn);
      }
      for (int k = p.rot_dims + threadIdx.x; k < p.rot; k += blockDim.x) dst[k] = src[k];
    } else if (threadIdx.x == 0) {
      TTB_NOTE_VIOLATION(latent);
    }
  }

  T* q = static_cast<T*>(p.q) + row * p.ld_q + p.dim;
  T* out = p.q_out != nullptr ? static_cast<T*>(p.q_out) + row * p.heads * (p.rank + p.rot) + p.rank : nullptr;
  const int out_pitch = p.rank + p.rot;
  for (int w = threadIdx.x; w < p.heads * half; w += blockDim.x) {
    const int h = w / half, k = w - h * half;
    T* src = q + h * (p.dim + p.rot);
    const float u = to_f(src[2 * k]), v = to_f(src[2 * k + 1]), c = cs[2 * k], sn = cs[2 * k + 1];
    T* dst = out != nullptr ? out + h * out_pitch : src;
    dst[2 * k] = from_f<T>(u * c - v * sn);
    dst[2 * k + 1] = from_f<T>(v * c + u * sn);
  }
  if (out != nullptr && p.rot_dims < p.rot) {
    const int rest = p.rot - p.rot_dims;
    for (int w = threadIdx.x; w < p.heads * rest; w += blockDim.x) {
      const int h = w / rest, k = p.rot_dims + w - h * rest;
      out[h * out_pitch + k] = q[h * (p.dim + p.rot) + k];
    }
  }
}

// ------------------------------------------------------------------------------- absorb: contraction over weight rows
// out[r, h, n] = sum_k a[r, h, k] * w[h * K + k, n].  A warp owns 32 * VEC output columns and every eighth k; the eight partial sums
// meet in shared memory.  ROWS batch rows share the streamed weights.
template <typename T, int VEC>
struct WVec;
template <>
struct WVec<float, 4> {
  static __device__ __forceinline__ void load(const float* p, float (&f)[4]) {
    const float4 v = __ldg(reinterpret_cast<const float4*>(p));
    f[0] = v.x, f[1] = v.y, f[2] = v.z, f[3] = v.w;
  }
  static __device__ __forceinline__ void load_shared(const float* p, float (&f)[4]) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    f[0] = v.x, f[1] = v.y, f[2] = v.z, f[3] = v.w;
  }
};
template <>
struct WVec<__nv_bfloat16, 4> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&f)[4]) {
    const uint2 u = __ldg(reinterpret_cast<const uint2*>(p));
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    f[0] = a.x, f[1] = a.y, f[2] = b.x, f[3] = b.y;
  }
};
template <typename T>
struct WVec<T, 1> {
  static __device__ __forceinline__ void load(const T* p, float (&f)[1]) { f[0] = to_f(*p); }
  static __device__ __forceinline__ void load_shared(const T* p, float (&f)[1]) { f[0] = to_f(*p); }
};

static constexpr int kRows = 8;

template <typename T, int VEC>
__global__ void __launch_bounds__(256) latent_absorb_kernel(const T* __restrict__ a, long long a_row, int a_head, const T* __restrict__ w, T* __restrict__ out,
                                                            long long out_row, int out_head, int R, int K, int N) {
  extern __shared__ float sm[];
  float* sA = sm;                  // [kRows][K]
  float* sP = sm + kRows * K;      // [8][kRows][32 * VEC]
  const int h = blockIdx.y, r0 = blockIdx.z * kRows;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n = blockIdx.x * 32 * VEC + lane * VEC;
  const T* wp = w + static_cast<long long>(h) * K * N + n;
  if (n < N)  // the weights are on their way while the rows are staged
    for (int k = warp; k < K; k += 8) asm volatile("prefetch.global.L2 [%0];" ::"l"(wp + static_cast<long long>(k) * N));
#pragma unroll 4
  for (int t = threadIdx.x; t < kRows * K; t += 256) {
    const int r = t / K, k = t - r * K;
    sA[t] = r0 + r < R ? to_f(a[(r0 + r) * a_row + static_cast<long long>(h) * a_head + k]) : 0.f;
  }
  __syncthreads();
  float acc[kRows][VEC];
#pragma unroll
  for (int r = 0; r < kRows; ++r)
#pragma unroll
    for (int v = 0; v < VEC; ++v) acc[r][v] = 0.f;
  if (n < N) {
#pragma unroll 8
    for (int k = warp; k < K; k += 8) {
      float f[VEC];
      WVec<T, VEC>::load(wp + static_cast<long long>(k) * N, f);
#pragma unroll
      for (int r = 0; r < kRows; ++r) {
        const float x = sA[r * K + k];
#pragma unroll
        for (int v = 0; v < VEC; ++v) acc[r][v] += x * f[v];
      }
    }
  }
#pragma unroll
  for (int r = 0; r < kRows; ++r)
#pragma unroll
    for (int v = 0; v < VEC; ++v) sP[(warp * kRows + r) * 32 * VEC + lane * VEC + v] = acc[r][v];
  __syncthreads();
  for (int t = threadIdx.x; t < kRows * 32 * VEC; t += 256) {
    const int r = t / (32 * VEC), c = t - r * 32 * VEC;
    const int col = blockIdx.x * 32 * VEC + c;
    if (r0 + r >= R || col >= N) continue;
    float s = 0.f;
#pragma unroll
    for (int g = 0; g < 8; ++g) s += sP[(g * kRows + r) * 32 * VEC + c];
    out[(r0 + r) * out_row + static_cast<long long>(h) * out_head + col] = from_f<T>(s);
  }
}

// ------------------------------------------------------------------------------- split-key partials
// o [splits, R, heads, K] fp32 with ml [splits, R, heads] (log2-domain maximum, sum) -> the normalised rows, [R, heads, K] fp32 or
// head-major [heads, R, K] bf16 (the row order of a grouped GEMM whose groups are heads), or [R, heads, K] bf16.  One CTA per (row, head,
// 128 columns).
__device__ __forceinline__ float warp_max_of(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}

// GROUPS groups of 128 threads, each adding up every GROUPS-th range: several when there are many ranges (few rows).
enum CombineForm { kRowsF32 = 0, kHeadsBf16 = 1, kRowsBf16 = 2 };

template <int FORM, int GROUPS>
__global__ void __launch_bounds__(128 * GROUPS) latent_combine_kernel(const float* __restrict__ o, const float2* __restrict__ ml, void* __restrict__ out, int splits,
                                                                              int R, int heads, int K) {
  extern __shared__ float wts[];  // [splits]: exp2(m_s - m) / sum, 0 for a split without keys (which has written nothing)
  __shared__ float part[GROUPS][128];
  const int r = blockIdx.x, h = blockIdx.y, group = threadIdx.x >> 7, col = threadIdx.x & 127;
  const long long rh = static_cast<long long>(r) * heads + h, RH = static_cast<long long>(R) * heads;
  if (threadIdx.x < 32) {
    float m = -INFINITY, l = 0.f;
#pragma unroll 2
    for (int s = threadIdx.x; s < splits; s += 32) {
      const float2 v = ml[s * RH + rh];
      if (v.y > 0.f) {
        const float m_new = fmaxf(m, v.x);
        l = l * exp2f(m - m_new) + v.y * exp2f(v.x - m_new);  // m = -inf: the first factor is 0
        m = m_new;
      }
    }
    const float top = warp_max_of(m);
    l = warp_sum(m == -INFINITY ? 0.f : l * exp2f(m - top));
    const float inv = l > 0.f ? 1.f / l : 0.f;
    for (int s = threadIdx.x; s < splits; s += 32) {
      const float2 v = ml[s * RH + rh];
      wts[s] = v.y > 0.f ? exp2f(v.x - top) * inv : 0.f;
    }
  }
  __syncthreads();
  const int k = blockIdx.z * 128 + col;
  float acc = 0.f;
  if (k < K) {
    const float* src = o + rh * K + k;
#pragma unroll 8
    for (int s = group; s < splits; s += GROUPS) {
      const float v = src[s * RH * K];  // loaded in any case, so the loads of many ranges are in flight together
      acc += wts[s] != 0.f ? wts[s] * v : 0.f;
    }
  }
  if constexpr (GROUPS > 1) {
    part[group][col] = acc;
    __syncthreads();
  }
  if (group == 0 && k < K) {
#pragma unroll
    for (int g = 1; g < GROUPS; ++g) acc += part[g][col];
    if constexpr (FORM == kRowsBf16) static_cast<__nv_bfloat16*>(out)[rh * K + k] = __float2bfloat16_rn(acc);
    else if constexpr (FORM == kHeadsBf16) static_cast<__nv_bfloat16*>(out)[(static_cast<long long>(h) * R + r) * K + k] = __float2bfloat16_rn(acc);
    else static_cast<float*>(out)[rh * K + k] = acc;
  }
}

// ------------------------------------------------------------------------------- value projection: contraction along weight rows
// out[r, h, n] = (sum_k o[r, h, k] * w[h * N + n, k]) / l[r, h] * sigmoid(gate[r, h * N + n]); ml (of one split) == nullptr: l = 1.
static constexpr int kValueCols = 16;

template <typename T, int VEC, int ROWS>
__global__ void __launch_bounds__(256) latent_value_kernel(const float* __restrict__ o, const float2* __restrict__ ml, const T* __restrict__ w,
                                                           const T* __restrict__ gate, long long gate_ld, T* __restrict__ out, int R, int heads, int K, int N) {
  extern __shared__ __align__(16) float sA[];  // [ROWS][K]
  const int h = blockIdx.y, r0 = blockIdx.z * ROWS;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n0 = blockIdx.x * kValueCols + warp * 2;
  const T* wp = w + (static_cast<long long>(h) * N + n0) * K;
#pragma unroll
  for (int c = 0; c < 2; ++c)
    if (n0 + c < N)
      for (int k = lane * (128 / static_cast<int>(sizeof(T))); k < K; k += 32 * (128 / static_cast<int>(sizeof(T))))
        asm volatile("prefetch.global.L2 [%0];" ::"l"(wp + static_cast<long long>(c) * K + k));
  const int vec_k = K / VEC;
#pragma unroll 4
  for (int t = threadIdx.x; t < ROWS * vec_k; t += 256) {
    const int r = t / vec_k, k = (t - r * vec_k) * VEC;
    float f[VEC];
#pragma unroll
    for (int v = 0; v < VEC; ++v) f[v] = 0.f;
    if (r0 + r < R) WVec<float, VEC>::load(o + (static_cast<long long>(r0 + r) * heads + h) * K + k, f);
#pragma unroll
    for (int v = 0; v < VEC; ++v) sA[r * K + k + v] = f[v];
  }
  float inv = 1.f;  // of row `lane`
  if (ml != nullptr && lane < ROWS && r0 + lane < R) {
    const float l = ml[static_cast<long long>(r0 + lane) * heads + h].y;
    inv = l > 0.f ? 1.f / l : 0.f;
  }
  __syncthreads();
  if (n0 >= N) return;
  const bool two = n0 + 1 < N;  // the two columns of a warp share every read of the rows
  float acc[2][ROWS];
#pragma unroll
  for (int r = 0; r < ROWS; ++r) acc[0][r] = acc[1][r] = 0.f;
#pragma unroll 4
  for (int k = lane * VEC; k < K; k += 32 * VEC) {
    float f[VEC], g[VEC];
    WVec<T, VEC>::load(wp + k, f);
    WVec<T, VEC>::load(wp + (two ? K : 0) + k, g);
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
      float a[VEC];
      WVec<float, VEC>::load_shared(sA + r * K + k, a);
#pragma unroll
      for (int v = 0; v < VEC; ++v) {
        acc[0][r] += a[v] * f[v];
        acc[1][r] += a[v] * g[v];
      }
    }
  }
#pragma unroll
  for (int c = 0; c < 2; ++c) {
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
      const float sum = warp_sum(acc[c][r]);
      if (lane == r && r0 + r < R && (c == 0 || two)) {
        const long long col = static_cast<long long>(h) * N + n0 + c;
        float v = inv == 0.f ? 0.f : sum * inv;  // a row without keys was never written
        if (gate != nullptr) v *= sigmoid_as<T>(to_f(gate[(r0 + r) * gate_ld + col]));
        out[static_cast<long long>(r0 + r) * heads * N + col] = from_f<T>(v);
      }
    }
  }
}

// x [heads, R, N] head-major -> out [R, heads * N] with the gate applied; and the way back in for the queries (copy of the unrotated
// parts to head-major order).
__global__ void latent_gate_rows_kernel(const __nv_bfloat16* __restrict__ x, const __nv_bfloat16* __restrict__ gate, long long gate_ld, __nv_bfloat16* __restrict__ out,
                                        int R, int heads, int N) {
  const long long total = static_cast<long long>(R) * heads * N;
  for (long long t = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; t < total; t += static_cast<long long>(gridDim.x) * blockDim.x) {
    const int n = static_cast<int>(t % N);
    const long long rh = t / N;
    const int h = static_cast<int>(rh % heads);
    const long long r = rh / heads;
    float v = __bfloat162float(x[(static_cast<long long>(h) * R + r) * N + n]);
    if (gate != nullptr) v *= sigmoid_as<__nv_bfloat16>(__bfloat162float(gate[r * gate_ld + static_cast<long long>(h) * N + n]));
    out[t] = __float2bfloat16_rn(v);
  }
}

// ------------------------------------------------------------------------------- attention for any size
struct AnyParams {
  const void* q;   // row (bi, i, h): q + bi*q_b + i*q_i + h*q_h, d1 + d2 contiguous values
  long long q_b, q_i, q_h;
  const void* k1;  // first d1 values of key (bi, j, h)
  long long k1_b, k1_j, k1_h;
  const void* k2;  // last d2 values of key (bi, j), shared by the heads
  long long k2_b, k2_j;
  const void* v;
  long long v_b, v_j, v_h;
  void* o;         // [b, s, heads, dv] of type T, or fp32 when out_f32
  float2* ml;      // out_f32: [b * s, heads] gets (0, 1) for rows that saw a key (their output is normalised), (0, 0) otherwise
  const void* gate;
  long long gate_ld;
  int b, s, sk, heads, d1, d2, dv;
  int group;       // query heads per key head (k1_h, v_h: pitch of key heads)
  int heads_as_rows, out_f32, key_tile;
  const int* slot;
  int slot_host;
  const int* lo;
  long long lo_row, lo_query;
  const int* hi;
  long long hi_row, hi_query;
  float scale;
};

static constexpr int kAnyRows = 16;

// 128 threads, 16 rows per CTA: 16 queries of one head, or (heads_as_rows, one query per sequence) 16 of the heads that share a key head.
template <typename T>
__global__ void __launch_bounds__(128) latent_attention_any_kernel(AnyParams p) {
  extern __shared__ float sm[];
  const int d = p.d1 + p.d2, KT = p.key_tile;
  float* sQ = sm;                           // [16][d]
  float* sK = sQ + kAnyRows * d;            // [KT][d + 1]
  float* sV = sK + KT * (d + 1);            // [KT][dv]
  float* sO = sV + KT * p.dv;               // [16][dv]
  float* sS = sO + kAnyRows * p.dv;         // [16][KT]
  float* sM = sS + kAnyRows * KT;           // [16] maximum
  float* sL = sM + kAnyRows;                // [16] sum
  float* sA = sL + kAnyRows;                // [16] rescale factor
  __shared__ int s_lo[kAnyRows], s_hi[kAnyRows];
  const int bi = blockIdx.z;
  const int row0 = blockIdx.x * kAnyRows;
  const int n_rows = min(kAnyRows, (p.heads_as_rows ? p.group : p.s) - row0);
  const int h_shared = p.heads_as_rows ? static_cast<int>(blockIdx.y) : static_cast<int>(blockIdx.y) / p.group;
  auto query_of = [&](int r) { return p.heads_as_rows ? 0 : row0 + r; };
  auto head_of = [&](int r) { return p.heads_as_rows ? h_shared * p.group + row0 + r : static_cast<int>(blockIdx.y); };
  const int slot0 = p.slot != nullptr ? *p.slot : p.slot_host;

  for (int t = threadIdx.x; t < kAnyRows * d; t += 128) {
    const int r = t / d, k = t - r * d;
    sQ[t] = r < n_rows ? to_f(static_cast<const T*>(p.q)[bi * p.q_b + query_of(r) * p.q_i + head_of(r) * p.q_h + k]) * p.scale : 0.f;
  }
  for (int t = threadIdx.x; t < kAnyRows * p.dv; t += 128) sO[t] = 0.f;
  if (threadIdx.x < kAnyRows) {
    const int r = threadIdx.x;
    int lo = 0, hi = -1;
    if (r < n_rows) {
      const int i = query_of(r);
      lo = p.lo != nullptr ? max(p.lo[bi * p.lo_row + i * p.lo_query], 0) : 0;
      hi = p.hi != nullptr ? p.hi[bi * p.hi_row + i * p.hi_query] : slot0 + i;
      hi = min(hi, p.sk - 1);
    }
    s_lo[r] = lo, s_hi[r] = hi;
    sM[r] = -INFINITY, sL[r] = 0.f;
  }
  __syncthreads();
  int first = p.sk, last = -1;
#pragma unroll
  for (int r = 0; r < kAnyRows; ++r)
    if (s_hi[r] >= s_lo[r]) first = min(first, s_lo[r]), last = max(last, s_hi[r]);

  for (int j0 = first; j0 <= last; j0 += KT) {
    const int kn = min(KT, last - j0 + 1);
    for (int t = threadIdx.x; t < KT * d; t += 128) {
      const int j = t / d, k = t - j * d;
      float v = 0.f;
      if (j < kn) {
        const long long jj = j0 + j;
        v = k < p.d1 ? to_f(static_cast<const T*>(p.k1)[bi * p.k1_b + jj * p.k1_j + h_shared * p.k1_h + k])
                     : to_f(static_cast<const T*>(p.k2)[bi * p.k2_b + jj * p.k2_j + k - p.d1]);
      }
      sK[j * (d + 1) + k] = v;
    }
    for (int t = threadIdx.x; t < KT * p.dv; t += 128) {
      const int j = t / p.dv, k = t - j * p.dv;
      sV[t] = j < kn ? to_f(static_cast<const T*>(p.v)[bi * p.v_b + (j0 + j) * p.v_j + h_shared * p.v_h + k]) : 0.f;
    }
    __syncthreads();
    for (int t = threadIdx.x; t < kAnyRows * KT; t += 128) {
      const int r = t / KT, j = t - r * KT;
      const int jj = j0 + j;
      float acc = -INFINITY;
      if (j < kn && jj >= s_lo[r] && jj <= s_hi[r]) {
        acc = 0.f;
        const float* a = sQ + r * d;
        const float* k = sK + j * (d + 1);
        for (int e = 0; e < d; ++e) acc += a[e] * k[e];
      }
      sS[t] = acc;
    }
    __syncthreads();
    if (threadIdx.x < kAnyRows) {
      const int r = threadIdx.x;
      float m = sM[r];
      for (int j = 0; j < KT; ++j) m = fmaxf(m, sS[r * KT + j]);
      const float a = m == -INFINITY ? 1.f : expf(sM[r] - m);
      float l = sL[r] * a;
      for (int j = 0; j < KT; ++j) {
        const float e = m == -INFINITY ? 0.f : expf(sS[r * KT + j] - m);
        sS[r * KT + j] = e;
        l += e;
      }
      sM[r] = m, sL[r] = l, sA[r] = a;
    }
    __syncthreads();
    for (int t = threadIdx.x; t < kAnyRows * p.dv; t += 128) {
      const int r = t / p.dv, k = t - r * p.dv;
      float acc = sO[t] * sA[r];
      for (int j = 0; j < KT; ++j) acc += sS[r * KT + j] * sV[j * p.dv + k];
      sO[t] = acc;
    }
    __syncthreads();
  }

  for (int t = threadIdx.x; t < n_rows * p.dv; t += 128) {
    const int r = t / p.dv, k = t - r * p.dv;
    const int i = query_of(r), h = head_of(r);
    const long long token = static_cast<long long>(bi) * p.s + i;
    const long long at = (token * p.heads + h) * p.dv + k;
    float v = sL[r] > 0.f ? sO[t] / sL[r] : 0.f;
    if (p.out_f32) {
      static_cast<float*>(p.o)[at] = v;
      if (k == 0 && p.ml != nullptr) p.ml[token * p.heads + h] = make_float2(0.f, sL[r] > 0.f ? 1.f : 0.f);
    } else {
      if (p.gate != nullptr) v *= sigmoid_as<T>(to_f(static_cast<const T*>(p.gate)[token * p.gate_ld + static_cast<long long>(h) * p.dv + k]));
      static_cast<T*>(p.o)[at] = from_f<T>(v);
    }
  }
}

static constexpr int kSmemMax = 227 * 1024;

template <typename K>
static bool allow_smem(K kernel, int bytes, int& granted) {
  if (bytes <= 48 * 1024 || bytes <= granted) return true;
  if (bytes > kSmemMax) return false;
  if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes) != cudaSuccess) return false;
  granted = bytes;
  return true;
}

template <typename T>
static int launch_absorb(const void* a, long long a_row, int a_head, const void* w, void* out, long long out_row, int out_head, int R, int heads, int K, int N,
                         cudaStream_t st) {
  const bool vec = N % 4 == 0 && !(reinterpret_cast<uintptr_t>(w) & 15);
  const int cols = vec ? 128 : 32;
  const int smem = (kRows * K + 8 * kRows * cols) * 4;
  static int g4 = 0, g1 = 0;
  if (!(vec ? allow_smem(latent_absorb_kernel<T, 4>, smem, g4) : allow_smem(latent_absorb_kernel<T, 1>, smem, g1))) return kErrTooLarge;
  const dim3 grid((N + cols - 1) / cols, heads, (R + kRows - 1) / kRows);
  TTB_COUNT_LAUNCH(1);
  if (vec)
    latent_absorb_kernel<T, 4><<<grid, 256, smem, st>>>(static_cast<const T*>(a), a_row, a_head, static_cast<const T*>(w), static_cast<T*>(out), out_row, out_head, R, K, N);
  else
    latent_absorb_kernel<T, 1><<<grid, 256, smem, st>>>(static_cast<const T*>(a), a_row, a_head, static_cast<const T*>(w), static_cast<T*>(out), out_row, out_head, R, K, N);
  return cudaGetLastError() == cudaSuccess ? kOk : kErrDriver;
}

template <typename T, int VEC, int ROWS>
static int launch_value_rows(const float* o, const float2* ml, const void* w, const void* gate, long long gate_ld, void* out, int R, int heads, int K, int N,
                             cudaStream_t st) {
  const int smem = ROWS * K * 4;
  static int granted = 0;
  if (!allow_smem(latent_value_kernel<T, VEC, ROWS>, smem, granted)) return kErrTooLarge;
  TTB_COUNT_LAUNCH(1);
  latent_value_kernel<T, VEC, ROWS><<<dim3((N + kValueCols - 1) / kValueCols, heads, (R + ROWS - 1) / ROWS), 256, smem, st>>>(
      o, ml, static_cast<const T*>(w), static_cast<const T*>(gate), gate_ld, static_cast<T*>(out), R, heads, K, N);
  return cudaGetLastError() == cudaSuccess ? kOk : kErrDriver;
}

template <typename T>
static int launch_value(const float* o, const float* ml, const void* w, const void* gate, long long gate_ld, void* out, int R, int heads, int K, int N,
                        cudaStream_t st) {
  auto m = reinterpret_cast<const float2*>(ml);
  if (K % 4 || (reinterpret_cast<uintptr_t>(w) & 15)) return launch_value_rows<T, 1, kRows>(o, m, w, gate, gate_ld, out, R, heads, K, N, st);
  if (R == 1) return launch_value_rows<T, 4, 1>(o, m, w, gate, gate_ld, out, R, heads, K, N, st);
  if (R <= 4) return launch_value_rows<T, 4, 4>(o, m, w, gate, gate_ld, out, R, heads, K, N, st);
  return launch_value_rows<T, 4, kRows>(o, m, w, gate, gate_ld, out, R, heads, K, N, st);
}

}  // namespace latent
}  // namespace ttb

using namespace ttb;
using namespace ttb::latent;

// `wide`: fp32 tensors, else bf16 (here and below).
extern "C" int ttb_latent_prepare(const void* kv, long long ld_kv, const void* kv_gain, void* q, long long ld_q, void* q_out, void* cache, const float* table,
                                  const int* pos, const int* slot, int slot_host, int rows, int s, int slots, int heads, int dim, int rot, int rot_dims, int rank,
                                  int table_len, float eps, int wide, void* stream) {
  if (rows <= 0 || s <= 0 || rows % s || heads <= 0 || rot_dims < 0 || (rot_dims & 1) || rot_dims > rot || table_len <= 0) return kErrBadShape;
  if (kv != nullptr && (kv_gain == nullptr || cache == nullptr || slots <= 0)) return kErrBadShape;
  PrepareParams p{kv, ld_kv, kv_gain, q, ld_q, q_out, cache, table, pos, slot, slot_host, s, slots, heads, dim, rot, rot_dims, rank, table_len, eps, 0};
  const uintptr_t at = reinterpret_cast<uintptr_t>(kv) | reinterpret_cast<uintptr_t>(kv_gain) | reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(q_out) |
                       reinterpret_cast<uintptr_t>(cache);
  p.vec = !wide && !(at & 15) && !((ld_kv | ld_q | dim | rot | rot_dims | rank) & 7) && rank <= 1024;
  auto st = static_cast<cudaStream_t>(stream);
  TTB_COUNT_LAUNCH(1);
  if (wide) latent_prepare_kernel<float><<<rows, 128, rot_dims * 4, st>>>(p);
  else latent_prepare_kernel<__nv_bfloat16><<<rows, 128, rot_dims * 4, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? kOk : kErrDriver;
}

// out[r, h, :N] = a[r, h, :K] * w[h*K : (h+1)*K, :N]
extern "C" int ttb_latent_absorb(const void* a, long long a_row, int a_head, const void* w, void* out, long long out_row, int out_head, int rows, int heads, int K,
                                 int N, int wide, void* stream) {
  if (rows <= 0 || heads <= 0 || K <= 0 || N <= 0) return kErrBadShape;
  auto st = static_cast<cudaStream_t>(stream);
  return wide ? launch_absorb<float>(a, a_row, a_head, w, out, out_row, out_head, rows, heads, K, N, st)
              : launch_absorb<__nv_bfloat16>(a, a_row, a_head, w, out, out_row, out_head, rows, heads, K, N, st);
}

// o [rows, heads, K] fp32, w [heads*N, K]; out [rows, heads*N].  ml [rows, heads, 2] (of one split) divides by the sum, nullptr: o is normalised.
extern "C" int ttb_latent_value(const float* o, const float* ml, const void* w, const void* gate, long long gate_ld, void* out, int rows, int heads, int K, int N,
                                int wide, void* stream) {
  if (rows <= 0 || heads <= 0 || K <= 0 || N <= 0) return kErrBadShape;
  auto st = static_cast<cudaStream_t>(stream);
  return wide ? launch_value<float>(o, ml, w, gate, gate_ld, out, rows, heads, K, N, st)
              : launch_value<__nv_bfloat16>(o, ml, w, gate, gate_ld, out, rows, heads, K, N, st);
}

// form 0: [rows, heads, K] fp32, 1: [heads, rows, K] bf16, 2: [rows, heads, K] bf16
extern "C" int ttb_latent_combine(const float* o, const float* ml, void* out, int splits, int rows, int heads, int K, int form, void* stream) {
  if (rows <= 0 || heads <= 0 || K <= 0 || splits <= 0 || splits > 8192 || form < 0 || form > 2) return kErrBadShape;
  auto st = static_cast<cudaStream_t>(stream);
  auto m = reinterpret_cast<const float2*>(ml);
  TTB_COUNT_LAUNCH(1);
  const dim3 grid(rows, heads, (K + 127) / 128);
#define TTB_COMBINE(FORM, GROUPS) latent_combine_kernel<FORM, GROUPS><<<grid, 128 * GROUPS, splits * 4, st>>>(o, m, out, splits, rows, heads, K)
  if (splits < 8) {
    if (form == kRowsBf16) TTB_COMBINE(kRowsBf16, 1);
    else if (form == kHeadsBf16) TTB_COMBINE(kHeadsBf16, 1);
    else TTB_COMBINE(kRowsF32, 1);
  } else {
    if (form == kRowsBf16) TTB_COMBINE(kRowsBf16, 4);
    else if (form == kHeadsBf16) TTB_COMBINE(kHeadsBf16, 4);
    else TTB_COMBINE(kRowsF32, 4);
  }
#undef TTB_COMBINE
  return cudaGetLastError() == cudaSuccess ? kOk : kErrDriver;
}

// x [heads, rows, N] -> out [rows, heads*N], multiplied by the sigmoid of the gate (bf16)
extern "C" int ttb_latent_gate_rows(const void* x, const void* gate, long long gate_ld, void* out, int rows, int heads, int N, void* stream) {
  if (rows <= 0 || heads <= 0 || N <= 0) return kErrBadShape;
  const long long total = static_cast<long long>(rows) * heads * N;
  const long long cap = static_cast<long long>(sm_count()) * 16;
  const long long blocks = (total + 255) / 256;
  TTB_COUNT_LAUNCH(1);
  latent_gate_rows_kernel<<<static_cast<int>(blocks < cap ? blocks : cap), 256, 0, static_cast<cudaStream_t>(stream)>>>(
      static_cast<const __nv_bfloat16*>(x), static_cast<const __nv_bfloat16*>(gate), gate_ld, static_cast<__nv_bfloat16*>(out), rows, heads, N);
  return cudaGetLastError() == cudaSuccess ? kOk : kErrDriver;
}

extern "C" int ttb_latent_attention_any(const void* q, long long q_b, long long q_i, long long q_h, const void* k1, long long k1_b, long long k1_j, long long k1_h,
                                        const void* k2, long long k2_b, long long k2_j, const void* v, long long v_b, long long v_j, long long v_h, void* o,
                                        float* ml, const void* gate, long long gate_ld, int b, int s, int sk, int heads, int group, int d1, int d2, int dv,
                                        int heads_as_rows, int out_f32, const int* slot, int slot_host, const int* lo, long long lo_row, long long lo_query, const int* hi,
                                        long long hi_row, long long hi_query, float scale, int wide, void* stream) {
  if (b <= 0 || s <= 0 || sk <= 0 || heads <= 0 || group <= 0 || heads % group || d1 < 0 || d2 < 0 || d1 + d2 <= 0 || dv <= 0 || (heads_as_rows && s != 1)) return kErrBadShape;
  AnyParams p{q, q_b, q_i, q_h, k1, k1_b, k1_j, k1_h, k2, k2_b, k2_j, v, v_b, v_j, v_h, o, reinterpret_cast<float2*>(ml), gate, gate_ld,
              b, s, sk, heads, d1, d2, dv, group, heads_as_rows, out_f32, 32, slot, slot_host, lo, lo_row, lo_query, hi, hi_row, hi_query, scale};
  const int d = d1 + d2;
  auto need = [&](int kt) { return (kAnyRows * d + kt * (d + 1) + kt * dv + kAnyRows * dv + kAnyRows * kt + 3 * kAnyRows) * 4; };
  while (p.key_tile > 1 && need(p.key_tile) > kSmemMax - 1024) p.key_tile /= 2;
  const int smem = need(p.key_tile);
  if (smem > kSmemMax - 1024) return kErrTooLarge;
  static int gf = 0, gb = 0;
  if (!(wide ? allow_smem(latent_attention_any_kernel<float>, smem, gf) : allow_smem(latent_attention_any_kernel<__nv_bfloat16>, smem, gb))) return kErrDriver;
  const int rows = heads_as_rows ? group : s, other = heads_as_rows ? heads / group : heads;
  if (other > 65535 || b > 65535) return kErrTooLarge;
  const dim3 grid((rows + kAnyRows - 1) / kAnyRows, other, b);
  auto st = static_cast<cudaStream_t>(stream);
  TTB_COUNT_LAUNCH(1);
  if (wide) latent_attention_any_kernel<float><<<grid, 128, smem, st>>>(p);
  else latent_attention_any_kernel<__nv_bfloat16><<<grid, 128, smem, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? kOk : kErrDriver;
}
