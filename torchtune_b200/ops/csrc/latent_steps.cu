// The steps around latent attention, for bf16 and fp32 tensors:
//
//   latent_prepare     one launch per layer after the input projections: norm of the latent, rotation of the shared key part and of
//                      the queries' rotated parts, and the write of the latent row into the cache
//   latent_absorb      q_lat[r, h, :] = W_uk[h]^T q[r, h, :]            (few rows: weight-streaming)
//   latent_value       out[r, h, :] = (W_uv[h] o_lat[r, h, :]) * sigmoid(gate), combining the split-key partials of the decode kernel
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
};

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
  for (int t = threadIdx.x; t < kRows * K; t += 256) {
    const int r = t / K, k = t - r * K;
    sA[t] = r0 + r < R ? to_f(a[(r0 + r) * a_row + static_cast<long long>(h) * a_head + k]) : 0.f;
  }
  __syncthreads();
  const int n = blockIdx.x * 32 * VEC + lane * VEC;
  float acc[kRows][VEC];
#pragma unroll
  for (int r = 0; r < kRows; ++r)
#pragma unroll
    for (int v = 0; v < VEC; ++v) acc[r][v] = 0.f;
  if (n < N) {
    const T* wp = w + static_cast<long long>(h) * K * N + n;
#pragma unroll 4
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

// ------------------------------------------------------------------------------- value projection: contraction along weight rows
// o [splits, R, heads, K] fp32 with ml [splits, R, heads] (log2-domain maximum, sum).  Each CTA first combines the partials of its rows
// in shared memory, then out[r, h, n] = (sum_k c[r, h, k] * w[h * N + n, k]) * sigmoid(gate[r, h * N + n]).
static constexpr int kValueCols = 32;

__device__ __forceinline__ void combine_rows(const float* __restrict__ o, const float2* __restrict__ ml, float* __restrict__ dst, int dst_pitch, int splits, int R,
                                             int heads, int h, int r0, int n_rows, int K, float* wts) {
  // wts [n_rows][splits]: exp2(m_s - m) / sum
  if (static_cast<int>(threadIdx.x) < n_rows) {
    const int r = threadIdx.x;
    float m = -INFINITY, l = 0.f;
    if (r0 + r < R) {
      for (int s = 0; s < splits; ++s) {
        const float2 v = ml[(static_cast<long long>(s) * R + r0 + r) * heads + h];
        if (v.y > 0.f) m = fmaxf(m, v.x);
      }
      for (int s = 0; s < splits; ++s) {
        const float2 v = ml[(static_cast<long long>(s) * R + r0 + r) * heads + h];
        if (v.y > 0.f) l += v.y * exp2f(v.x - m);
      }
    }
    const float inv = l > 0.f ? 1.f / l : 0.f;
    for (int s = 0; s < splits; ++s) {
      const float2 v = r0 + r < R ? ml[(static_cast<long long>(s) * R + r0 + r) * heads + h] : make_float2(0.f, 0.f);
      wts[r * splits + s] = v.y > 0.f ? exp2f(v.x - m) * inv : 0.f;
    }
  }
  __syncthreads();
  for (int t = threadIdx.x; t < n_rows * K; t += blockDim.x) {
    const int r = t / K, k = t - r * K;
    float acc = 0.f;
    if (r0 + r < R) {
      const float* src = o + (static_cast<long long>(r0 + r) * heads + h) * K + k;
      const long long pitch = static_cast<long long>(R) * heads * K;
#pragma unroll 4
      for (int s = 0; s < splits; ++s) {
        const float wt = wts[r * splits + s];
        if (wt != 0.f) acc += wt * src[s * pitch];  // a split without keys has written nothing
      }
    }
    dst[r * dst_pitch + k] = acc;
  }
  __syncthreads();
}

template <typename T, int VEC>
__global__ void __launch_bounds__(256) latent_value_kernel(const float* __restrict__ o, const float2* __restrict__ ml, const T* __restrict__ w,
                                                           const T* __restrict__ gate, long long gate_ld, T* __restrict__ out, int splits, int R, int heads, int K,
                                                           int N) {
  extern __shared__ float sm[];
  float* sA = sm;                 // [kRows][K]
  float* wts = sm + kRows * K;    // [kRows][splits]
  const int h = blockIdx.y, r0 = blockIdx.z * kRows;
  const int n_rows = min(kRows, R - r0);
  combine_rows(o, ml, sA, K, splits, R, heads, h, r0, n_rows, K, wts);
  for (int t = n_rows * K + threadIdx.x; t < kRows * K; t += 256) sA[t] = 0.f;
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int c = warp; c < kValueCols; c += 8) {
    const int n = blockIdx.x * kValueCols + c;
    if (n >= N) break;
    const T* wp = w + (static_cast<long long>(h) * N + n) * K;
    float acc[kRows];
#pragma unroll
    for (int r = 0; r < kRows; ++r) acc[r] = 0.f;
#pragma unroll 4
    for (int k = lane * VEC; k < K; k += 32 * VEC) {
      float f[VEC];
      WVec<T, VEC>::load(wp + k, f);
#pragma unroll
      for (int r = 0; r < kRows; ++r)
#pragma unroll
        for (int v = 0; v < VEC; ++v) acc[r] += sA[r * K + k + v] * f[v];
    }
#pragma unroll
    for (int r = 0; r < kRows; ++r) acc[r] = warp_sum(acc[r]);
    if (lane == 0) {
#pragma unroll
      for (int r = 0; r < kRows; ++r) {
        if (r >= n_rows) continue;
        const long long col = static_cast<long long>(h) * N + n;
        float v = acc[r];
        if (gate != nullptr) v *= sigmoid_as<T>(to_f(gate[(r0 + r) * gate_ld + col]));
        out[static_cast<long long>(r0 + r) * heads * N + col] = from_f<T>(v);
      }
    }
  }
}

// Combined latent outputs only, head-major [heads, R, K] (bf16): the row order of a grouped GEMM whose groups are heads.
__global__ void __launch_bounds__(128) latent_combine_kernel(const float* __restrict__ o, const float2* __restrict__ ml, __nv_bfloat16* __restrict__ out, int splits,
                                                             int R, int heads, int K) {
  extern __shared__ float sm[];
  float* row = sm;
  float* wts = sm + K;
  const int r = blockIdx.x, h = blockIdx.y;
  combine_rows(o, ml, row, K, splits, R, heads, h, r, 1, K, wts);
  for (int k = threadIdx.x; k < K; k += blockDim.x) out[(static_cast<long long>(h) * R + r) * K + k] = __float2bfloat16_rn(row[k]);
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

// 128 threads, 16 rows per CTA: 16 queries of one head, or (heads_as_rows) 16 heads of one query when all heads share keys and values.
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
  const int n_rows = min(kAnyRows, (p.heads_as_rows ? p.heads : p.s) - row0);
  auto query_of = [&](int r) { return p.heads_as_rows ? static_cast<int>(blockIdx.y) : row0 + r; };
  auto head_of = [&](int r) { return p.heads_as_rows ? row0 + r : static_cast<int>(blockIdx.y); };
  const int h_shared = p.heads_as_rows ? 0 : static_cast<int>(blockIdx.y);
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

template <typename T>
static int launch_value(const float* o, const float* ml, const void* w, const void* gate, long long gate_ld, void* out, int splits, int R, int heads, int K, int N,
                        cudaStream_t st) {
  const bool vec = K % 4 == 0 && !(reinterpret_cast<uintptr_t>(w) & 15);
  const int smem = (kRows * K + kRows * splits) * 4;
  static int g4 = 0, g1 = 0;
  if (!(vec ? allow_smem(latent_value_kernel<T, 4>, smem, g4) : allow_smem(latent_value_kernel<T, 1>, smem, g1))) return kErrTooLarge;
  const dim3 grid((N + kValueCols - 1) / kValueCols, heads, (R + kRows - 1) / kRows);
  auto mlp = reinterpret_cast<const float2*>(ml);
  TTB_COUNT_LAUNCH(1);
  if (vec)
    latent_value_kernel<T, 4><<<grid, 256, smem, st>>>(o, mlp, static_cast<const T*>(w), static_cast<const T*>(gate), gate_ld, static_cast<T*>(out), splits, R, heads, K, N);
  else
    latent_value_kernel<T, 1><<<grid, 256, smem, st>>>(o, mlp, static_cast<const T*>(w), static_cast<const T*>(gate), gate_ld, static_cast<T*>(out), splits, R, heads, K, N);
  return cudaGetLastError() == cudaSuccess ? kOk : kErrDriver;
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
  PrepareParams p{kv, ld_kv, kv_gain, q, ld_q, q_out, cache, table, pos, slot, slot_host, s, slots, heads, dim, rot, rot_dims, rank, table_len, eps};
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

// o [splits, rows, heads, K] / ml [splits, rows, heads, 2] fp32, w [heads*N, K]; out [rows, heads*N]
extern "C" int ttb_latent_value(const float* o, const float* ml, const void* w, const void* gate, long long gate_ld, void* out, int splits, int rows, int heads, int K,
                                int N, int wide, void* stream) {
  if (rows <= 0 || heads <= 0 || K <= 0 || N <= 0 || splits <= 0) return kErrBadShape;
  auto st = static_cast<cudaStream_t>(stream);
  return wide ? launch_value<float>(o, ml, w, gate, gate_ld, out, splits, rows, heads, K, N, st)
              : launch_value<__nv_bfloat16>(o, ml, w, gate, gate_ld, out, splits, rows, heads, K, N, st);
}

// bf16, head-major [heads, rows, K]
extern "C" int ttb_latent_combine(const float* o, const float* ml, void* out, int splits, int rows, int heads, int K, void* stream) {
  if (rows <= 0 || heads <= 0 || K <= 0 || splits <= 0 || (K + splits) * 4 > 48 * 1024) return kErrBadShape;
  TTB_COUNT_LAUNCH(1);
  latent_combine_kernel<<<dim3(rows, heads), 128, (K + splits) * 4, static_cast<cudaStream_t>(stream)>>>(o, reinterpret_cast<const float2*>(ml),
                                                                                                       static_cast<__nv_bfloat16*>(out), splits, rows, heads, K);
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
                                        float* ml, const void* gate, long long gate_ld, int b, int s, int sk, int heads, int d1, int d2, int dv, int heads_as_rows,
                                        int out_f32, const int* slot, int slot_host, const int* lo, long long lo_row, long long lo_query, const int* hi,
                                        long long hi_row, long long hi_query, float scale, int wide, void* stream) {
  if (b <= 0 || s <= 0 || sk <= 0 || heads <= 0 || d1 < 0 || d2 < 0 || d1 + d2 <= 0 || dv <= 0) return kErrBadShape;
  AnyParams p{q, q_b, q_i, q_h, k1, k1_b, k1_j, k1_h, k2, k2_b, k2_j, v, v_b, v_j, v_h, o, reinterpret_cast<float2*>(ml), gate, gate_ld,
              b, s, sk, heads, d1, d2, dv, heads_as_rows, out_f32, 32, slot, slot_host, lo, lo_row, lo_query, hi, hi_row, hi_query, scale};
  const int d = d1 + d2;
  auto need = [&](int kt) { return (kAnyRows * d + kt * (d + 1) + kt * dv + kAnyRows * dv + kAnyRows * kt + 3 * kAnyRows) * 4; };
  while (p.key_tile > 1 && need(p.key_tile) > kSmemMax - 1024) p.key_tile /= 2;
  const int smem = need(p.key_tile);
  if (smem > kSmemMax - 1024) return kErrTooLarge;
  static int gf = 0, gb = 0;
  if (!(wide ? allow_smem(latent_attention_any_kernel<float>, smem, gf) : allow_smem(latent_attention_any_kernel<__nv_bfloat16>, smem, gb))) return kErrDriver;
  const int rows = heads_as_rows ? heads : s, other = heads_as_rows ? s : heads;
  if (other > 65535 || b > 65535) return kErrTooLarge;
  const dim3 grid((rows + kAnyRows - 1) / kAnyRows, other, b);
  auto st = static_cast<cudaStream_t>(stream);
  TTB_COUNT_LAUNCH(1);
  if (wide) latent_attention_any_kernel<float><<<grid, 128, smem, st>>>(p);
  else latent_attention_any_kernel<__nv_bfloat16><<<grid, 128, smem, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? kOk : kErrDriver;
}
