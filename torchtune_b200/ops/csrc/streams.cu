// Steps of a decoder with several 32-bit residual streams, for bf16 and fp32 sublayers:
//
//   stream_step       x'_t = sum_s mix[s, t] x_s + out[t] * gain * y         y: a sublayer's output
//                     h    = norm(sum_t read[t] x'_t) * (offset + w)         the next sublayer's input
//                     Either line may be left out.  The norm is a layer norm without bias or an RMS norm; everything is fp32.  The
//                     streams are read and written once per sublayer.
//   embed_positions   token embedding + position embedding, summed in fp32
//   clamped_glu       g * sigmoid(alpha * g) * (u + 1) with g = min(gate, limit), u = clamp(up, -limit, limit)
#include "common/convert.cuh"
#include "common/tmap.h"

TTB_DEFINE_VIOLATION_COUNTER(streams)

namespace ttb {
namespace streams {

static constexpr int kMaxStreams = 16;

template <typename T>
struct StepParams {
  const float* x;   // [rows, x_streams, D]
  int x_streams;    // 1: all streams are equal
  const T* y;       // [rows, D], or nullptr: x' = x
  const T* gain;    // [D]
  const T* mix;     // [S, S], [from, to]
  const T* out;     // [S]
  float* x_out;     // [rows, S, D], or nullptr: x' is not needed afterwards.  May not alias x
  const T* read;    // [S], or nullptr: ones
  const T* w;       // [D]
  T* h;             // [rows, D], or nullptr
  int D, S;
  float eps, offset;
  int centered;
};

// One CTA per row, the row's streams in registers between the passes.  D % 4 == 0, D <= 4 * THREADS * V.
template <typename T, int THREADS, int V, int S>
__global__ void __launch_bounds__(THREADS) stream_step_kernel(const StepParams<T> p) {
  __shared__ float scratch[THREADS / 32];
  __shared__ float c_mix[S * S], c_out[S], c_read[S];
  const long long row = blockIdx.x;
  if (threadIdx.x < S * S) c_mix[threadIdx.x] = p.y != nullptr ? as_float(p.mix[threadIdx.x]) : 0.f;
  if (threadIdx.x < S) {
    c_out[threadIdx.x] = p.y != nullptr ? as_float(p.out[threadIdx.x]) : 0.f;
    c_read[threadIdx.x] = p.read != nullptr ? as_float(p.read[threadIdx.x]) : 1.f;
  }
  const int D = p.D;
  const float* x = p.x + row * p.x_streams * D;
  float xv[V][S][4];
#pragma unroll
  for (int k = 0; k < V; ++k) {
    const int i = (threadIdx.x + k * THREADS) * 4;
#pragma unroll
    for (int s = 0; s < S; ++s) {
      if (i >= D) xv[k][s][0] = xv[k][s][1] = xv[k][s][2] = xv[k][s][3] = 0.f;
      else load4(x + (p.x_streams == 1 ? 0 : s) * static_cast<long long>(D) + i, xv[k][s]);
    }
  }
  float u[V][4];
  __syncthreads();
#pragma unroll
  for (int k = 0; k < V; ++k) {
    const int i = (threadIdx.x + k * THREADS) * 4;
    if (p.y != nullptr && i < D) {
      float yv[4], g[4];
      load4(p.y + row * D + i, yv);
      load4(p.gain + i, g);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float z = yv[j] * g[j];
        float n[S];
#pragma unroll
        for (int t = 0; t < S; ++t) {
          n[t] = c_out[t] * z;
#pragma unroll
          for (int s = 0; s < S; ++s) n[t] += c_mix[s * S + t] * xv[k][s][j];
        }
#pragma unroll
        for (int t = 0; t < S; ++t) xv[k][t][j] = n[t];
      }
      if (p.x_out != nullptr) {
#pragma unroll
        for (int t = 0; t < S; ++t) store4(p.x_out + (row * S + t) * D + i, xv[k][t]);
      }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      u[k][j] = 0.f;
#pragma unroll
      for (int t = 0; t < S; ++t) u[k][j] += c_read[t] * xv[k][t][j];
    }
  }
  if (p.h == nullptr) return;
  const float inv_d = 1.f / static_cast<float>(D);
  float mean = 0.f;
  if (p.centered) {
    float sum = 0.f;
#pragma unroll
    for (int k = 0; k < V; ++k)
#pragma unroll
      for (int j = 0; j < 4; ++j) sum += u[k][j];  // columns past D are zero
    mean = cta_sum<THREADS>(sum, scratch) * inv_d;
  }
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < V; ++k) {
    if ((threadIdx.x + k * THREADS) * 4 >= D) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      u[k][j] -= mean;
      ss += u[k][j] * u[k][j];
    }
  }
  const float rs = 1.f / sqrtf(cta_sum<THREADS>(ss, scratch) * inv_d + p.eps);
#pragma unroll
  for (int k = 0; k < V; ++k) {
    const int i = (threadIdx.x + k * THREADS) * 4;
    if (i >= D) continue;
    float w[4], o[4];
    load4(p.w + i, w);
#pragma unroll
    for (int j = 0; j < 4; ++j) o[j] = u[k][j] * rs * (p.offset + w[j]);
    store4(p.h + row * D + i, o);
  }
}

// Any width and up to kMaxStreams streams: every pass recomputes the row from memory.
template <typename T>
__global__ void __launch_bounds__(256) stream_step_any_kernel(const StepParams<T> p) {
  __shared__ float scratch[8];
  __shared__ float c_mix[kMaxStreams * kMaxStreams], c_out[kMaxStreams], c_read[kMaxStreams];
  const int S = p.S, D = p.D;
  const long long row = blockIdx.x;
  for (int i = threadIdx.x; i < S * S; i += 256) c_mix[i] = p.y != nullptr ? as_float(p.mix[i]) : 0.f;
  if (threadIdx.x < S) {
    c_out[threadIdx.x] = p.y != nullptr ? as_float(p.out[threadIdx.x]) : 0.f;
    c_read[threadIdx.x] = p.read != nullptr ? as_float(p.read[threadIdx.x]) : 1.f;
  }
  __syncthreads();
  const float* x = p.x + row * p.x_streams * D;
  auto value = [&](int i, bool store) {
    float u = 0.f;
    const float z = p.y != nullptr ? as_float(p.y[row * D + i]) * as_float(p.gain[i]) : 0.f;
    for (int t = 0; t < S; ++t) {
      float n;
      if (p.y != nullptr) {
        n = c_out[t] * z;
        for (int s = 0; s < S; ++s) n += c_mix[s * S + t] * x[(p.x_streams == 1 ? 0 : s) * static_cast<long long>(D) + i];
        if (store) p.x_out[(row * S + t) * D + i] = n;
      } else {
        n = x[(p.x_streams == 1 ? 0 : t) * static_cast<long long>(D) + i];
      }
      u += c_read[t] * n;
    }
    return u;
  };
  const bool store = p.x_out != nullptr;
  float sum = 0.f;
  for (int i = threadIdx.x; i < D; i += 256) sum += value(i, store);
  if (p.h == nullptr) return;
  const float inv_d = 1.f / static_cast<float>(D);
  const float mean = p.centered ? cta_sum<256>(sum, scratch) * inv_d : 0.f;
  float ss = 0.f;
  for (int i = threadIdx.x; i < D; i += 256) {
    const float d = value(i, false) - mean;
    ss += d * d;
  }
  const float rs = 1.f / sqrtf(cta_sum<256>(ss, scratch) * inv_d + p.eps);
  for (int i = threadIdx.x; i < D; i += 256) p.h[row * D + i] = float_as<T>((value(i, false) - mean) * rs * (p.offset + as_float(p.w[i])));
}

template <typename T, int S>
static bool launch_step_s(const StepParams<T>& p, int rows, cudaStream_t st) {
  const int D = p.D;
  if (D <= 512) stream_step_kernel<T, 128, 1, S><<<rows, 128, 0, st>>>(p);
  else if (D <= 1024) stream_step_kernel<T, 256, 1, S><<<rows, 256, 0, st>>>(p);
  else if (D <= 2048) stream_step_kernel<T, 256, 2, S><<<rows, 256, 0, st>>>(p);
  else if (D <= 4096) stream_step_kernel<T, 512, 2, S><<<rows, 512, 0, st>>>(p);
  else if (D <= 8192) stream_step_kernel<T, 512, 4, S><<<rows, 512, 0, st>>>(p);
  else return false;
  return true;
}

template <typename T>
static int launch_step(const StepParams<T>& p, int rows, cudaStream_t st) {
  const uintptr_t at = reinterpret_cast<uintptr_t>(p.x) | reinterpret_cast<uintptr_t>(p.y) | reinterpret_cast<uintptr_t>(p.gain) | reinterpret_cast<uintptr_t>(p.x_out) |
                       reinterpret_cast<uintptr_t>(p.w) | reinterpret_cast<uintptr_t>(p.h);
  const bool vec = p.D % 4 == 0 && !(at & 15);
  TTB_COUNT_LAUNCH(1);
  bool done = false;
  if (vec && p.S == 1) done = launch_step_s<T, 1>(p, rows, st);
  else if (vec && p.S == 2) done = launch_step_s<T, 2>(p, rows, st);
  else if (vec && p.S == 3) done = launch_step_s<T, 3>(p, rows, st);
  else if (vec && p.S == 4) done = launch_step_s<T, 4>(p, rows, st);
  if (!done) stream_step_any_kernel<T><<<rows, 256, 0, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? kOk : kErrDriver;
}

template <typename T>
static StepParams<T> step_params(const float* x, int x_streams, const void* y, const void* gain, const void* mix, const void* out, float* x_out, const void* read, const void* w, void* h,
                                 int D, int S, float eps, float offset, int centered) {
  return {x, x_streams, static_cast<const T*>(y), static_cast<const T*>(gain), static_cast<const T*>(mix), static_cast<const T*>(out), x_out, static_cast<const T*>(read),
          static_cast<const T*>(w), static_cast<T*>(h), D, S, eps, offset, centered};
}

template <typename T, bool VEC>
__global__ void __launch_bounds__(256) embed_positions_kernel(const long long* __restrict__ ids, const long long* __restrict__ pos, const T* __restrict__ table,
                                                              const T* __restrict__ pos_table, float* __restrict__ out, long long n, int D, long long vocab, long long positions) {
  for (long long t = blockIdx.x; t < n; t += gridDim.x) {
    long long id = ids[t], p = pos[t];
    if (id < 0 || id >= vocab || p < 0 || p >= positions) {  // never read out of bounds: row 0 stands in and the event is counted
      if (threadIdx.x == 0) TTB_NOTE_VIOLATION(streams);
      if (id < 0 || id >= vocab) id = 0;
      if (p < 0 || p >= positions) p = 0;
    }
    const T* a = table + id * D;
    const T* b = pos_table + p * D;
    if constexpr (VEC) {
      for (int i = threadIdx.x * 4; i < D; i += 1024) {
        float u[4], v[4];
        load4(a + i, u);
        load4(b + i, v);
#pragma unroll
        for (int j = 0; j < 4; ++j) u[j] += v[j];
        store4(out + t * D + i, u);
      }
    } else {
      for (int i = threadIdx.x; i < D; i += 256) out[t * D + i] = as_float(a[i]) + as_float(b[i]);
    }
  }
}

template <typename T>
static int launch_embed(const long long* ids, const long long* pos, const void* table, const void* pos_table, float* out, long long n, int D, long long vocab, long long positions,
                        cudaStream_t st) {
  const bool vec = D % 4 == 0 && !((reinterpret_cast<uintptr_t>(table) | reinterpret_cast<uintptr_t>(pos_table) | reinterpret_cast<uintptr_t>(out)) & 15);
  const long long cap = static_cast<long long>(sm_count()) * 16;
  const int grid = static_cast<int>(n < cap ? n : cap);
  auto a = static_cast<const T*>(table);
  auto b = static_cast<const T*>(pos_table);
  TTB_COUNT_LAUNCH(1);
  if (vec) embed_positions_kernel<T, true><<<grid, 256, 0, st>>>(ids, pos, a, b, out, n, D, vocab, positions);
  else embed_positions_kernel<T, false><<<grid, 256, 0, st>>>(ids, pos, a, b, out, n, D, vocab, positions);
  return cudaGetLastError() == cudaSuccess ? kOk : kErrDriver;
}

template <typename T>
__device__ __forceinline__ float clamped_glu_of(float g, float u, float limit, float alpha) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g * logistic<T>(alpha * g) * (u + 1.f);
}

template <typename T, int W>
__global__ void __launch_bounds__(256) clamped_glu_kernel(const T* __restrict__ g, const T* __restrict__ u, T* __restrict__ y, long long rows, int H, long long ldg, long long ldu,
                                                          float limit, float alpha) {
  const int per = H / W;
  const long long total = rows * per;
  for (long long i = blockIdx.x * 256ll + threadIdx.x; i < total; i += gridDim.x * 256ll) {
    const long long r = i / per;
    const int c = static_cast<int>(i - r * per) * W;
    if constexpr (W == 8) {
      float a[8], b[8];
      unpack_bf16x8(*reinterpret_cast<const uint4*>(g + r * ldg + c), a);
      unpack_bf16x8(*reinterpret_cast<const uint4*>(u + r * ldu + c), b);
#pragma unroll
      for (int j = 0; j < 8; ++j) a[j] = clamped_glu_of<T>(a[j], b[j], limit, alpha);
      *reinterpret_cast<uint4*>(y + r * H + c) = pack_bf16x8(a);
    } else {
      y[r * H + c] = float_as<T>(clamped_glu_of<T>(as_float(g[r * ldg + c]), as_float(u[r * ldu + c]), limit, alpha));
    }
  }
}

}  // namespace streams
}  // namespace ttb

using namespace ttb;
using namespace ttb::streams;

// `wide`: sublayer tensors and parameters are fp32, else bf16.  x [rows, x_streams, D] with x_streams S or 1; x_out [rows, S, D] must not
// overlap x.  y == nullptr: x' = x, only h is computed.  h == nullptr: the streams only.
extern "C" int ttb_stream_step(const float* x, int x_streams, const void* y, const void* gain, const void* mix, const void* out, float* x_out, const void* read, const void* w, void* h,
                               int rows, int D, int S, float eps, float offset, int centered, int wide, void* stream) {
  if (rows <= 0 || D <= 0 || S <= 0 || (x_streams != 1 && x_streams != S) || (y == nullptr && h == nullptr) || (h != nullptr && w == nullptr)) return kErrBadShape;
  if (y != nullptr && (gain == nullptr || mix == nullptr || out == nullptr || (h == nullptr && x_out == nullptr))) return kErrBadShape;
  if (S > kMaxStreams) return kErrTooLarge;
  auto st = static_cast<cudaStream_t>(stream);
  if (wide) return launch_step(step_params<float>(x, x_streams, y, gain, mix, out, x_out, read, w, h, D, S, eps, offset, centered), rows, st);
  return launch_step(step_params<__nv_bfloat16>(x, x_streams, y, gain, mix, out, x_out, read, w, h, D, S, eps, offset, centered), rows, st);
}

// out [n, D] fp32 = table[ids] + pos_table[pos]
extern "C" int ttb_embed_positions(const long long* ids, const long long* pos, const void* table, const void* pos_table, float* out, long long n, int D, long long vocab,
                                   long long positions, int wide, void* stream) {
  if (n <= 0 || D <= 0 || vocab <= 0 || positions <= 0) return kErrBadShape;
  auto st = static_cast<cudaStream_t>(stream);
  return wide ? launch_embed<float>(ids, pos, table, pos_table, out, n, D, vocab, positions, st) : launch_embed<__nv_bfloat16>(ids, pos, table, pos_table, out, n, D, vocab, positions, st);
}

// y [rows, H] from gate and up with row pitches ldg, ldu
extern "C" int ttb_clamped_glu(const void* g, const void* u, void* y, long long rows, int H, long long ldg, long long ldu, float limit, float alpha, int wide, void* stream) {
  if (rows <= 0 || H <= 0) return kErrBadShape;
  auto st = static_cast<cudaStream_t>(stream);
  const bool vec = !wide && !((H | ldg | ldu) & 7) && !((reinterpret_cast<uintptr_t>(g) | reinterpret_cast<uintptr_t>(u) | reinterpret_cast<uintptr_t>(y)) & 15);
  const long long items = rows * (vec ? H / 8 : H), blocks = (items + 255) / 256, cap = static_cast<long long>(sm_count()) * 16;
  const int grid = static_cast<int>(blocks < cap ? blocks : cap);
  using bf = __nv_bfloat16;
  TTB_COUNT_LAUNCH(1);
  if (wide)
    clamped_glu_kernel<float, 1><<<grid, 256, 0, st>>>(static_cast<const float*>(g), static_cast<const float*>(u), static_cast<float*>(y), rows, H, ldg, ldu, limit, alpha);
  else if (vec)
    clamped_glu_kernel<bf, 8><<<grid, 256, 0, st>>>(static_cast<const bf*>(g), static_cast<const bf*>(u), static_cast<bf*>(y), rows, H, ldg, ldu, limit, alpha);
  else
    clamped_glu_kernel<bf, 1><<<grid, 256, 0, st>>>(static_cast<const bf*>(g), static_cast<const bf*>(u), static_cast<bf*>(y), rows, H, ldg, ldu, limit, alpha);
  return cudaGetLastError() == cudaSuccess ? kOk : kErrDriver;
}
