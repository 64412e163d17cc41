// Linear attention with one decay per head: S_t = d S_{t-1} + k_t v_t^T, o_t = S_t^T q_t, the state S [dim, vdim] in fp32.
//
// * `lightning_recurrent_kernel`: token by token, fp32 arithmetic, for every size and both tensor types.  A CTA owns 32 state columns of one
//   head in registers.  One token per row (decoding) is one pass over the state; SiLU of the three projections is applied on the way in.
//
// * chunks of 128 tokens on tcgen05 tensor cores (bf16, dim and vdim at most 128), the tokens of a head cut into runs of several chunks:
//     lightning_run_state_kernel   what each run adds to the state:     U = sum_j d^(end - 1 - j) k_j v_j^T, accumulated in tensor memory
//     lightning_scan_kernel        state in front of every run (fp32)
//     lightning_run_kernel         run by run, chunk after chunk:  o_i = d^(i+1) S^T q_i + sum_{j<=i} d^(i-j) (q_i k_j) v_j, the state kept in
//                                  tensor memory as an fp32 accumulator
//   The state enters a product only as a pair of bf16 numbers (value and rounding remainder), and so do the decayed values that enter the
//   state, which keeps both at 16 or more bits; decays are applied in fp32.
//
// * `gated_norm_kernel`: o / rms(o) * gain * sigmoid(gate) over all heads of a token; `silu_rows_kernel`: SiLU in place.
//
// Rows that start at a later slot (left padding): tokens in front of starts[row] leave nothing in the state.
#include "common/attn_math.cuh"
#include "common/convert.cuh"
#include "common/ptx.cuh"
#include "common/tmap.h"

namespace ttb {
namespace lightning {

using namespace attn;
using bf16 = __nv_bfloat16;

// ===================================================================================== token by token
struct RecurrentParams {
  const void *q, *k, *v;  // [b * s, ld], head h at column h * dim | h * vdim
  long long ld_q, ld_k, ld_v;
  const float* decay;     // [heads]
  float* state;           // [b, heads, dk, dv], or nullptr: nothing is kept
  float* o;               // [b * s, heads * dv]
  int s, heads, dk, dv, fresh, first;
  const int* starts;      // [b], or nullptr
};

static constexpr int kTokens = 8;

template <typename T>
__device__ __forceinline__ float silu_of(float z) { return z * logistic<T>(z); }

// 256 threads: 8 groups of 4 columns x 32 state rows, ROWS times.
template <typename T, int ROWS>
__global__ void __launch_bounds__(256) lightning_recurrent_kernel(const RecurrentParams p) {
  extern __shared__ float sm[];
  float* sq = sm;                        // [kTokens][dk]
  float* sk = sq + kTokens * p.dk;       // [kTokens][dk]
  float* sv = sk + kTokens * p.dk;       // [kTokens][32]
  float* part = sv + kTokens * 32;       // [kTokens][8][32]
  const int h = blockIdx.y, bi = blockIdx.z, n0 = blockIdx.x * 32;
  const int quad = threadIdx.x & 7, group = threadIdx.x >> 3, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int col = n0 + quad * 4;
  const float decay = p.decay[h];
  float* state = p.state != nullptr ? p.state + (static_cast<long long>(bi) * p.heads + h) * p.dk * p.dv : nullptr;
  const bool vec = p.dv % 4 == 0;
  float S[ROWS][4];
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    const int d = group + 32 * i;
    S[i][0] = S[i][1] = S[i][2] = S[i][3] = 0.f;
    if (!p.fresh && state != nullptr && d < p.dk) {
      const float* src = state + static_cast<long long>(d) * p.dv + col;
      if (vec && col < p.dv) load4(src, S[i]);
      else if (!vec)
        for (int j = 0; j < 4; ++j)
          if (col + j < p.dv) S[i][j] = src[j];
    }
  }
  const int start = p.starts != nullptr ? p.starts[bi] - p.first : 0;  // first own token of this row
  for (int t0 = 0; t0 < p.s; t0 += kTokens) {
    const int n = min(kTokens, p.s - t0);
    for (int i = threadIdx.x; i < n * p.dk; i += 256) {
      const int t = i / p.dk, d = i - t * p.dk;
      const long long row = static_cast<long long>(bi) * p.s + t0 + t;
      sq[i] = silu_of<T>(as_float(static_cast<const T*>(p.q)[row * p.ld_q + h * p.dk + d]));
      sk[i] = t0 + t >= start ? silu_of<T>(as_float(static_cast<const T*>(p.k)[row * p.ld_k + h * p.dk + d])) : 0.f;
    }
    for (int i = threadIdx.x; i < n * 32; i += 256) {
      const int t = i >> 5, c = n0 + (i & 31);
      const long long row = static_cast<long long>(bi) * p.s + t0 + t;
      sv[i] = c < p.dv ? silu_of<T>(as_float(static_cast<const T*>(p.v)[row * p.ld_v + h * p.dv + c])) : 0.f;
    }
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      const float4 v4 = *reinterpret_cast<const float4*>(sv + t * 32 + quad * 4);
      const float v[4] = {v4.x, v4.y, v4.z, v4.w};
      float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int i = 0; i < ROWS; ++i) {
        const int d = group + 32 * i;
        const float kd = d < p.dk ? sk[t * p.dk + d] : 0.f, qd = d < p.dk ? sq[t * p.dk + d] : 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          S[i][j] = decay * S[i][j] + kd * v[j];
          acc[j] += qd * S[i][j];
        }
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        acc[j] += __shfl_xor_sync(0xffffffffu, acc[j], 8);
        acc[j] += __shfl_xor_sync(0xffffffffu, acc[j], 16);
      }
      if (lane < 8) store4(part + (t * 8 + warp) * 32 + quad * 4, acc);
    }
    __syncthreads();
    const int t = threadIdx.x >> 5, c = threadIdx.x & 31;
    if (t < n && n0 + c < p.dv) {
      float sum = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) sum += part[(t * 8 + w) * 32 + c];
      p.o[(static_cast<long long>(bi) * p.s + t0 + t) * p.heads * p.dv + h * p.dv + n0 + c] = sum;
    }
    __syncthreads();
  }
  if (state == nullptr) return;
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    const int d = group + 32 * i;
    if (d >= p.dk) continue;
    float* dst = state + static_cast<long long>(d) * p.dv + col;
    if (vec && col < p.dv) store4(dst, S[i]);
    else if (!vec)
      for (int j = 0; j < 4; ++j)
        if (col + j < p.dv) dst[j] = S[i][j];
  }
}

template <typename T>
static int launch_recurrent(const RecurrentParams& p, int b, cudaStream_t st) {
  const dim3 grid((p.dv + 31) / 32, p.heads, b);
  const int smem = (2 * kTokens * p.dk + kTokens * 32 + kTokens * 8 * 32) * 4;
  TTB_COUNT_LAUNCH(1);
  if (p.dk <= 32) lightning_recurrent_kernel<T, 1><<<grid, 256, smem, st>>>(p);
  else if (p.dk <= 64) lightning_recurrent_kernel<T, 2><<<grid, 256, smem, st>>>(p);
  else if (p.dk <= 128) lightning_recurrent_kernel<T, 4><<<grid, 256, smem, st>>>(p);
  else if (p.dk <= 256) lightning_recurrent_kernel<T, 8><<<grid, 256, smem, st>>>(p);
  else lightning_recurrent_kernel<T, 16><<<grid, 256, smem, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? kOk : kErrDriver;
}

// ===================================================================================== chunks
struct ChunkParams {
  int s, heads, dk, dv;
  int q_panels, v_panels, dk_steps;
  int run_chunks, runs;   // chunks per run, runs per row
  const float* powers;    // [heads, 129]: decay^0 ... decay^128
  const float* chunk_powers;  // [heads, run_chunks + 1]: powers of decay^128
  const float* begin;     // state in front of every run [b, heads, runs, dk, dv], or nullptr: zeros
  float* run_state;       // [b, heads, runs, dk, dv]
  float* state;           // [b, heads, dk, dv] the state behind the last run, or nullptr
  bf16* o;                // [b * s, heads * dv]
  const int* starts;
  int first;
  int* err;
};

static constexpr int kChunkThreads = 384;
static constexpr int kRunThreads = 640;
static constexpr int kTile = 2 * kPanelBytes;  // 128 rows x 128 columns
static constexpr int kRunSmem = 7 * kTile + 1024 + 32 * 8 + 260 * 4;
static constexpr int kRunStateSmem = 6 * kTile + 1024 + 32 * 8 + 132 * 4;
static_assert(kRunSmem <= 227 * 1024 && kRunStateSmem <= 227 * 1024, "shared memory of one CTA");

// f as the sum of two bf16 numbers
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 back = __bfloat1622float2(h);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = pack_bf16x2(a - back.x, b - back.y);
}
__device__ __forceinline__ uint32_t swizzled(int row, int chunk) { return row * 128 + ((chunk ^ (row & 7)) << 4); }

// One row of a 64-column panel of V, times w, as value and remainder.  `hi` may be the panel itself.
__device__ __forceinline__ void scale_panel_row(const uint8_t* v, uint8_t* hi, uint8_t* lo, int row, float w) {
#pragma unroll
  for (int c = 0; c < 8; ++c) {
    const uint32_t at = swizzled(row, c);
    float f[8];
    unpack_bf16x8(*reinterpret_cast<const uint4*>(v + at), f);
    uint4 a, b;
    split2(f[0] * w, f[1] * w, a.x, b.x);
    split2(f[2] * w, f[3] * w, a.y, b.y);
    split2(f[4] * w, f[5] * w, a.z, b.z);
    split2(f[6] * w, f[7] * w, a.w, b.w);
    *reinterpret_cast<uint4*>(hi + at) = a;
    *reinterpret_cast<uint4*>(lo + at) = b;
  }
}

// 32 columns of a state row per lane (rows row0 + lane) <-> the state in memory [dk, dv], 64 bytes of a row at a time.
__device__ __forceinline__ void store_state_piece(float* state, const uint32_t (&v)[32], int row0, int col0, int dk, int dv) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int g = 0; g < 2; ++g) {
    uint4 q[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) q[j] = make_uint4(v[g * 16 + j * 4], v[g * 16 + j * 4 + 1], v[g * 16 + j * 4 + 2], v[g * 16 + j * 4 + 3]);
    transpose_quads(q);
    const int row = row0 + (lane & ~3), col = col0 + g * 16 + (lane & 3) * 4;
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (row + j < dk && col < dv) *reinterpret_cast<uint4*>(state + static_cast<long long>(row + j) * dv + col) = q[j];
  }
}
__device__ __forceinline__ void load_state_piece(const float* state, uint32_t (&v)[32], int row0, int col0, int dk, int dv) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int g = 0; g < 2; ++g) {
    uint4 q[4];
    const int row = row0 + (lane & ~3), col = col0 + g * 16 + (lane & 3) * 4;
#pragma unroll
    for (int j = 0; j < 4; ++j)
      q[j] = state != nullptr && row + j < dk && col < dv ? *reinterpret_cast<const uint4*>(state + static_cast<long long>(row + j) * dv + col) : make_uint4(0u, 0u, 0u, 0u);
    transpose_quads(q);
#pragma unroll
    for (int j = 0; j < 4; ++j) v[g * 16 + j * 4] = q[j].x, v[g * 16 + j * 4 + 1] = q[j].y, v[g * 16 + j * 4 + 2] = q[j].z, v[g * 16 + j * 4 + 3] = q[j].w;
  }
}

// What a whole run adds to the state.  Warp 0 loads, warp 1 issues the products, warps 4 - 11 scale the values.
__global__ void __launch_bounds__(kChunkThreads, 1)
lightning_run_state_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV, const ChunkParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sK = smem;              // [2]
  uint8_t* sV = smem + 2 * kTile;  // [2], scaled in place
  uint8_t* sL = smem + 4 * kTile;  // [2] remainders
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + 6 * kTile);
  uint64_t* full = bars;        // [2]
  uint64_t* ready = bars + 2;   // [2] values scaled
  uint64_t* empty = bars + 4;   // [2]
  uint64_t* done = bars + 6;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 7);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* pw = reinterpret_cast<float*>(bars + 32);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int run = blockIdx.x, h = blockIdx.y, bi = blockIdx.z;
  const int n = p.run_chunks;  // only runs with a successor are computed, and those are whole
  const int tok0 = run * n * kBlk;
  const int start = p.starts != nullptr ? p.starts[bi] - p.first : 0;

  if (threadIdx.x == 0) {
    for (int i = 0; i < 2; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&ready[i], 8);
      mbar_init(&empty[i], 1);
    }
    mbar_init(done, 1);
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (threadIdx.x < kBlk + 1) pw[threadIdx.x] = p.powers[h * (kBlk + 1) + threadIdx.x];
  if (warp == 2) {
    tmem_alloc(tmem_slot, 128);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tH = *tmem_slot;

  if (warp == 0) {
    for (int c = 0; c < n && !*abort_flag; ++c) {
      const int st = c & 1;
      if (!mbar_wait(&empty[st], ((c >> 1) & 1) ^ 1)) {
        fail(abort_flag, p.err, 241);
        break;
      }
      if (lane == 0) {
        mbar_arrive_expect_tx(&full[st], (2 + p.v_panels) * kPanelBytes);
        for (int j = 0; j < 2; ++j) tma_load_4d(sK + st * kTile + j * kPanelBytes, &tmK, &full[st], j * 64, h, tok0 + c * kBlk, bi);
        for (int j = 0; j < p.v_panels; ++j) tma_load_4d(sV + st * kTile + j * kPanelBytes, &tmV, &full[st], j * 64, h, tok0 + c * kBlk, bi);
      }
      __syncwarp();
    }
  } else if (warp == 1) {
    const uint32_t idesc = make_idesc_bf16(128, p.v_panels * 64, true, true);
    bool ok = true;
    for (int c = 0; c < n && ok && !*abort_flag; ++c) {
      const int st = c & 1;
      ok = mbar_wait(&full[st], (c >> 1) & 1) && mbar_wait(&ready[st], (c >> 1) & 1);
      tc_fence_after();
      if (ok && elect_one()) {
        const uint32_t k = smem_u32(sK + st * kTile), v = smem_u32(sV + st * kTile), l = smem_u32(sL + st * kTile);
#pragma unroll
        for (int i = 0; i < kBlk / 16; ++i) umma_f16(tH, desc_mnmajor(k, i), desc_mnmajor(v, i), idesc, (c | i) != 0);
#pragma unroll
        for (int i = 0; i < kBlk / 16; ++i) umma_f16(tH, desc_mnmajor(k, i), desc_mnmajor(l, i), idesc, 1);
        umma_commit(&empty[st]);
        if (c + 1 == n) umma_commit(done);
      }
      __syncwarp();
    }
    if (!ok) fail(abort_flag, p.err, 242);
  } else if (warp >= 4) {
    const int row = (warp & 3) * 32 + lane, panel = (warp - 4) >> 2;
    bool ok = true;
    for (int c = 0; c < n && ok && !*abort_flag; ++c) {
      const int st = c & 1;
      ok = mbar_wait(&full[st], (c >> 1) & 1);
      if (!ok) break;
      const int tok = tok0 + c * kBlk + row;
      const float w = tok >= start ? pw[kBlk - 1 - row] * p.chunk_powers[h * (p.run_chunks + 1) + n - 1 - c] : 0.f;
      if (panel < p.v_panels) {
        uint8_t* v = sV + st * kTile + panel * kPanelBytes;
        scale_panel_row(v, v, sL + st * kTile + panel * kPanelBytes, row, w);
      }
      fence_proxy_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(&ready[st]);
    }
    if (warp < 8) {
      if (ok && !*abort_flag) ok = mbar_wait(done, 0);
      if (ok && !*abort_flag) {
        tc_fence_after();
        float* dst = p.run_state + ((static_cast<long long>(bi) * p.heads + h) * p.runs + run) * p.dk * p.dv;
#pragma unroll 1
        for (int ch = 0; ch < p.v_panels * 2; ++ch) {
          uint32_t v[32];
          tmem_ld_32x32(tH + (static_cast<uint32_t>((warp & 3) * 32) << 16) + ch * 32, v);
          tmem_ld_wait();
          store_state_piece(dst, v, (warp & 3) * 32, ch * 32, p.dk, p.dv);
        }
      }
    }
    if (!ok) fail(abort_flag, p.err, 243);
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  if (warp == 2) tmem_dealloc(tH, 128);
}

// What runs add -> the state in front of each run, in place: work [b, heads, runs, n].
__global__ void __launch_bounds__(256) lightning_scan_kernel(float* __restrict__ work, const float* __restrict__ state, const float* __restrict__ chunk_powers, int heads, int runs,
                                                             int run_chunks, long long n) {
  const int h = blockIdx.y, bi = blockIdx.z;
  const long long i = (blockIdx.x * 256ll + threadIdx.x) * 4;
  if (i >= n) return;
  const float by = chunk_powers[h * (run_chunks + 1) + run_chunks];
  const long long row = static_cast<long long>(bi) * heads + h;
  float cur[4] = {0.f, 0.f, 0.f, 0.f};
  if (state != nullptr) load4(state + row * n + i, cur);
  float* w = work + row * runs * n + i;
  for (int r0 = 0; r0 < runs; r0 += 8) {
    float add[8][4];
#pragma unroll
    for (int r = 0; r < 8; ++r) {  // the loads of eight runs are in flight together
      add[r][0] = add[r][1] = add[r][2] = add[r][3] = 0.f;
      if (r0 + r + 1 < runs) load4(w + (r0 + r) * n, add[r]);
    }
#pragma unroll
    for (int r = 0; r < 8; ++r) {
      if (r0 + r >= runs) break;
      store4(w + (r0 + r) * n, cur);
#pragma unroll
      for (int j = 0; j < 4; ++j) cur[j] = by * cur[j] + add[r][j];
    }
  }
}

// One run of one head.  Warp 0 loads, warp 1 issues the products, warps 4 - 11 turn scores into weights and write the output, warps 12 - 19
// keep the state (each group of four warps has all rows and half of the columns): once per chunk its two bf16 parts go to shared memory for the product with the queries, it is decayed in place, and the
// scaled values (also in two parts, in the same shared memory) are multiplied onto it.
__global__ void __launch_bounds__(kRunThreads, 1)
lightning_run_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV, const ChunkParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;
  uint8_t* sK = smem + kTile;      // [2]
  uint8_t* sV = smem + 3 * kTile;  // [2]
  uint8_t* sX = smem + 5 * kTile;  // state, then scaled values
  uint8_t* sY = smem + 6 * kTile;  // their remainders
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + 7 * kTile);
  uint64_t* q_full = bars;
  uint64_t* q_empty = bars + 1;
  uint64_t* k_full = bars + 2;    // [2]
  uint64_t* v_full = bars + 4;    // [2]
  uint64_t* kv_empty = bars + 6;  // [2]
  uint64_t* s_full = bars + 8;
  uint64_t* p_full = bars + 9;
  uint64_t* st_full = bars + 10;  // state parts written, state decayed
  uint64_t* t_done = bars + 11;   // the product with the state has read them
  uint64_t* vs_full = bars + 12;  // scaled values written
  uint64_t* h_done = bars + 13;   // state updated
  uint64_t* o_full = bars + 14;
  uint64_t* o_free = bars + 15;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 16);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* pw = reinterpret_cast<float*>(bars + 32) + kBlk;  // powers of the decay: pw[-128 ... -1] = 0, pw[0 ... 128]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int run = blockIdx.x, h = blockIdx.y, bi = blockIdx.z;
  const int tok0 = run * p.run_chunks * kBlk;
  const int n = min(p.run_chunks, (p.s - tok0 + kBlk - 1) / kBlk);
  const int start = p.starts != nullptr ? p.starts[bi] - p.first : 0;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    mbar_init(q_empty, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&v_full[i], 1);
      mbar_init(&kv_empty[i], 1);
    }
    mbar_init(s_full, 1);
    mbar_init(p_full, 8);
    mbar_init(st_full, 8);
    mbar_init(t_done, 1);
    mbar_init(vs_full, 8);
    mbar_init(h_done, 1);
    mbar_init(o_full, 1);
    mbar_init(o_free, 8);
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (threadIdx.x < kBlk + 1) pw[threadIdx.x] = p.powers[h * (kBlk + 1) + threadIdx.x];
  else if (threadIdx.x < 2 * kBlk + 1) pw[kBlk - static_cast<int>(threadIdx.x)] = 0.f;
  if (warp == 2) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tS = tmem_base, tT = tmem_base + 128, tO = tmem_base + 256, tH = tmem_base + 384;

  if (warp == 0) {
    // ---------------------------------------------------------------- loads
    for (int c = 0; c < n && !*abort_flag; ++c) {
      const int st = c & 1, tok = tok0 + c * kBlk;
      if (!mbar_wait(&kv_empty[st], ((c >> 1) & 1) ^ 1)) {
        fail(abort_flag, p.err, 251);
        break;
      }
      if (lane == 0) {
        mbar_arrive_expect_tx(&k_full[st], kTile);
        for (int j = 0; j < 2; ++j) tma_load_4d(sK + st * kTile + j * kPanelBytes, &tmK, &k_full[st], j * 64, h, tok, bi);
        mbar_arrive_expect_tx(&v_full[st], p.v_panels * kPanelBytes);
        for (int j = 0; j < p.v_panels; ++j) tma_load_4d(sV + st * kTile + j * kPanelBytes, &tmV, &v_full[st], j * 64, h, tok, bi);
      }
      __syncwarp();
      if (!mbar_wait(q_empty, (c & 1) ^ 1)) {
        fail(abort_flag, p.err, 252);
        break;
      }
      if (lane == 0) {
        mbar_arrive_expect_tx(q_full, p.q_panels * kPanelBytes);
        for (int j = 0; j < p.q_panels; ++j) tma_load_4d(sQ + j * kPanelBytes, &tmQ, q_full, j * 64, h, tok, bi);
      }
      __syncwarp();
    }
  } else if (warp == 1) {
    // ---------------------------------------------------------------- products
    constexpr uint32_t idesc_s = make_idesc_bf16(128, 128, false, false);
    const int N = p.v_panels * 64;
    const uint32_t idesc_o = make_idesc_bf16(128, N, false, true), idesc_h = make_idesc_bf16(128, N, true, true);
    const uint32_t aQ = smem_u32(sQ), aX = smem_u32(sX), aY = smem_u32(sY);
    bool ok = true;
    for (int c = 0; c < n && ok && !*abort_flag; ++c) {
      const int st = c & 1;
      const uint32_t ph = c & 1, kv_ph = (c >> 1) & 1;
      const uint32_t aK = smem_u32(sK + st * kTile), aV = smem_u32(sV + st * kTile);
      // scores; the weights of the previous chunk, which lie in the same columns, have been read by then: products run in issue order
      ok = mbar_wait(q_full, ph) && mbar_wait(&k_full[st], kv_ph);
      tc_fence_after();
      if (ok && elect_one()) {
        for (int i = 0; i < p.dk_steps; ++i) umma_f16(tS, desc_kmajor(aQ, i), desc_kmajor(aK, i), idesc_s, i != 0);
        umma_commit(s_full);
      }
      __syncwarp();
      // queries times the state in front of the chunk
      ok = ok && mbar_wait(st_full, ph) && (c == 0 || mbar_wait(o_free, ph ^ 1));
      tc_fence_after();
      if (ok && elect_one()) {
        for (int i = 0; i < p.dk_steps; ++i) umma_f16(tT, desc_kmajor(aQ, i), desc_mnmajor(aX, i), idesc_o, i != 0);
        for (int i = 0; i < p.dk_steps; ++i) umma_f16(tT, desc_kmajor(aQ, i), desc_mnmajor(aY, i), idesc_o, 1);
        umma_commit(q_empty);
        umma_commit(t_done);
      }
      __syncwarp();
      // weights times values
      ok = ok && mbar_wait(p_full, ph) && mbar_wait(&v_full[st], kv_ph);
      tc_fence_after();
      if (ok && elect_one()) {
#pragma unroll
        for (int i = 0; i < kBlk / 16; ++i) umma_f16_ts(tO, tS + (i >> 2) * 64 + (i & 3) * 8, desc_mnmajor(aV, i), idesc_o, i != 0);
        umma_commit(o_full);
      }
      __syncwarp();
      // keys times scaled values onto the decayed state
      ok = ok && mbar_wait(vs_full, ph);
      tc_fence_after();
      if (ok && elect_one()) {
#pragma unroll
        for (int i = 0; i < kBlk / 16; ++i) umma_f16(tH, desc_mnmajor(aK, i), desc_mnmajor(aX, i), idesc_h, 1);
#pragma unroll
        for (int i = 0; i < kBlk / 16; ++i) umma_f16(tH, desc_mnmajor(aK, i), desc_mnmajor(aY, i), idesc_h, 1);
        umma_commit(h_done);
        umma_commit(&kv_empty[st]);
      }
      __syncwarp();
    }
    if (!ok) fail(abort_flag, p.err, 253);
  } else if (warp >= 4 && warp < 12) {
    // ---------------------------------------------------------------- weights and output: one query row and 64 keys / one value panel per thread
    const int quarter = warp & 3, r = quarter * 32 + lane, part = (warp - 4) >> 2;
    const uint32_t lane_sel = static_cast<uint32_t>(quarter * 32) << 16;
    bool ok = true;
    for (int c = 0; c < n && ok && !*abort_flag; ++c) {
      const uint32_t ph = c & 1;
      const int tok = tok0 + c * kBlk, lo = start - tok;  // keys lo ... r of this chunk count
      ok = mbar_wait(s_full, ph);
      if (!ok) break;
      tc_fence_after();
      const uint32_t scores = tS + lane_sel + part * 64;
      uint32_t pk[32];
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t sv[32];
        tmem_ld_32x32(scores + half * 32, sv);
        tmem_ld_wait();
        const int j0 = part * 64 + half * 32;
        const float* w = pw + r - j0;
        if (lo > j0) {
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (j0 + i < lo) sv[i] = 0u;
        }
#pragma unroll
        for (int i = 0; i < 32; i += 2) pk[half * 16 + (i >> 1)] = pack_bf16x2(__uint_as_float(sv[i]) * w[-i], __uint_as_float(sv[i + 1]) * w[-i - 1]);
      }
      tmem_st_32x32(scores, pk);  // over this group's own scores
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full);
      ok = mbar_wait(o_full, ph);
      if (!ok) break;
      tc_fence_after();
      const float by = pw[r + 1];
      bf16* dst = p.o + ((static_cast<long long>(bi) * p.s + tok) * p.heads + h) * p.dv;
#pragma unroll 1
      for (int ch = part * 2; ch < part * 2 + 2 && part < p.v_panels; ++ch) {
        uint32_t t[32], o[32];
        tmem_ld_32x32(tT + lane_sel + ch * 32, t);
        tmem_ld_32x32(tO + lane_sel + ch * 32, o);
        tmem_ld_wait();
        uint4 q[4];
#pragma unroll
        for (int g = 0; g < 4; ++g) {
          float f[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) f[i] = by * __uint_as_float(t[g * 8 + i]) + __uint_as_float(o[g * 8 + i]);
          q[g] = pack_bf16x8(f);
        }
        transpose_quads(q);
        const int row = quarter * 32 + (lane & ~3), col = ch * 32 + (lane & 3) * 8;  // dv is a multiple of 8
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (tok + row + j < p.s && col < p.dv) *reinterpret_cast<uint4*>(dst + static_cast<long long>(row + j) * p.heads * p.dv + col) = q[j];
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(o_free);
    }
    if (!ok) fail(abort_flag, p.err, 254);
  } else if (warp >= 12) {
    // ---------------------------------------------------------------- state: one panel of one state row, later of one token's values, per thread
    const int quarter = warp & 3, r = quarter * 32 + lane, part = (warp - 12) >> 2;
    const int first_ch = part * 2, last_ch = part < p.v_panels ? first_ch + 2 : first_ch;  // 32-column pieces
    const uint32_t lane_sel = static_cast<uint32_t>(quarter * 32) << 16;
    const float* begin = p.begin != nullptr ? p.begin + ((static_cast<long long>(bi) * p.heads + h) * p.runs + run) * p.dk * p.dv : nullptr;
    bool ok = true;
    for (int c = 0; c < n && ok && !*abort_flag; ++c) {
      const uint32_t ph = c & 1;
      const int tok = tok0 + c * kBlk, count = min(kBlk, p.s - tok);
      if (c > 0) {
        ok = mbar_wait(h_done, ph ^ 1);
        if (!ok) break;
        tc_fence_after();
      }
      const float by = pw[count];
#pragma unroll 1
      for (int ch = first_ch; ch < last_ch; ++ch) {
        uint32_t v[32];
        if (c > 0) {
          tmem_ld_32x32(tH + lane_sel + ch * 32, v);
          tmem_ld_wait();
        } else {
          load_state_piece(begin, v, quarter * 32, ch * 32, p.dk, p.dv);
        }
        uint8_t* x = sX + (ch >> 1) * kPanelBytes;
        uint8_t* y = sY + (ch >> 1) * kPanelBytes;
#pragma unroll
        for (int g = 0; g < 4; ++g) {
          uint4 a, b;
          const uint32_t* u = v + g * 8;
          split2(__uint_as_float(u[0]), __uint_as_float(u[1]), a.x, b.x);
          split2(__uint_as_float(u[2]), __uint_as_float(u[3]), a.y, b.y);
          split2(__uint_as_float(u[4]), __uint_as_float(u[5]), a.z, b.z);
          split2(__uint_as_float(u[6]), __uint_as_float(u[7]), a.w, b.w);
          const uint32_t at = swizzled(r, (ch & 1) * 4 + g);
          *reinterpret_cast<uint4*>(x + at) = a;
          *reinterpret_cast<uint4*>(y + at) = b;
        }
#pragma unroll
        for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * by);
        tmem_st_32x32(tH + lane_sel + ch * 32, v);
      }
      tmem_st_wait();
      fence_proxy_async_smem();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(st_full);
      const int st = c & 1;
      ok = mbar_wait(&v_full[st], (c >> 1) & 1) && mbar_wait(t_done, ph);
      if (!ok) break;
      const float w = r < count && tok + r >= start ? pw[count - 1 - r] : 0.f;
      if (part < p.v_panels) scale_panel_row(sV + st * kTile + part * kPanelBytes, sX + part * kPanelBytes, sY + part * kPanelBytes, r, w);
      fence_proxy_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(vs_full);
    }
    if (ok && !*abort_flag) ok = mbar_wait(h_done, (n - 1) & 1);
    if (ok && !*abort_flag && p.state != nullptr && run + 1 == p.runs) {
      tc_fence_after();
      float* dst = p.state + (static_cast<long long>(bi) * p.heads + h) * p.dk * p.dv;
#pragma unroll 1
      for (int ch = first_ch; ch < last_ch; ++ch) {
        uint32_t v[32];
        tmem_ld_32x32(tH + lane_sel + ch * 32, v);
        tmem_ld_wait();
        store_state_piece(dst, v, quarter * 32, ch * 32, p.dk, p.dv);
      }
    }
    if (!ok) fail(abort_flag, p.err, 255);
  }

  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  if (warp == 2) tmem_dealloc(tmem_base, 512);
}

static int chunk_map(CUtensorMap* m, const void* base, int cols, int heads, int s, int b, long long ld) {
  const uint64_t row = static_cast<uint64_t>(ld) * 2;
  return make_tmap_4d(m, base, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, {static_cast<uint64_t>(cols), static_cast<uint64_t>(heads), static_cast<uint64_t>(s), static_cast<uint64_t>(b)},
                      {static_cast<uint64_t>(cols) * 2, row, row * s}, {64, 1, kBlk, 1}, CU_TENSOR_MAP_SWIZZLE_128B);
}

// ===================================================================================== element-wise steps
__global__ void __launch_bounds__(256) silu_rows_kernel(bf16* __restrict__ x, long long rows, long long ld, int width) {
  const int per = width >> 3;
  const long long total = rows * per;
  for (long long i = blockIdx.x * 256ll + threadIdx.x; i < total; i += gridDim.x * 256ll) {
    const long long r = i / per;
    uint4* at = reinterpret_cast<uint4*>(x + r * ld + (i - r * per) * 8);
    float f[8];
    unpack_bf16x8(*at, f);
#pragma unroll
    for (int j = 0; j < 8; ++j) f[j] = silu_of<bf16>(f[j]);
    *at = pack_bf16x8(f);
  }
}

// V > 0: width % 4 == 0 and width <= 1024 * V, the row waits in registers for its sum of squares.  V == 0: any width, the row is read again.
template <typename O, typename T, int V>
__global__ void __launch_bounds__(256) gated_norm_kernel(const O* __restrict__ o, const T* __restrict__ gain, const T* __restrict__ gate, long long ld_gate, T* __restrict__ out,
                                                         int width, float eps) {
  __shared__ float scratch[8];
  const long long row = blockIdx.x;
  const O* src = o + row * width;
  const T* g = gate + row * ld_gate;
  const float inv = 1.f / static_cast<float>(width);
  float ss = 0.f;
  if constexpr (V > 0) {
    float f[V][4], z[V][4];
#pragma unroll
    for (int k = 0; k < V; ++k) {
      const int i = (threadIdx.x + k * 256) * 4;
      f[k][0] = f[k][1] = f[k][2] = f[k][3] = 0.f;
      if (i < width) {
        load4(src + i, f[k]);
        load4(g + i, z[k]);
      }
    }
#pragma unroll
    for (int k = 0; k < V; ++k)
#pragma unroll
      for (int j = 0; j < 4; ++j) ss += f[k][j] * f[k][j];
    const float rs = 1.f / sqrtf(cta_sum<256>(ss, scratch) * inv + eps);
#pragma unroll
    for (int k = 0; k < V; ++k) {
      const int i = (threadIdx.x + k * 256) * 4;
      if (i >= width) continue;
      float w[4];
      load4(gain + i, w);
#pragma unroll
      for (int j = 0; j < 4; ++j) w[j] = f[k][j] * rs * w[j] * logistic<T>(z[k][j]);
      store4(out + row * width + i, w);
    }
  } else {
    for (int i = threadIdx.x; i < width; i += 256) {
      const float f = as_float(src[i]);
      ss += f * f;
    }
    const float rs = 1.f / sqrtf(cta_sum<256>(ss, scratch) * inv + eps);
    for (int i = threadIdx.x; i < width; i += 256) out[row * width + i] = float_as<T>(as_float(src[i]) * rs * as_float(gain[i]) * logistic<T>(as_float(g[i])));
  }
}

template <typename O, typename T>
static int launch_gated_norm(const void* o, const void* gain, const void* gate, long long ld_gate, void* out, long long rows, int width, float eps, cudaStream_t st) {
  const bool vec = width % 4 == 0 && ld_gate % 4 == 0 &&
                   !((reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(gain) | reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(out)) & 15);
  TTB_COUNT_LAUNCH(1);
#define TTB_GATED_NORM(V)                                                                                                                                                        \
  gated_norm_kernel<O, T, V><<<static_cast<unsigned>(rows), 256, 0, st>>>(static_cast<const O*>(o), static_cast<const T*>(gain), static_cast<const T*>(gate), ld_gate, \
                                                                          static_cast<T*>(out), width, eps)
  if (!vec || width > 8192) TTB_GATED_NORM(0);
  else if (width <= 1024) TTB_GATED_NORM(1);
  else if (width <= 2048) TTB_GATED_NORM(2);
  else if (width <= 4096) TTB_GATED_NORM(4);
  else TTB_GATED_NORM(8);
#undef TTB_GATED_NORM
  return cudaGetLastError() == cudaSuccess ? kOk : kErrDriver;
}

}  // namespace lightning
}  // namespace ttb

using namespace ttb;
using namespace ttb::lightning;

// Token by token.  `wide`: q, k, v are fp32, else bf16.  `fresh`: the state starts at zero whatever the buffer holds.  Token t of a row sits in
// slot first + t and belongs to the row from slot starts[row] on.
extern "C" int ttb_lightning_recurrent(const void* q, long long ld_q, const void* k, long long ld_k, const void* v, long long ld_v, const float* decay, float* state, float* o, int b, int s,
                                       int heads, int dk, int dv, int fresh, const int* starts, int first, int wide, void* stream) {
  if (b <= 0 || s <= 0 || heads <= 0 || dk <= 0 || dv <= 0 || b > 65535 || heads > 65535) return kErrBadShape;
  if (dk > 512) return kErrTooLarge;
  const RecurrentParams p{q, k, v, ld_q, ld_k, ld_v, decay, state, o, s, heads, dk, dv, fresh, first, starts};
  auto st = static_cast<cudaStream_t>(stream);
  return wide ? launch_recurrent<float>(p, b, st) : launch_recurrent<bf16>(p, b, st);
}

// In chunks of 128 tokens, bf16, SiLU already applied.  `work` [b, heads, runs, dk, dv] fp32 with runs = ceil(ceil(s / 128) / run_chunks); unused with one run.
extern "C" int ttb_lightning_chunks(const void* q, long long ld_q, const void* k, long long ld_k, const void* v, long long ld_v, const float* powers, const float* chunk_powers,
                                    float* state, float* work, void* o, int b, int s, int heads, int dk, int dv, int run_chunks, int fresh, const int* starts, int first, int* err,
                                    void* stream) {
  if (b <= 0 || s <= 0 || heads <= 0 || dk <= 0 || dv <= 0 || (dk & 7) || (dv & 7) || run_chunks <= 0 || b > 65535 || heads > 65535 || (reinterpret_cast<uintptr_t>(o) & 15)) return kErrBadShape;
  if (dk > 128 || dv > 128) return kErrTooLarge;
  ChunkParams p{};
  p.s = s, p.heads = heads, p.dk = dk, p.dv = dv;
  p.q_panels = (dk + 63) / 64, p.v_panels = (dv + 63) / 64, p.dk_steps = (dk + 15) / 16;
  p.run_chunks = run_chunks, p.runs = ((s + kBlk - 1) / kBlk + run_chunks - 1) / run_chunks;
  p.powers = powers, p.chunk_powers = chunk_powers, p.state = state, p.run_state = work;
  p.o = static_cast<bf16*>(o), p.starts = starts, p.first = first, p.err = err;
  const float* before = fresh ? nullptr : state;
  p.begin = p.runs > 1 ? work : before;
  CUtensorMap tq, tk, tv;
  int rc;
  if ((rc = chunk_map(&tq, q, dk, heads, s, b, ld_q)) != kOk || (rc = chunk_map(&tk, k, dk, heads, s, b, ld_k)) != kOk || (rc = chunk_map(&tv, v, dv, heads, s, b, ld_v)) != kOk) return rc;
  static bool attr = false;
  if (!attr) {
    if (cudaFuncSetAttribute(lightning_run_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kRunSmem) != cudaSuccess) return kErrDriver;
    if (cudaFuncSetAttribute(lightning_run_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kRunStateSmem) != cudaSuccess) return kErrDriver;
    attr = true;
  }
  auto st = static_cast<cudaStream_t>(stream);
  if (p.runs > 1) {
    if (work == nullptr) return kErrBadShape;
    const long long n = static_cast<long long>(dk) * dv;
    TTB_COUNT_LAUNCH(2);
    lightning_run_state_kernel<<<dim3(p.runs - 1, heads, b), kChunkThreads, kRunStateSmem, st>>>(tk, tv, p);
    lightning_scan_kernel<<<dim3(static_cast<unsigned>((n / 4 + 255) / 256), heads, b), 256, 0, st>>>(work, before, chunk_powers, heads, p.runs, run_chunks, n);
  }
  TTB_COUNT_LAUNCH(1);
  lightning_run_kernel<<<dim3(p.runs, heads, b), kRunThreads, kRunSmem, st>>>(tq, tk, tv, p);
  return cudaGetLastError() == cudaSuccess ? kOk : kErrDriver;
}

// SiLU in place on the first `width` columns of rows with pitch ld (bf16).
extern "C" int ttb_silu_rows(void* x, long long rows, long long ld, int width, void* stream) {
  if (rows <= 0 || width <= 0 || (width & 7) || (ld & 7) || (reinterpret_cast<uintptr_t>(x) & 15)) return kErrBadShape;
  const long long blocks = (rows * (width / 8) + 255) / 256, cap = static_cast<long long>(sm_count()) * 16;
  TTB_COUNT_LAUNCH(1);
  silu_rows_kernel<<<static_cast<int>(blocks < cap ? blocks : cap), 256, 0, static_cast<cudaStream_t>(stream)>>>(static_cast<bf16*>(x), rows, ld, width);
  return cudaGetLastError() == cudaSuccess ? kOk : kErrDriver;
}

// o [rows, width] (`o_wide`: fp32, else bf16); gain [width], gate [rows, ld_gate] and out [rows, width] are fp32 if `wide`, else bf16.
extern "C" int ttb_gated_norm(const void* o, int o_wide, const void* gain, const void* gate, long long ld_gate, void* out, long long rows, int width, float eps, int wide, void* stream) {
  if (rows <= 0 || width <= 0 || rows > 0x7fffffffll || (wide && !o_wide)) return kErrBadShape;
  auto st = static_cast<cudaStream_t>(stream);
  if (wide) return launch_gated_norm<float, float>(o, gain, gate, ld_gate, out, rows, width, eps, st);
  return o_wide ? launch_gated_norm<float, bf16>(o, gain, gate, ld_gate, out, rows, width, eps, st) : launch_gated_norm<bf16, bf16>(o, gain, gate, ld_gate, out, rows, width, eps, st);
}
