// Attention over latent keys (multi-head latent attention) on tcgen05 tensor cores.
//
// A token leaves one latent c (`rank` values) and one rotated key part r (`rot` values, shared by all heads) in the cache.  Per head
//   score(i, j) = (q_i · W_uk c_j + rot(q)_i · r_j) * scale,     out_i = Σ_j softmax_j W_uv c_j.
//
// Two kernels, one per side of the trade between expanding keys and absorbing W_uk into the query:
//
// * prefill (`latent_prefill_kernel`): many queries per sequence.  W_uk c and W_uv c have been expanded by one GEMM; the key of a head
//   is the pair (expanded part, shared rotated part), which two tensor maps bring into one shared-memory tile as consecutive 64-column
//   panels, so the concatenated key is never written to memory.  Three-dimensional maps with the true inner extent let TMA zero-fill
//   the last panel: `dim`, `rot` and `vdim` need not be multiples of 64.  Two 128-row query tiles per CTA, scores, probabilities and
//   outputs in tensor memory (the scheme of attention_fwd2.cu); the epilogue multiplies by the sigmoid of a gate row.
//
// * decode (`latent_decode_kernel`): one query per sequence, queries already multiplied by W_ukᵀ.  All heads share the keys, so a
//   tile of cached rows is loaded once and used twice: Sᵀ = C · Qᵀ (M = keys, N = heads) and Oᵀ += Cᵀ · Pᵀ (M = 128 latent
//   columns, N = heads).  Heads sit in the N dimension, so 16 heads cost 16 columns rather than a padded 128-row tile.  Cache
//   rows are cut over CTAs (split keys); the partial outputs are combined by the value projection.
//
// Grouped-query attention over a key/value cache is the same pair of kernels without the two-part key: in prefill the second key part is
// empty and `group` query heads read one key head; in decode the scores come from the keys alone (the second operand of the latent form,
// up to 256 columns) and the pieces are the values.
//
// Row bounds: key j is visible to query i of batch row b iff lo(b, i) <= j <= hi(b, i), by default 0 <= j <= slot(i).  Every wait is
// bounded and reports through the error word.
#include "common/attn_math.cuh"
#include "common/ptx.cuh"
#include "common/tmap.h"

namespace ttb {
namespace latent {

using namespace attn;

__device__ __forceinline__ float sigmoid_of(float z) { return 1.f / (1.f + __expf(-z)); }

// ===================================================================================== prefill
struct PrefillParams {
  int b, s, sk, heads;
  int group;          // query heads per head of tmKn / tmV
  int slot0;          // cache slot of query 0 (sk = slot0 + s keys exist)
  int dim_panels, rot_panels, v_panels;
  int dim_steps, rot_steps;  // contraction steps of 16 columns
  int k_stages, v_stages;
  int vdim;
  float scale;
  const int* lo;      // lower bound of (batch row bi, query i) at lo[bi * lo_row + i * lo_query], or nullptr (0)
  long long lo_row, lo_query;
  const int* hi;      // the same for the upper bound, or nullptr (slot0 + i)
  long long hi_row, hi_query;
  const __nv_bfloat16* gate;  // gate of (token, head, column) at gate[token * gate_ld + head * vdim + column], or nullptr
  long long gate_ld;
  __nv_bfloat16* o;  // [b * s, heads * vdim]
  int* err;
};

static constexpr int kPrefillThreads = 384;

__global__ void __launch_bounds__(kPrefillThreads, 1)
latent_prefill_kernel(const __grid_constant__ CUtensorMap tmQn, const __grid_constant__ CUtensorMap tmQr, const __grid_constant__ CUtensorMap tmKn,
                      const __grid_constant__ CUtensorMap tmKr, const __grid_constant__ CUtensorMap tmV, PrefillParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int k_panels = p.dim_panels + p.rot_panels;
  const int q_bytes = k_panels * kPanelBytes, v_bytes = p.v_panels * kPanelBytes;
  uint8_t* sQ = smem;                                 // [2] query tiles
  uint8_t* sK = sQ + 2 * q_bytes;                     // [k_stages]
  uint8_t* sV = sK + p.k_stages * q_bytes;            // [v_stages]
  uint64_t* bars = reinterpret_cast<uint64_t*>(sV + p.v_stages * v_bytes);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;
  uint64_t* k_empty = bars + 3;
  uint64_t* v_full = bars + 5;
  uint64_t* v_empty = bars + 7;
  uint64_t* s_full = bars + 9;
  uint64_t* p_full = bars + 11;
  uint64_t* o_done = bars + 13;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 15);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, bi = blockIdx.z;
  const int q0 = (gridDim.x - 1 - blockIdx.x) * 2 * kBlk;  // the longest rows of a causal pattern start first
  const int row_base = bi * p.s;
  const int hk = h / p.group;
  auto lo_of = [&](int i) { return p.lo != nullptr ? p.lo[bi * p.lo_row + i * p.lo_query] : 0; };
  auto hi_of = [&](int i) { return p.hi != nullptr ? p.hi[bi * p.hi_row + i * p.hi_query] : p.slot0 + i; };

  int begin[2], count[2];
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    const int qa = q0 + x * kBlk;
    begin[x] = 0, count[x] = 0;
    if (qa >= p.s) continue;
    const int qz = min(qa + kBlk, p.s) - 1;
    const int end_tok = min(p.sk, hi_of(qz) + 1);
    begin[x] = max(lo_of(qa), 0) / kBlk;
    count[x] = max((end_tok + kBlk - 1) / kBlk - begin[x], 0);
  }
  int u_begin, u_end;
  if (count[0] > 0 && count[1] > 0) {
    u_begin = min(begin[0], begin[1]);
    u_end = max(begin[0] + count[0], begin[1] + count[1]);
  } else if (count[0] > 0) {
    u_begin = begin[0], u_end = begin[0] + count[0];
  } else {
    u_begin = begin[1], u_end = begin[1] + count[1];
  }
  const int n_union = u_end - u_begin;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
      mbar_init(&v_full[i], 1);
      mbar_init(&v_empty[i], 1);
      mbar_init(&s_full[i], 1);
      mbar_init(&p_full[i], 4);
      mbar_init(&o_done[i], 1);
    }
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 2) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tS[2] = {tmem_base, tmem_base + 128};
  const uint32_t tO[2] = {tmem_base + 256, tmem_base + 384};

  if (warp == 0) {
    // ---------------------------------------------------------------- TMA producer
    if (lane == 0 && n_union > 0) {
      mbar_arrive_expect_tx(q_full, 2 * q_bytes);
      for (int x = 0; x < 2; ++x) {
        uint8_t* dst = sQ + x * q_bytes;
        for (int j = 0; j < p.dim_panels; ++j) tma_load_3d(dst + j * kPanelBytes, &tmQn, q_full, j * 64, h, row_base + q0 + x * kBlk);
        for (int j = 0; j < p.rot_panels; ++j) tma_load_3d(dst + (p.dim_panels + j) * kPanelBytes, &tmQr, q_full, j * 64, h, row_base + q0 + x * kBlk);
      }
    }
    int ks = 0, vs = 0;
    uint32_t kph = 0, vph = 0;
    for (int i = 0; i < n_union && !*abort_flag; ++i) {
      const int kv0 = (u_begin + i) * kBlk;
      if (!mbar_wait(&k_empty[ks], kph ^ 1)) {
        fail(abort_flag, p.err, 221);
        break;
      }
      if (lane == 0) {
        uint8_t* dst = sK + ks * q_bytes;
        mbar_arrive_expect_tx(&k_full[ks], q_bytes);
        for (int j = 0; j < p.dim_panels; ++j) tma_load_4d(dst + j * kPanelBytes, &tmKn, &k_full[ks], j * 64, hk, kv0, bi);
        for (int j = 0; j < p.rot_panels; ++j) tma_load_4d(dst + (p.dim_panels + j) * kPanelBytes, &tmKr, &k_full[ks], j * 64, 0, kv0, bi);
      }
      __syncwarp();
      if (!mbar_wait(&v_empty[vs], vph ^ 1)) {
        fail(abort_flag, p.err, 222);
        break;
      }
      if (lane == 0) {
        uint8_t* dst = sV + vs * v_bytes;
        mbar_arrive_expect_tx(&v_full[vs], v_bytes);
        for (int j = 0; j < p.v_panels; ++j) tma_load_4d(dst + j * kPanelBytes, &tmV, &v_full[vs], j * 64, hk, kv0, bi);
      }
      __syncwarp();
      if (++ks == p.k_stages) ks = 0, kph ^= 1;
      if (++vs == p.v_stages) vs = 0, vph ^= 1;
    }
  } else if (warp == 1) {
    // ---------------------------------------------------------------- MMA issuer (an elected lane: the compiler then keeps descriptors uniform)
    constexpr uint32_t idesc_s = make_idesc_bf16(128, 128, false, false);
    const uint32_t idesc_o = make_idesc_bf16(128, p.v_panels * 64, false, true);
    const uint32_t aQ = smem_u32(sQ), aK = smem_u32(sK), aV = smem_u32(sV);
    bool ok = n_union == 0 || mbar_wait(q_full, 0);
    int k_ready = u_begin - 1, v_ready = u_begin - 1;
    auto active = [&](int x, int j) { return count[x] > 0 && j >= begin[x] && j < begin[x] + count[x]; };
    auto issue_s = [&](int x, int j) -> bool {
      const int i = j - u_begin, st = i % p.k_stages;
      if (j > k_ready) {
        if (!mbar_wait(&k_full[st], (i / p.k_stages) & 1)) return false;
        k_ready = j;
      }
      tc_fence_after();
      if (elect_one()) {
        const uint32_t q_base = aQ + x * q_bytes, k_base = aK + st * q_bytes;
        for (int k = 0; k < p.dim_steps; ++k) umma_f16(tS[x], desc_kmajor(q_base, k), desc_kmajor(k_base, k), idesc_s, k != 0);
        const uint32_t off = p.dim_panels * kPanelBytes;
        for (int k = 0; k < p.rot_steps; ++k) umma_f16(tS[x], desc_kmajor(q_base + off, k), desc_kmajor(k_base + off, k), idesc_s, 1);
        umma_commit(&s_full[x]);
        const bool other_later = (x == 0) && active(1, j);  // tile 1 issues its S(j) after tile 0's
        if (!other_later) umma_commit(&k_empty[st]);
      }
      __syncwarp();
      return true;
    };
    for (int j = u_begin; j < u_end && ok && !*abort_flag; ++j) {
      for (int x = 0; x < 2 && ok; ++x)
        if (active(x, j) && j == begin[x]) ok = issue_s(x, j);
      for (int x = 0; x < 2 && ok; ++x) {
        if (!active(x, j)) continue;
        const int n = j - begin[x];
        const int i = j - u_begin, st = i % p.v_stages;
        if (!mbar_wait(&p_full[x], n & 1)) {
          ok = false;
          break;
        }
        if (j > v_ready) {
          if (!mbar_wait(&v_full[st], (i / p.v_stages) & 1)) {
            ok = false;
            break;
          }
          v_ready = j;
        }
        tc_fence_after();
        if (elect_one()) {
          const uint64_t dv = desc_mnmajor(aV + st * v_bytes, 0);
#pragma unroll
          for (int k = 0; k < kBlk / 16; ++k) umma_f16_ts(tO[x], tS[x] + k * 8, dv + k * (2048 >> 4), idesc_o, (n | k) != 0);
          const bool other_later = (x == 0) && active(1, j);
          if (!other_later) umma_commit(&v_empty[st]);
          if (n + 1 == count[x]) umma_commit(&o_done[x]);
        }
        __syncwarp();
        if (n + 1 < count[x]) ok = issue_s(x, j + 1);
      }
    }
    if (!ok) fail(abort_flag, p.err, 223);
  } else if (warp >= 4) {
    // ---------------------------------------------------------------- softmax / correction / epilogue, one warpgroup per tile
    const int x = (warp - 4) >> 2;
    const int quarter = warp & 3;
    const int r = quarter * 32 + lane;
    const int qa = q0 + x * kBlk;
    const int q_idx = qa + r;
    const int q_last = min(qa + kBlk, p.s) - 1;
    const uint32_t lane_sel = static_cast<uint32_t>(quarter * 32) << 16;
    const bool row_valid = q_idx < p.s;
    const bool tile_valid = qa < p.s;
    const int lo_row = row_valid ? lo_of(q_idx) : 0;
    const int hi_row = row_valid ? hi_of(q_idx) : -1;
    const int lo_max = tile_valid ? lo_of(q_last) : 0;
    const int hi_min = tile_valid ? hi_of(qa) : -1;
    const bool ragged_rows = qa + kBlk > p.s;
    const float c = p.scale * kLog2e;
    float m_used = -INFINITY, l = 0.f;
    bool ok = true;
    for (int n = 0; n < count[x] && !*abort_flag; ++n) {
      const int kv0 = (begin[x] + n) * kBlk;
      if (!mbar_wait(&s_full[x], n & 1)) {
        ok = false;
        break;
      }
      tc_fence_after();
      const bool need_mask = ragged_rows || (kv0 + kBlk - 1 > hi_min) || (kv0 < lo_max) || (kv0 + kBlk > p.sk);
      uint32_t sv[4][32];
#pragma unroll
      for (int ch = 0; ch < 4; ++ch) tmem_ld_32x32(tS[x] + lane_sel + ch * 32, sv[ch]);
      tmem_ld_wait();
      // raw scores in registers; a negative scale would turn the maximum around, so it is folded in here only when positive
      if (p.scale <= 0.f) {
#pragma unroll
        for (int ch = 0; ch < 4; ++ch)
#pragma unroll
          for (int i = 0; i < 32; ++i) sv[ch][i] = __float_as_uint(__uint_as_float(sv[ch][i]) * c);
      }
      const float cc = p.scale <= 0.f ? 1.f : c;
      if (need_mask) {
#pragma unroll
        for (int ch = 0; ch < 4; ++ch) {
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const int j = kv0 + ch * 32 + i;
            if (j < lo_row || j > hi_row || j >= p.sk) sv[ch][i] = 0xff800000u;  // -inf
          }
        }
      }
      float mx2[2] = {-INFINITY, -INFINITY};
#pragma unroll
      for (int ch = 0; ch < 4; ++ch) {
#pragma unroll
        for (int i = 0; i < 32; i += 4) {
          mx2[0] = max3(mx2[0], __uint_as_float(sv[ch][i]), __uint_as_float(sv[ch][i + 1]));
          mx2[1] = max3(mx2[1], __uint_as_float(sv[ch][i + 2]), __uint_as_float(sv[ch][i + 3]));
        }
      }
      const float mx = fmaxf(mx2[0], mx2[1]) * cc;
      float alpha = 1.f;
      const float m_new = fmaxf(m_used, mx);
      bool rescale = false;
      if (m_new > m_used + kRescaleThreshold || m_used == -INFINITY) {
        if (m_new != -INFINITY) {
          alpha = (m_used == -INFINITY) ? 0.f : fast_exp2(m_used - m_new);
          rescale = (m_used != -INFINITY);
          m_used = m_new;
        }
      }
      const float neg_m = (m_used == -INFINITY) ? 0.f : -m_used;
      const uint64_t c2 = pack_f32x2(cc, cc), nm2 = pack_f32x2(neg_m, neg_m);
      uint64_t sum2[2] = {0ull, 0ull};
      uint32_t pk[2][32];
#pragma unroll
      for (int ch = 0; ch < 4; ++ch) {
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          const uint64_t t = fma_f32x2(pack_u32x2(sv[ch][i], sv[ch][i + 1]), c2, nm2);
          float t0, t1;
          unpack_f32x2(t, t0, t1);
          const float e0 = fast_exp2(t0), e1 = fast_exp2(t1);
          sum2[(i >> 1) & 1] = add_f32x2(sum2[(i >> 1) & 1], pack_f32x2(e0, e1));
          pk[ch >> 1][(ch & 1) * 16 + (i >> 1)] = pack_bf16x2(e0, e1);
        }
      }
      float s0, s1, s2, s3;
      unpack_f32x2(sum2[0], s0, s1);
      unpack_f32x2(sum2[1], s2, s3);
      l = l * alpha + (s0 + s1) + (s2 + s3);
      // O_x is idle here: the S_x MMA that produced these scores was issued after the previous P_x·V
      if (n > 0 && __any_sync(0xffffffffu, rescale)) {
#pragma unroll 1
        for (int ch = 0; ch < p.v_panels * 2; ++ch) {
          uint32_t v[32];
          tmem_ld_32x32(tO[x] + lane_sel + ch * 32, v);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * alpha);
          tmem_st_32x32(tO[x] + lane_sel + ch * 32, v);
        }
      }
      tmem_st_32x32(tS[x] + lane_sel, pk[0]);
      tmem_st_32x32(tS[x] + lane_sel + 32, pk[1]);
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[x]);
    }
    if (ok && count[x] > 0 && !*abort_flag) ok = mbar_wait(&o_done[x], 0);
    if (!ok) {
      fail(abort_flag, p.err, 224);
    } else if (tile_valid) {
      tc_fence_after();
      const float inv_l = l > 0.f ? 1.f / l : 0.f;
      const long long token = row_base + q_idx;
      __nv_bfloat16* orow = p.o + (token * p.heads + h) * p.vdim;
      const __nv_bfloat16* grow = p.gate != nullptr ? p.gate + token * p.gate_ld + static_cast<long long>(h) * p.vdim : nullptr;
#pragma unroll 1
      for (int ch = 0; ch < p.v_panels * 2; ++ch) {
        uint32_t v[32];
        if (count[x] > 0) {
          tmem_ld_32x32(tO[x] + lane_sel + ch * 32, v);
          tmem_ld_wait();
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i) v[i] = 0;
        }
        if (row_valid) {
#pragma unroll
          for (int g = 0; g < 4; ++g) {
            const int col = ch * 32 + g * 8;
            if (col >= p.vdim) continue;  // vdim is a multiple of 8
            float f[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) f[i] = __uint_as_float(v[g * 8 + i]) * inv_l;
            if (grow != nullptr) {
              const uint4 gu = *reinterpret_cast<const uint4*>(grow + col);
              const __nv_bfloat162* gb = reinterpret_cast<const __nv_bfloat162*>(&gu);
#pragma unroll
              for (int i = 0; i < 4; ++i) {
                const float2 gf = __bfloat1622float2(gb[i]);
                f[2 * i] *= sigmoid_of(gf.x);
                f[2 * i + 1] *= sigmoid_of(gf.y);
              }
            }
            uint4 u;
            u.x = pack_bf16x2(f[0], f[1]);
            u.y = pack_bf16x2(f[2], f[3]);
            u.z = pack_bf16x2(f[4], f[5]);
            u.w = pack_bf16x2(f[6], f[7]);
            *reinterpret_cast<uint4*>(orow + col) = u;
          }
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  if (warp == 2) tmem_dealloc(tmem_base, 512);
}

// ===================================================================================== decode
struct DecodeParams {
  int b, heads, rank, rot, slots;
  int group, group_ctas;  // query heads that share keys, CTAs they take
  int pairs;       // 128-column pieces of the latent (grouped form: of the values)
  int q_panels;    // query panels multiplied with the pieces (grouped form: none)
  int c_steps, rot_panels, rot_steps;
  int ring;        // 32 KB slots for pieces
  int rot_stages;
  int lookahead;   // the ring holds two tiles: loads and scores of the next run beside this tile's outputs
  int tmem_cols;
  float scale;
  const int* slot;  // device: cache slot of the newest token (nullptr: slot_host)
  int slot_host;
  const int* lo;    // first visible slot of batch row bi at lo[bi * lo_row], or nullptr (0)
  long long lo_row;
  const int* hi;    // last visible slot, or nullptr (the newest token)
  long long hi_row;
  float* o;         // [splits, b, heads, rank] unnormalised
  float2* ml;       // [splits, b, heads] (maximum in the log2 domain, sum)
  int* err;
};

static constexpr int kDecodeThreads = 256;
static constexpr int kMaxRing = 12;
static constexpr int kDecodeBarriers = 2 * kMaxRing + 4 + 4 + 5;

__device__ __forceinline__ float warp_max(float v) {
  float r;
  asm volatile("redux.sync.max.f32 %0, %1, 0xffffffff;" : "=f"(r) : "f"(v));
  return r;
}
// logical or over the 128 softmax threads (named barrier 1)
__device__ __forceinline__ bool group_any(bool v) {
  uint32_t out;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.u32 q, %1, 0;\n\t"
      "barrier.cta.red.or.pred p, 1, 128, q;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t}"
      : "=r"(out)
      : "r"(static_cast<uint32_t>(v))
      : "memory");
  return out != 0;
}
__device__ __forceinline__ void group_sync() { asm volatile("barrier.cta.sync 1, 128;" ::: "memory"); }

// Up to four contraction steps (of 16 columns) of one pair of 64-column K-major panels.  `da` / `db` describe the panels' first steps; a step
// further is 32 bytes, i.e. 2 in the descriptors' address fields, so the issuing thread spends one addition per operand.
__device__ __forceinline__ void umma_panel(uint32_t d, uint64_t da, uint64_t db, int steps, uint32_t idesc, bool accumulate) {
#pragma unroll
  for (int k = 0; k < 4; ++k)
    if (k < steps) umma_f16(d, da + 2 * k, db + 2 * k, idesc, accumulate || k > 0);
}

template <int HN>
__device__ __forceinline__ void tmem_ld_heads(uint32_t addr, uint32_t (&v)[HN]) {
  if constexpr (HN == 16) tmem_ld_32x16(addr, v);
  else tmem_ld_32x32(addr, v);
}
template <int HN>
__device__ __forceinline__ void tmem_st_heads(uint32_t addr, const uint32_t (&v)[HN]) {
  if constexpr (HN == 16) tmem_st_32x16(addr, v);
  else tmem_st_32x32(addr, v);
}

// HN: heads per CTA (16 or 32).  KB: keys per tile.  A wide latent leaves room for one and a bit 128-key tiles; tiles of 64 keys are then
// double-buffered instead.  The 64 rows of such a score tile land in the first 16 lanes of each warp's quarter of tensor memory.
template <int HN, int KB>
__global__ void __launch_bounds__(kDecodeThreads, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmC, const __grid_constant__ CUtensorMap tmR, DecodeParams p) {
  constexpr int kQPanel = HN * 128;  // bytes of a 64-column panel of HN rows
  constexpr int kKeyPanel = KB * 128, kPairBytes = 2 * kKeyPanel, kPBytes = KB / 64 * kQPanel;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sC = smem;                                        // [ring] pieces: KB rows x 128 columns
  uint8_t* sR = sC + p.ring * kPairBytes;                    // [rot_stages]
  uint8_t* sQ = sR + p.rot_stages * p.rot_panels * kKeyPanel;  // 2 * pairs latent panels, then the rotated ones
  uint8_t* sP = sQ + (p.q_panels + p.rot_panels) * kQPanel;     // [2] tiles of [HN heads, KB keys]
  uint64_t* bars = reinterpret_cast<uint64_t*>(sP + 2 * kPBytes);
  uint64_t* c_full = bars;                 // [ring]
  uint64_t* c_empty = bars + kMaxRing;     // [ring]
  uint64_t* r_full = bars + 2 * kMaxRing;  // [rot_stages <= 2]
  uint64_t* r_empty = r_full + 2;
  uint64_t* s_full = r_empty + 2;          // [2]
  uint64_t* s_free = s_full + 2;           // [2]
  uint64_t* q_full = s_free + 2;
  uint64_t* p_full = q_full + 1;           // [2]
  uint64_t* pv_done = p_full + 2;          // [2]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(pv_done + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* s_red = reinterpret_cast<float*>(tmem_slot + 2);  // [4][HN]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int split = blockIdx.x, splits = gridDim.x, bi = blockIdx.z;
  const int hk = blockIdx.y / p.group_ctas, h0 = hk * p.group + (blockIdx.y % p.group_ctas) * HN, h_end = (hk + 1) * p.group;
  const int newest = p.slot != nullptr ? *p.slot : p.slot_host;
  const int hi = min(p.hi != nullptr ? p.hi[bi * p.hi_row] : newest, p.slots - 1);
  const int lo = max(p.lo != nullptr ? p.lo[bi * p.lo_row] : 0, 0);
  const int blk0 = lo / KB;
  const int total = hi >= lo ? hi / KB - blk0 + 1 : 0;
  const int per = (total + splits - 1) / splits;
  const int first = blk0 + split * per;
  const int n_blocks = max(min(per, total - split * per), 0);

  if (threadIdx.x == 0) {
    for (int i = 0; i < p.ring; ++i) {
      mbar_init(&c_full[i], 1);
      mbar_init(&c_empty[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&r_full[i], 1);
      mbar_init(&r_empty[i], 1);
      mbar_init(&s_full[i], 1);
      mbar_init(&s_free[i], 4);
      mbar_init(&p_full[i], 4);
      mbar_init(&pv_done[i], 1);
    }
    mbar_init(q_full, 1);
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 2) {
    tmem_alloc(tmem_slot, p.tmem_cols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tO = tmem_base + 2 * HN;  // after the two score tiles

  if (warp == 0) {
    // ---------------------------------------------------------------- TMA producer
    if (lane == 0 && n_blocks > 0) {
      mbar_arrive_expect_tx(q_full, (p.q_panels + p.rot_panels) * kQPanel);
      for (int j = 0; j < p.q_panels; ++j) tma_load_3d(sQ + j * kQPanel, &tmQ, q_full, j * 64, h0, bi);
      for (int j = 0; j < p.rot_panels; ++j) tma_load_3d(sQ + (p.q_panels + j) * kQPanel, &tmQ, q_full, (p.q_panels > 0 ? p.rank : 0) + j * 64, h0, bi);
    }
    int cs = 0, rs = 0;
    uint32_t cph = 0, rph = 0;
    for (int it = 0; it < n_blocks && !*abort_flag; ++it) {
      const int key0 = (first + it) * KB;
      bool ok = true;
      for (int u = 0; u < p.pairs && ok; ++u) {
        ok = mbar_wait(&c_empty[cs], cph ^ 1);
        if (ok && lane == 0) {
          mbar_arrive_expect_tx(&c_full[cs], kPairBytes);
          tma_load_4d(sC + cs * kPairBytes, &tmC, &c_full[cs], u * 128, hk, key0, bi);
          tma_load_4d(sC + cs * kPairBytes + kKeyPanel, &tmC, &c_full[cs], u * 128 + 64, hk, key0, bi);
        }
        __syncwarp();
        if (++cs == p.ring) cs = 0, cph ^= 1;
      }
      ok = ok && mbar_wait(&r_empty[rs], rph ^ 1);
      if (!ok) {
        fail(abort_flag, p.err, 231);
        break;
      }
      if (lane == 0) {
        uint8_t* dst = sR + rs * p.rot_panels * kKeyPanel;
        mbar_arrive_expect_tx(&r_full[rs], p.rot_panels * kKeyPanel);
        for (int j = 0; j < p.rot_panels; ++j) tma_load_4d(dst + j * kKeyPanel, &tmR, &r_full[rs], j * 64, hk, key0, bi);
      }
      __syncwarp();
      if (++rs == p.rot_stages) rs = 0, rph ^= 1;
    }
  } else if (warp == 1) {
    // ---------------------------------------------------------------- scores: Sᵀ(it) = C(it) · Qᵀ
    // With few columns an MMA is over in less time than its issue takes, so scores and outputs are issued by two warps.
    constexpr uint32_t idesc = make_idesc_bf16(KB, HN, false, false);
    const uint64_t dC = make_smem_desc_sw128(smem_u32(sC), 16, 1024), dR = make_smem_desc_sw128(smem_u32(sR), 16, 1024), dQ = make_smem_desc_sw128(smem_u32(sQ), 16, 1024);
    bool ok = n_blocks == 0 || mbar_wait(q_full, 0);
    int cs = 0, rs = 0;
    uint32_t cph = 0, rph = 0;
    for (int it = 0; it < n_blocks && ok && !*abort_flag; ++it) {
      const int st = it & 1;
      const uint32_t tS = tmem_base + st * HN;
      ok = mbar_wait(&s_free[st], ((it >> 1) & 1) ^ 1);
      for (int u = 0; 2 * u < p.q_panels && ok; ++u) {
        ok = mbar_wait(&c_full[cs], cph);
        tc_fence_after();
        if (ok && elect_one()) {
          const uint64_t da = dC + cs * (kPairBytes >> 4), db = dQ + u * (2 * kQPanel >> 4);
          const int steps = p.c_steps - 8 * u;
          umma_panel(tS, da, db, steps, idesc, u > 0);
          umma_panel(tS, da + (kKeyPanel >> 4), db + (kQPanel >> 4), steps - 4, idesc, true);
        }
        __syncwarp();
        if (++cs == p.ring) cs = 0, cph ^= 1;
      }
      ok = ok && mbar_wait(&r_full[rs], rph);
      tc_fence_after();
      if (ok && elect_one()) {
        for (int j = 0; j < p.rot_panels; ++j)
          umma_panel(tS, dR + (rs * p.rot_panels + j) * (kKeyPanel >> 4), dQ + (p.q_panels + j) * (kQPanel >> 4), p.rot_steps - 4 * j, idesc, p.q_panels > 0 || j > 0);
        umma_commit(&r_empty[rs]);
        umma_commit(&s_full[st]);
      }
      __syncwarp();
      if (++rs == p.rot_stages) rs = 0, rph ^= 1;
    }
    if (!ok) fail(abort_flag, p.err, 232);
  } else if (warp == 3) {
    // ---------------------------------------------------------------- outputs: Oᵀ += C(it)ᵀ · Pᵀ(it), then the pieces are handed back
    constexpr uint32_t idesc = make_idesc_bf16(128, HN, true, false);
    const uint64_t dC = make_smem_desc_sw128(smem_u32(sC), kKeyPanel, 1024), dP = make_smem_desc_sw128(smem_u32(sP), 16, 1024);
    bool ok = true;
    int cs = 0;
    uint32_t cph = 0;
    for (int it = 0; it < n_blocks && ok && !*abort_flag; ++it) {
      ok = mbar_wait(&p_full[it & 1], (it >> 1) & 1);
      const uint64_t db = dP + (it & 1) * (kPBytes >> 4);
      for (int u = 0; u < p.pairs && ok; ++u) {
        ok = mbar_wait(&c_full[cs], cph);
        tc_fence_after();
        if (ok && elect_one()) {
          const uint64_t da = dC + cs * (kPairBytes >> 4);
#pragma unroll
          for (int k = 0; k < KB / 16; ++k) umma_f16(tO + u * HN, da + k * (2048 >> 4), db + (k >> 2) * (kQPanel >> 4) + (k & 3) * 2, idesc, (it | k) != 0);
          umma_commit(&c_empty[cs]);
          if (u + 1 == p.pairs) umma_commit(&pv_done[it & 1]);
        }
        __syncwarp();
        if (++cs == p.ring) cs = 0, cph ^= 1;
      }
    }
    if (!ok) fail(abort_flag, p.err, 234);
  } else if (warp >= 4) {
    // ---------------------------------------------------------------- softmax over the keys of a tile: one key per thread, all heads
    // After a failed wait the warp keeps going without waiting, so all four warps meet at the same named barriers.
    const int quarter = warp & 3;
    const int r = quarter * 32 + lane;
    const int r_key = KB == 64 ? quarter * 16 + lane : r;  // this thread's key of a tile ...
    const bool has_key = KB == 128 || lane < 16;           // ... if it has one
    const uint32_t lane_sel = static_cast<uint32_t>(quarter * 32) << 16;
    const float c = p.scale * kLog2e;
    float m[HN], l[HN];
#pragma unroll
    for (int h = 0; h < HN; ++h) m[h] = -INFINITY, l[h] = 0.f;
    bool ok = true;
    for (int it = 0; it < n_blocks; ++it) {
      const int st = it & 1;
      const int key = (first + it) * KB + r_key;
      if (ok && !*abort_flag) ok = mbar_wait(&s_full[st], (it >> 1) & 1);
      tc_fence_after();
      uint32_t sv[HN];
      tmem_ld_heads<HN>(tmem_base + st * HN + lane_sel, sv);
      tmem_ld_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&s_free[st]);
      const bool visible = has_key && key >= lo && key <= hi;
      bool grows = false;
#pragma unroll
      for (int h = 0; h < HN; ++h) {
        const float x = visible ? __uint_as_float(sv[h]) * c : -INFINITY;
        sv[h] = __float_as_uint(x);
        grows |= x > m[h] + kRescaleThreshold;
      }
      const bool update = group_any(grows);  // uniform over the four warps
      float alpha[HN];
      if (update) {
#pragma unroll
        for (int h = 0; h < HN; ++h) {
          const float v = warp_max(__uint_as_float(sv[h]));
          if (lane == h % 32) s_red[quarter * HN + h] = v;
        }
        group_sync();
#pragma unroll
        for (int h = 0; h < HN; ++h) {
          const float v = fmaxf(fmaxf(s_red[h], s_red[HN + h]), fmaxf(s_red[2 * HN + h], s_red[3 * HN + h]));
          const float m_new = fmaxf(m[h], v);
          alpha[h] = m[h] == -INFINITY ? 0.f : fast_exp2(m[h] - m_new);
          m[h] = m_new;
          l[h] *= alpha[h];
        }
      }
#pragma unroll
      for (int h = 0; h < HN; ++h) {
        const float e = m[h] == -INFINITY ? 0.f : fast_exp2(__uint_as_float(sv[h]) - m[h]);
        l[h] += e;
        sv[h] = __float_as_uint(e);
      }
      // P(it) may be overwritten once the outputs of tile it - 2 are finished; the running outputs may be rescaled only once those of
      // tile it - 1 are (a maximum rarely moves after the first tiles)
      if (it > 1 && ok && !*abort_flag) ok = mbar_wait(&pv_done[it & 1], ((it >> 1) & 1) ^ 1);
      if (it > 0 && update) {
        if (ok && !*abort_flag) ok = mbar_wait(&pv_done[(it - 1) & 1], ((it - 1) >> 1) & 1);
        tc_fence_after();
#pragma unroll 1
        for (int u = 0; u < p.pairs; ++u) {
          uint32_t v[HN];
          tmem_ld_heads<HN>(tO + lane_sel + u * HN, v);
          tmem_ld_wait();
#pragma unroll
          for (int h = 0; h < HN; ++h) v[h] = __float_as_uint(__uint_as_float(v[h]) * alpha[h]);
          tmem_st_heads<HN>(tO + lane_sel + u * HN, v);
        }
        tmem_st_wait();
      }
      if (has_key) {
        uint8_t* panel = sP + (it & 1) * kPBytes + (r_key >> 6) * kQPanel;
        const int chunk = (r_key & 63) >> 3, byte = (r_key & 7) * 2;
#pragma unroll
        for (int h = 0; h < HN; ++h)
          *reinterpret_cast<__nv_bfloat16*>(panel + h * 128 + ((chunk ^ (h & 7)) << 4) + byte) = __float2bfloat16_rn(__uint_as_float(sv[h]));
      }
      fence_proxy_async_smem();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[it & 1]);
    }
    if (ok && n_blocks > 0 && !*abort_flag) ok = mbar_wait(&pv_done[(n_blocks - 1) & 1], ((n_blocks - 1) >> 1) & 1);
    if (!ok) fail(abort_flag, p.err, 233);
    tc_fence_after();
    group_sync();  // the last maxima have been read
#pragma unroll
    for (int h = 0; h < HN; ++h) {
      float v = l[h];
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
      if (lane == h % 32) s_red[quarter * HN + h] = v;
    }
    group_sync();
    const long long row0 = (static_cast<long long>(split) * p.b + bi) * p.heads + h0;
#pragma unroll
    for (int h = 0; h < HN; ++h)
      if (r == h && h0 + h < h_end) p.ml[row0 + h] = make_float2(m[h], s_red[h] + s_red[HN + h] + s_red[2 * HN + h] + s_red[3 * HN + h]);
    if (n_blocks > 0 && ok) {
#pragma unroll 1
      for (int u = 0; u < p.pairs; ++u) {
        uint32_t v[HN];
        tmem_ld_heads<HN>(tO + lane_sel + u * HN, v);
        tmem_ld_wait();
        const int col = u * 128 + r;
        if (col < p.rank) {
          float* dst = p.o + row0 * p.rank + col;
#pragma unroll
          for (int h = 0; h < HN; ++h)
            if (h0 + h < h_end) dst[static_cast<long long>(h) * p.rank] = __uint_as_float(v[h]);
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  if (warp == 2) tmem_dealloc(tmem_base, p.tmem_cols);
}

static constexpr int kSmemLimit = 227 * 1024;

// rows of 64-column panels: [batch, keys, heads, columns] with the given row, head and batch pitches
static int map4(CUtensorMap* m, const void* base, uint64_t cols, uint64_t heads, uint64_t keys, uint64_t batch, uint64_t head_pitch, uint64_t key_pitch, uint64_t batch_pitch,
                uint32_t box_keys) {
  return make_tmap_4d(m, base, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, {cols, heads, keys, batch}, {head_pitch * 2, key_pitch * 2, batch_pitch * 2}, {64, 1, box_keys, 1},
                      CU_TENSOR_MAP_SWIZZLE_128B);
}
static int map3(CUtensorMap* m, const void* base, uint64_t d0, uint64_t d1, uint64_t d2, uint64_t s1_elems, uint64_t s2_elems, uint32_t b1, uint32_t b2) {
  return make_tmap_3d(m, base, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, d0, d1, d2, s1_elems * 2, s2_elems * 2, 64, b1, b2, CU_TENSOR_MAP_SWIZZLE_128B);
}

// Shared memory of one CTA: fixed part and how many 128-column pieces fit next to it.
template <int HN, int KB>
static int plan_decode(DecodeParams& p) {
  const int q_panel = HN * 128, key_panel = KB * 128;
  const int fixed = (p.q_panels + p.rot_panels + 2 * (KB / 64)) * q_panel + 1024 + (kDecodeBarriers + 2) * 8 + 4 * HN * 4;
  const int rot_bytes = p.rot_panels * key_panel;
  p.rot_stages = fixed + 2 * rot_bytes + 2 * p.pairs * 2 * key_panel <= kSmemLimit ? 2 : 1;
  int ring = (kSmemLimit - fixed - p.rot_stages * rot_bytes) / (2 * key_panel);
  if (ring > 3 * p.pairs) ring = 3 * p.pairs;
  if (ring > kMaxRing) ring = kMaxRing;
  p.ring = ring;
  p.lookahead = ring >= 2 * p.pairs;
  return fixed + p.rot_stages * rot_bytes + ring * 2 * key_panel;
}

template <int HN>
static bool small_tiles(DecodeParams p) {
  plan_decode<HN, 128>(p);
  return !p.lookahead;
}

// What the decode kernel reads: queries [b, heads, q_width] with a batch pitch, pieces and second operand as [b, slots, key heads, columns].
struct DecodeInputs {
  const void* q;
  uint64_t q_width, q_batch;
  const void* c;
  uint64_t c_head, c_key, c_batch;
  const void* r;
  uint64_t r_head, r_key, r_batch;
  int key_heads;
};

template <int HN, int KB>
static int launch_decode(DecodeParams& p, const DecodeInputs& in, int splits, cudaStream_t st) {
  const int smem = plan_decode<HN, KB>(p);
  if (p.ring < p.pairs || smem > kSmemLimit) return kErrTooLarge;
  int cols = 32;
  while (cols < 2 * HN + p.pairs * HN) cols *= 2;
  p.tmem_cols = cols;
  p.group_ctas = (p.group + HN - 1) / HN;
  CUtensorMap tq, tc, tr;
  int rc;
  if ((rc = map3(&tq, in.q, in.q_width, p.heads, p.b, in.q_width, in.q_batch, HN, 1)) != kOk) return rc;
  if ((rc = map4(&tc, in.c, p.rank, in.key_heads, p.slots, p.b, in.c_head, in.c_key, in.c_batch, KB)) != kOk) return rc;
  if ((rc = map4(&tr, in.r, p.rot, in.key_heads, p.slots, p.b, in.r_head, in.r_key, in.r_batch, KB)) != kOk) return rc;
  static bool attr = false;
  if (!attr) {
    if (cudaFuncSetAttribute(latent_decode_kernel<HN, KB>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmemLimit) != cudaSuccess) return kErrDriver;
    attr = true;
  }
  TTB_COUNT_LAUNCH(1);
  latent_decode_kernel<HN, KB><<<dim3(splits, in.key_heads * p.group_ctas, p.b), kDecodeThreads, smem, st>>>(tq, tc, tr, p);
  return cudaGetLastError() == cudaSuccess ? kOk : kErrDriver;
}

static int launch_decode_any(DecodeParams& p, const DecodeInputs& in, int splits, cudaStream_t st) {
  if (p.group <= 16) return small_tiles<16>(p) ? launch_decode<16, 64>(p, in, splits, st) : launch_decode<16, 128>(p, in, splits, st);
  return small_tiles<32>(p) ? launch_decode<32, 64>(p, in, splits, st) : launch_decode<32, 128>(p, in, splits, st);
}

// `pieces_score`: the pieces are keys as well as values (latents)
static DecodeParams decode_shape(int heads, int group, int rank, int rot, bool pieces_score) {
  DecodeParams p{};
  p.heads = heads, p.group = group, p.rank = rank, p.rot = rot;
  p.pairs = (rank + 127) / 128, p.q_panels = pieces_score ? 2 * p.pairs : 0, p.c_steps = (rank + 15) / 16, p.rot_panels = (rot + 63) / 64, p.rot_steps = (rot + 15) / 16;
  return p;
}

static int launch_prefill(PrefillParams& p, int dim, int rot, const CUtensorMap& tqn, const CUtensorMap& tqr, const CUtensorMap& tkn, const CUtensorMap& tkr, const CUtensorMap& tv,
                          cudaStream_t st) {
  p.dim_panels = (dim + 63) / 64, p.rot_panels = (rot + 63) / 64, p.v_panels = (p.vdim + 63) / 64;
  p.dim_steps = (dim + 15) / 16, p.rot_steps = (rot + 15) / 16;
  const int kp = p.dim_panels + p.rot_panels;
  if (p.v_panels > 2 || kp > 4) return kErrTooLarge;
  p.k_stages = p.v_stages = 2;
  if (2 * kp + p.k_stages * kp + p.v_stages * p.v_panels > 14) p.v_stages = 1;
  if (2 * kp + p.k_stages * kp + p.v_stages * p.v_panels > 14) p.k_stages = 1;
  const int smem = (2 * kp + p.k_stages * kp + p.v_stages * p.v_panels) * kPanelBytes + 1024 + 256;
  if (smem > kSmemLimit) return kErrTooLarge;
  static bool attr = false;
  if (!attr) {
    if (cudaFuncSetAttribute(latent_prefill_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmemLimit) != cudaSuccess) return kErrDriver;
    attr = true;
  }
  TTB_COUNT_LAUNCH(1);
  latent_prefill_kernel<<<dim3((p.s + 2 * kBlk - 1) / (2 * kBlk), p.heads, p.b), kPrefillThreads, smem, st>>>(tqn, tqr, tkn, tkr, tv, p);
  return cudaGetLastError() == cudaSuccess ? kOk : kErrDriver;
}

}  // namespace latent
}  // namespace ttb

// Many queries per sequence.  q [b*s, ld_q] with head h at column h*(dim+rot) laid out [dim | rot] (rotation applied); kn and v: expanded
// keys / values [b*sk, ...] with row pitches ld_kn / ld_v and head pitches dim / vdim; kr: the rotated key part, slot j of batch row bi at
// kr + (bi*kr_batch + j*ld_kr); o [b*s, heads*vdim].
extern "C" int ttb_latent_prefill(const void* q, long long ld_q, const void* kn, long long ld_kn, const void* kr, long long ld_kr, long long kr_batch,
                                  const void* v, long long ld_v, const void* gate, long long gate_ld, void* o, int b, int s, int sk, int heads, int dim,
                                  int rot, int vdim, int slot0, const int* lo, long long lo_row, long long lo_query, const int* hi, long long hi_row,
                                  long long hi_query, float scale, int* err, void* stream) {
  using namespace ttb;
  using namespace ttb::latent;
  if (b <= 0 || s <= 0 || heads <= 0 || sk < slot0 + s || slot0 < 0) return kErrBadShape;
  if ((dim & 7) || (rot & 7) || (vdim & 7) || dim <= 0 || rot <= 0 || vdim <= 0 || (gate != nullptr && ((gate_ld & 7) || (reinterpret_cast<uintptr_t>(gate) & 15)))) return kErrBadShape;
  PrefillParams p{};
  p.b = b, p.s = s, p.sk = sk, p.heads = heads, p.group = 1, p.slot0 = slot0, p.vdim = vdim, p.scale = scale;
  p.lo = lo, p.lo_row = lo_row, p.lo_query = lo_query, p.hi = hi, p.hi_row = hi_row, p.hi_query = hi_query;
  p.gate = static_cast<const __nv_bfloat16*>(gate), p.gate_ld = gate_ld, p.o = static_cast<__nv_bfloat16*>(o), p.err = err;
  CUtensorMap tqn, tqr, tkn, tkr, tv;
  const uint64_t tq = static_cast<uint64_t>(b) * s;
  int rc;
  if ((rc = map3(&tqn, q, dim, heads, tq, dim + rot, ld_q, 1, kBlk)) != kOk) return rc;
  if ((rc = map3(&tqr, static_cast<const __nv_bfloat16*>(q) + dim, rot, heads, tq, dim + rot, ld_q, 1, kBlk)) != kOk) return rc;
  if ((rc = map4(&tkn, kn, dim, heads, sk, b, dim, ld_kn, sk * ld_kn, kBlk)) != kOk) return rc;
  if ((rc = map4(&tkr, kr, rot, 1, sk, b, ld_kr, ld_kr, kr_batch, kBlk)) != kOk) return rc;
  if ((rc = map4(&tv, v, vdim, heads, sk, b, vdim, ld_v, sk * ld_v, kBlk)) != kOk) return rc;
  return launch_prefill(p, dim, rot, tqn, tqr, tkn, tkr, tv, static_cast<cudaStream_t>(stream));
}

// Grouped-query attention of many queries per sequence: q [b*s, ld_q] with head h at column h*dim; k [b, slots, key_heads, dim] and
// v [b, slots, key_heads, vdim], of which the first sk slots exist; o [b*s, heads*vdim].  heads is a multiple of key_heads.
extern "C" int ttb_span_prefill(const void* q, long long ld_q, const void* k, const void* v, void* o, int b, int s, int sk, int slots, int heads, int key_heads, int dim, int vdim,
                                int slot0, const int* lo, long long lo_row, long long lo_query, const int* hi, long long hi_row, long long hi_query, float scale, int* err, void* stream) {
  using namespace ttb;
  using namespace ttb::latent;
  if (b <= 0 || s <= 0 || heads <= 0 || key_heads <= 0 || heads % key_heads || sk < slot0 + s || sk > slots || slot0 < 0) return kErrBadShape;
  if ((dim & 7) || (vdim & 7) || dim <= 0 || vdim <= 0) return kErrBadShape;
  PrefillParams p{};
  p.b = b, p.s = s, p.sk = sk, p.heads = heads, p.group = heads / key_heads, p.slot0 = slot0, p.vdim = vdim, p.scale = scale;
  p.lo = lo, p.lo_row = lo_row, p.lo_query = lo_query, p.hi = hi, p.hi_row = hi_row, p.hi_query = hi_query;
  p.o = static_cast<__nv_bfloat16*>(o), p.err = err;
  CUtensorMap tq, tk, tv;
  const uint64_t k_row = static_cast<uint64_t>(key_heads) * dim, v_row = static_cast<uint64_t>(key_heads) * vdim;
  int rc;
  if ((rc = map3(&tq, q, dim, heads, static_cast<uint64_t>(b) * s, dim, ld_q, 1, kBlk)) != kOk) return rc;
  if ((rc = map4(&tk, k, dim, key_heads, sk, b, dim, k_row, k_row * slots, kBlk)) != kOk) return rc;
  if ((rc = map4(&tv, v, vdim, key_heads, sk, b, vdim, v_row, v_row * slots, kBlk)) != kOk) return rc;
  return launch_prefill(p, dim, 0, tq, tq, tk, tk, tv, static_cast<cudaStream_t>(stream));
}

// One query per batch row, absorbed: q [b, heads, rank + rot], cache [b, slots, rank + rot] (bf16); o [splits, b, heads, rank] and
// ml [splits, b, heads, 2] fp32 partial results.
extern "C" int ttb_latent_decode(const void* q, const void* cache, float* o, float* ml, int b, int heads, int rank, int rot, int slots, int splits,
                                 const int* slot, int slot_host, const int* lo, long long lo_row, const int* hi, long long hi_row, float scale, int* err,
                                 void* stream) {
  using namespace ttb;
  using namespace ttb::latent;
  if (b <= 0 || heads <= 0 || slots <= 0 || splits <= 0 || (rank & 7) || (rot & 7) || rank <= 0 || rot <= 0) return kErrBadShape;
  if (rank > 512 || rot > 128) return kErrTooLarge;
  DecodeParams p = decode_shape(heads, heads, rank, rot, true);
  p.b = b, p.slots = slots, p.scale = scale;
  p.slot = slot, p.slot_host = slot_host, p.lo = lo, p.lo_row = lo_row, p.hi = hi, p.hi_row = hi_row;
  p.o = o, p.ml = reinterpret_cast<float2*>(ml), p.err = err;
  const uint64_t row = rank + rot;
  const DecodeInputs in{q, row, row * heads, cache, row, row, row * slots, static_cast<const __nv_bfloat16*>(cache) + rank, row, row, row * slots, 1};
  return launch_decode_any(p, in, splits, static_cast<cudaStream_t>(stream));
}

// Grouped-query attention of one query per batch row: q [b, heads, dim] with row pitch ld_q, k [b, slots, key_heads, dim], v [b, slots, key_heads, vdim]
// (bf16); o [splits, b, heads, vdim] and ml [splits, b, heads, 2] fp32 partial results.
extern "C" int ttb_span_decode(const void* q, long long ld_q, const void* k, const void* v, float* o, float* ml, int b, int heads, int key_heads, int dim, int vdim, int slots, int splits,
                               const int* slot, int slot_host, const int* lo, long long lo_row, const int* hi, long long hi_row, float scale, int* err, void* stream) {
  using namespace ttb;
  using namespace ttb::latent;
  if (b <= 0 || heads <= 0 || key_heads <= 0 || heads % key_heads || slots <= 0 || splits <= 0 || (dim & 7) || (vdim & 7) || dim <= 0 || vdim <= 0) return kErrBadShape;
  if (vdim > 512 || dim > 256) return kErrTooLarge;
  DecodeParams p = decode_shape(heads, heads / key_heads, vdim, dim, false);
  p.b = b, p.slots = slots, p.scale = scale;
  p.slot = slot, p.slot_host = slot_host, p.lo = lo, p.lo_row = lo_row, p.hi = hi, p.hi_row = hi_row;
  p.o = o, p.ml = reinterpret_cast<float2*>(ml), p.err = err;
  const uint64_t k_row = static_cast<uint64_t>(key_heads) * dim, v_row = static_cast<uint64_t>(key_heads) * vdim;
  const DecodeInputs in{q, static_cast<uint64_t>(dim), static_cast<uint64_t>(ld_q), v, static_cast<uint64_t>(vdim), v_row, v_row * slots, k, static_cast<uint64_t>(dim), k_row, k_row * slots, key_heads};
  return launch_decode_any(p, in, splits, static_cast<cudaStream_t>(stream));
}

// Keys per tile of ttb_latent_decode for these sizes (a key range should not be shorter).
extern "C" int ttb_latent_decode_tile(int heads, int rank, int rot) {
  using namespace ttb::latent;
  if (rank <= 0 || rank > 512 || rot <= 0 || rot > 128) return 128;
  const DecodeParams p = decode_shape(heads, heads, rank, rot, true);
  return (heads <= 16 ? small_tiles<16>(p) : small_tiles<32>(p)) ? 64 : 128;
}

// The same for ttb_span_decode, with the number of query heads that share a key head.
extern "C" int ttb_span_decode_tile(int group, int dim, int vdim) {
  using namespace ttb::latent;
  if (group <= 0 || dim <= 0 || dim > 256 || vdim <= 0 || vdim > 512) return 128;
  const DecodeParams p = decode_shape(group, group, vdim, dim, false);
  return (group <= 16 ? small_tiles<16>(p) : small_tiles<32>(p)) ? 64 : 128;
}
