// Small pieces shared by the attention kernels that keep score rows in registers: descriptors of operand tiles stored as 64-column
// panels of 128 rows, three-input maximum, two-wide fp32 arithmetic and the failure report of a bounded wait.
#pragma once
#include "ptx.cuh"

namespace ttb {
namespace attn {

static constexpr int kBlk = 128;           // query rows / key rows per tile
static constexpr int kPanelBytes = 16384;  // 128 rows x 128 B (64 bf16 columns)
static constexpr float kLog2e = 1.4426950408889634f;
static constexpr float kRescaleThreshold = 8.0f;  // log2 units: a running maximum moves only when it grows by more than 2^8

// Contraction index contiguous: slice k covers columns [16k, 16k + 16) of a tile of 128-row panels.
__device__ __forceinline__ uint64_t desc_kmajor(uint32_t base, int k) {
  return make_smem_desc_sw128(base + (k >> 2) * kPanelBytes + (k & 3) * 32, 16, 1024);
}
// Row index as contraction: slice k covers rows [16k, 16k + 16); 64-column panels are kPanelBytes apart.
__device__ __forceinline__ uint64_t desc_mnmajor(uint32_t base, int k) {
  return make_smem_desc_sw128(base + k * 2048, kPanelBytes, 1024);
}
__device__ __forceinline__ float max3(float a, float b, float c) {
  float d;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
  return d;
}
__device__ __forceinline__ uint64_t pack_f32x2(float lo, float hi) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ uint64_t pack_u32x2(uint32_t lo, uint32_t hi) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "r"(lo), "r"(hi));
  return d;
}
__device__ __forceinline__ void unpack_f32x2(uint64_t v, float& lo, float& hi) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
}
__device__ __forceinline__ uint64_t fma_f32x2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t add_f32x2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ void fail(volatile int* abort_flag, int* err, int code) {
  *abort_flag = 1;
  atomicExch(err, code);
}

}  // namespace attn
}  // namespace ttb
