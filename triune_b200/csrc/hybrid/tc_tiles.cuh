// Device helpers shared by the tensor-core kernels of the heterogeneous-layer family: TMEM operands, fp32 values as pairs of
// bf16 numbers, and the per-token scalars of the recurrences.
#pragma once
#include "../common/ptx.cuh"
#include "hybrid.cuh"

namespace tb {
namespace {

// D[tmem] (+)= A[tmem] * B[smem]: A is bf16 with two K elements per 32-bit column, row = lane
__device__ __forceinline__ void umma_bf16_ts(uint32_t tmem_d, uint32_t tmem_a, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t"
      ".reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t"
      "}\n" ::"r"(tmem_d),
      "r"(tmem_a), "l"(bdesc), "r"(idesc), "r"(accumulate)
      : "memory");
}
// wait::ld that the loaded registers depend on, so that no use can be scheduled before it
__device__ __forceinline__ void tmem_ld_wait_regs(uint32_t (&r)[32]) {
  asm volatile("tcgen05.wait::ld.sync.aligned;"
               : "+r"(r[0]), "+r"(r[1]), "+r"(r[2]), "+r"(r[3]), "+r"(r[4]), "+r"(r[5]), "+r"(r[6]), "+r"(r[7]), "+r"(r[8]), "+r"(r[9]),
                 "+r"(r[10]), "+r"(r[11]), "+r"(r[12]), "+r"(r[13]), "+r"(r[14]), "+r"(r[15]), "+r"(r[16]), "+r"(r[17]), "+r"(r[18]),
                 "+r"(r[19]), "+r"(r[20]), "+r"(r[21]), "+r"(r[22]), "+r"(r[23]), "+r"(r[24]), "+r"(r[25]), "+r"(r[26]), "+r"(r[27]),
                 "+r"(r[28])
               :
               : "memory");
  asm volatile("" : "+r"(r[29]), "+r"(r[30]), "+r"(r[31])::"memory");
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// 16-byte piece `ch` (of 8) of row r of a swizzled tile
__device__ __forceinline__ uint32_t sw(int r, int ch) { return (uint32_t)(r * 128 + ((ch ^ (r & 7)) << 4)); }

__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_wait0() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

constexpr int CL = 64;  // tokens per chunk of the scalars below

__device__ __forceinline__ float lo_f(uint32_t x) { return __uint_as_float(x << 16); }
__device__ __forceinline__ float hi_f(uint32_t x) { return __uint_as_float(x & 0xffff0000u); }
// (a, b) as two bf16 pairs whose sum is the fp32 pair to 2^-17
__device__ __forceinline__ void split2(float a, float b, uint32_t& h, uint32_t& l) {
  h = pack_bf16x2(a, b);
  l = pack_bf16x2(a - lo_f(h), b - hi_f(h));
}
// e^x for x <= 0
__device__ __forceinline__ float exp_neg(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x * 1.4426950408889634f));
  return y;
}

// Log decay and gate of the 64 tokens of a chunk by one warp: lane i holds tokens 2 i and 2 i + 1. Tokens past T change
// nothing (no decay, zero gate). gate: dt (mamba2) or beta (delta).
__device__ __forceinline__ void chunk_scalars(const RecurrentArgs& p, float ra0, float ra1, float rb0, float rb1, float ea, float bias,
                                              int t0, float* sb, float* sgate) {
  const int lane = threadIdx.x & 31, t = t0 + 2 * lane;
  const float d0 = t < p.T ? softplus_f(ra0 + bias) : 0.f, d1 = t + 1 < p.T ? softplus_f(ra1 + bias) : 0.f;
  float x = -ea * (d0 + d1);
  const float own = x;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float y = __shfl_up_sync(0xffffffffu, x, o);
    if (lane >= o) x += y;
  }
  const float before = x - own;
  sb[2 * lane] = before - ea * d0;
  sb[2 * lane + 1] = x;
  if (p.kind == RK_DELTA) {
    sgate[2 * lane] = t < p.T ? sigmoid_f(rb0) : 0.f;
    sgate[2 * lane + 1] = t + 1 < p.T ? sigmoid_f(rb1) : 0.f;
  } else {
    sgate[2 * lane] = d0;
    sgate[2 * lane + 1] = d1;
  }
}
__device__ __forceinline__ float load_or0(const __nv_bfloat16* p, long long ld, int t, int T) {
  return t < T ? __bfloat162float(p[(long long)t * ld]) : 0.f;
}

}  // namespace
}  // namespace tb
