// Retention prompts on the tcgen05 tensor cores: chunks of 128 tokens, for aligned bf16 inputs and key sizes up to 128.
//
// With q and k turned and k scaled in fp32, d the head's decay and S_c the state before chunk c of n_c tokens:
//   U_c     = sum_j d^{n_c-1-j} k_j v_j^T                                (states kernel, every chunk on its own)
//   S_{c+1} = d^{n_c} S_c + U_c                                           (scan kernel, every state entry on its own)
//   out_i   = d^{i+1} S_c^T q_i + sum_{j<=i} d^{i-j} (q_i . k_j) v_j       (outputs kernel, every chunk on its own)
// The decay is a constant, so nothing but the small scan is sequential: both tensor-core kernels are a few hundred to a few
// thousand independent blocks without a walk. Values are exact bf16 operands; turned queries and keys, weighted keys,
// decayed scores and states are fp32 and enter the tensor core as the sum of two bf16 numbers (products of two such
// operands take three MMAs). Accumulators and the carried state are fp32.
//
// A block owns 128 value columns of a head and chunk. Shared-memory tiles are rows of 128 bytes in the 128B-swizzled layout:
// queries and keys are written by the threads that turn and split them, values and states come by TMA. 512 threads are
// four times 128 rows: a thread has the row of its TMEM lane and a quarter of the columns.
// TMEM columns of the outputs kernel: 0 scores (128), 128 decayed scores as bf16 pairs, high (64) and low (64) halves,
// 256 queries times state (128), 384 decayed scores times values (128).
#include "../common/ptx.cuh"
#include "../common/tma_desc.h"
#include "hybrid.cuh"
#include "tc_tiles.cuh"

namespace tb {
namespace {

constexpr int RT = 128, RTH = 512, RBOX = 128 * 128, RCOLS = 128;  // tokens, threads, bytes of a 128 x 64 tile, value columns

struct RetParams {
  RecurrentArgs a;
  int nchunks;
  float* own;                // [B H, nchunks, Dk, Dv] contributions U
  __nv_bfloat16 *hi, *lo;    // the same shape: states before the chunks
  int* status;
};

// eight fp32 values as 16-byte pieces of two tiles
__device__ __forceinline__ void put8(uint8_t* hi, uint8_t* lo, uint32_t at, const float (&f)[8]) {
  uint4 h, l;
  split2(f[0], f[1], h.x, l.x);
  split2(f[2], f[3], h.y, l.y);
  split2(f[4], f[5], h.z, l.z);
  split2(f[6], f[7], h.w, l.w);
  *reinterpret_cast<uint4*>(hi + at) = h;
  *reinterpret_cast<uint4*>(lo + at) = l;
}

// One of the operands that stage_turned writes: a head's rows, the tiles of their high and low halves, their factor and the
// rows' weights (or null).
struct Turned {
  const __nv_bfloat16* src;
  long long ld;
  uint8_t *hi, *lo;
  float scale;
  const float* weight;
};

// Rows t0 .. t0 + 127 of N operands, turned, times factor and weight, into `boxes` swizzled tiles of 64 columns each; rows past
// T and columns past D become zero. Dimensions come in pieces of eight: pieces below half the rotated dimensions together
// with the piece half of them away. The loads of AHEAD items of a thread are in flight before the first is used.
template <int N>
__device__ __forceinline__ void stage_turned(const Turned (&ops)[N], const float* rot, int rot_dims, int t0, int T, int D, int boxes, int tid) {
  constexpr int AHEAD = 2;
  const int hg = rot_dims / 16, items = boxes * 8 - hg, half = rot_dims / 2;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  for (int i0 = tid; i0 < RT * items; i0 += AHEAD * RTH) {
    uint4 u[AHEAD][N], v[AHEAD][N];
    float4 cs[AHEAD][4];
#pragma unroll
    for (int a = 0; a < AHEAD; ++a) {
      const int it = i0 + a * RTH, r = it / items, x = it % items, t = t0 + r;
      const bool on = it < RT * items && t < T, pair = x < hg;
#pragma unroll
      for (int n = 0; n < N; ++n) {
        const __nv_bfloat16* row = ops[n].src + (long long)t * ops[n].ld;
        u[a][n] = on && (pair ? x : x + hg) * 8 < D ? *reinterpret_cast<const uint4*>(row + (pair ? x : x + hg) * 8) : zero;
        v[a][n] = on && pair ? *reinterpret_cast<const uint4*>(row + half + x * 8) : zero;
      }
      if (on && pair) {
        const float4 *c = reinterpret_cast<const float4*>(rot + (long long)t * rot_dims + x * 8),
                     *s = reinterpret_cast<const float4*>(rot + (long long)t * rot_dims + half + x * 8);
        cs[a][0] = __ldg(c); cs[a][1] = __ldg(c + 1); cs[a][2] = __ldg(s); cs[a][3] = __ldg(s + 1);
      } else {
        cs[a][0] = cs[a][1] = make_float4(1.f, 1.f, 1.f, 1.f);
        cs[a][2] = cs[a][3] = make_float4(0.f, 0.f, 0.f, 0.f);
      }
    }
#pragma unroll
    for (int a = 0; a < AHEAD; ++a) {
      const int it = i0 + a * RTH, r = it / items, x = it % items, g = x + hg;
      if (it >= RT * items) break;
      const float c[8] = {cs[a][0].x, cs[a][0].y, cs[a][0].z, cs[a][0].w, cs[a][1].x, cs[a][1].y, cs[a][1].z, cs[a][1].w};
      const float s[8] = {cs[a][2].x, cs[a][2].y, cs[a][2].z, cs[a][2].w, cs[a][3].x, cs[a][3].y, cs[a][3].z, cs[a][3].w};
#pragma unroll
      for (int n = 0; n < N; ++n) {
        const float w = ops[n].weight != nullptr ? ops[n].scale * ops[n].weight[r] : ops[n].scale;
        const uint32_t ua[4] = {u[a][n].x, u[a][n].y, u[a][n].z, u[a][n].w}, va[4] = {v[a][n].x, v[a][n].y, v[a][n].z, v[a][n].w};
        float p[8], q[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const float x0 = (i & 1) ? hi_f(ua[i / 2]) : lo_f(ua[i / 2]), x1 = (i & 1) ? hi_f(va[i / 2]) : lo_f(va[i / 2]);
          p[i] = (x0 * c[i] - x1 * s[i]) * w;
          q[i] = (x1 * c[i] + x0 * s[i]) * w;
        }
        if (x < hg) put8(ops[n].hi + (x >> 3) * RBOX, ops[n].lo + (x >> 3) * RBOX, sw(r, x & 7), p);
        put8(ops[n].hi + (g >> 3) * RBOX, ops[n].lo + (g >> 3) * RBOX, sw(r, g & 7), x < hg ? q : p);
      }
    }
  }
}

struct Place {  // of a block: head, chunk, value columns
  int h, b, bh, c, c0, ncol, t0;
};
__device__ __forceinline__ Place place_of(const RetParams& sp) {
  Place p;
  const int slices = (sp.a.Dv + RCOLS - 1) / RCOLS, slice = blockIdx.x % slices, unit = blockIdx.x / slices;
  p.c = unit % sp.nchunks;
  p.bh = unit / sp.nchunks;
  p.h = p.bh % sp.a.H;
  p.b = p.bh / sp.a.H;
  p.c0 = slice * RCOLS;
  p.ncol = min(RCOLS, sp.a.Dv - p.c0);
  p.t0 = p.c * RT;
  return p;
}

// ------------------------------------------------------------------------------------------------ contributions
constexpr int RS_V = 4 * RBOX, RS_SMEM = 6 * RBOX + 1024;  // weighted keys high, low (two tiles each), values (two tiles)

__global__ void __launch_bounds__(RTH, 2) retention_states_kernel(const __grid_constant__ CUtensorMap tmV, const RetParams sp) {
  extern __shared__ uint8_t raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(raw) + 1023) & ~uintptr_t(1023));
  __shared__ __align__(8) uint64_t v_full, done;
  __shared__ uint32_t tmem_slot;
  __shared__ float weight[RT];
  const RecurrentArgs& p = sp.a;
  const Place at = place_of(sp);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int n = min(RT, p.T - at.t0), vb = (at.ncol + 63) / 64;
  if (tid == 0) {
    mbar_init(&v_full, 1);
    mbar_init(&done, 1);
    mbar_fence_init();
    mbar_expect_tx(&v_full, vb * RBOX);
    for (int x = 0; x < vb; ++x) tma_load_4d(smem + RS_V + x * RBOX, &tmV, &v_full, at.c0 + x * 64, at.t0, at.h, at.b);
  }
  __syncwarp();
  if (warp == 0) {
    tmem_alloc(&tmem_slot, RCOLS);
    tmem_relinquish();
  }
  const float lg = log2f((float)p.decay[at.h]);
  if (tid < RT) weight[tid] = tid < n ? exp2f(lg * (n - 1 - tid)) : 0.f;
  __syncthreads();
  const __nv_bfloat16* K = (const __nv_bfloat16*)p.k + (long long)at.b * p.rows * p.ldk + at.h * p.Dk;
  const Turned keys[1] = {{K, p.ldk, smem, smem + 2 * RBOX, 1.f / sqrtf((float)p.Dk), weight}};
  stage_turned(keys, p.rot, p.rot_dims, at.t0, p.T, p.Dk, 2, tid);
  fence_proxy_async_smem();
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = tmem_slot;
  if (tid == 0) {
    bool ok = mbar_wait(&v_full, 0);
    if (ok) {
      tc_fence_after_sync();
      const uint32_t id = make_idesc(128, (at.ncol + 15) / 16 * 16, 1, 1, 1, 1), ka = smem_u32(smem), va = smem_u32(smem + RS_V);
#pragma unroll
      for (int k = 0; k < RT / 16; ++k) {
        const uint64_t v = make_smem_desc(va + k * 2048, RBOX, 1024);
        umma_bf16(tmem, make_smem_desc(ka + k * 2048, RBOX, 1024), v, id, k > 0);
        umma_bf16(tmem, make_smem_desc(ka + 2 * RBOX + k * 2048, RBOX, 1024), v, id, 1);
      }
      umma_commit(&done);
    } else if (sp.status) {
      *sp.status = ST_TIMEOUT_FULL;
    }
  }
  __syncwarp();
  const bool ok = mbar_wait(&done, 0);
  if (!ok && sp.status) *sp.status = ST_TIMEOUT_TMEM;
  __syncwarp();
  tc_fence_after_sync();
  if (ok) {
    const int row = (warp & 3) * 32 + lane, col0 = (warp >> 2) * 32;
    const uint32_t t = tmem + ((uint32_t)((warp & 3) * 32) << 16);
    float* dst = sp.own + (((long long)at.bh * sp.nchunks + at.c) * p.Dk + row) * p.Dv + at.c0 + col0;
    uint32_t v[32];
    tmem_ld_32x32b_x32(t + col0, v);
    tmem_ld_wait_regs(v);
    if (row < p.Dk) {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        float f[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] = __uint_as_float(v[8 * i + j]);
        if (col0 + 8 * i < at.ncol) st8v(dst + 8 * i, f);
      }
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  if (warp == 0) tmem_dealloc(tmem, RCOLS);
}

// ------------------------------------------------------------------------------------------------ scan
// grid (ceil(Dk Dv / 1024), B H): a thread has four neighbouring entries of the state and goes through the chunks
__global__ void __launch_bounds__(256) retention_scan_kernel(const RetParams sp) {
  const RecurrentArgs& p = sp.a;
  const long long plane = (long long)p.Dk * p.Dv, i = ((long long)blockIdx.x * 256 + threadIdx.x) * 4, bh = blockIdx.y;
  if (i >= plane) return;
  const float lg = log2f((float)p.decay[bh % p.H]), dl = exp2f(lg * RT);
  float4 run = *reinterpret_cast<const float4*>(p.state + bh * plane + i);
  const long long base = bh * sp.nchunks * plane + i;
  constexpr int AHEAD = 8;  // loads do not wait for one another
  for (int c0 = 0; c0 < sp.nchunks; c0 += AHEAD) {
    float4 own[AHEAD];
#pragma unroll
    for (int g = 0; g < AHEAD; ++g)
      if (c0 + g < sp.nchunks) own[g] = *reinterpret_cast<const float4*>(sp.own + base + (c0 + g) * plane);
#pragma unroll
    for (int g = 0; g < AHEAD; ++g)
      if (c0 + g < sp.nchunks) {
        uint2 h, l;
        split2(run.x, run.y, h.x, l.x);
        split2(run.z, run.w, h.y, l.y);
        *reinterpret_cast<uint2*>(sp.hi + base + (c0 + g) * plane) = h;
        *reinterpret_cast<uint2*>(sp.lo + base + (c0 + g) * plane) = l;
        const float d = c0 + g + 1 < sp.nchunks ? dl : exp2f(lg * (p.T - (sp.nchunks - 1) * RT));
        run = make_float4(d * run.x + own[g].x, d * run.y + own[g].y, d * run.z + own[g].z, d * run.w + own[g].w);
      }
  }
  *reinterpret_cast<float4*>(p.state + bh * plane + i) = run;
}

// ------------------------------------------------------------------------------------------------ outputs
template <int DKB>
struct RetSmem {  // after alignment to 1024 bytes
  static constexpr int SBOX = DKB * 64 * 128;  // a state tile: Dk rows of 64 columns
  static constexpr int QH = 0, QL = QH + DKB * RBOX, KH = QL + DKB * RBOX, KL = KH + DKB * RBOX, V = KL + DKB * RBOX, SH = V + 2 * RBOX,
                       SL = SH + 2 * SBOX, END = SL + 2 * SBOX;
};

template <int DKB>
__global__ void __launch_bounds__(RTH, 1) retention_out_kernel(const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmH,
                                                               const __grid_constant__ CUtensorMap tmL, const RetParams sp) {
  using L = RetSmem<DKB>;
  extern __shared__ uint8_t raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(raw) + 1023) & ~uintptr_t(1023));
  __shared__ __align__(8) uint64_t v_full, s_full, scored, done;
  __shared__ uint32_t tmem_slot;
  __shared__ float power[RT + 1];  // d^n
  const RecurrentArgs& p = sp.a;
  const Place at = place_of(sp);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int vb = (at.ncol + 63) / 64;
  if (tid == 0) {
    mbar_init(&v_full, 1);
    mbar_init(&s_full, 1);
    mbar_init(&scored, 1);
    mbar_init(&done, 1);
    mbar_fence_init();
    mbar_expect_tx(&v_full, vb * RBOX);
    mbar_expect_tx(&s_full, 2 * vb * L::SBOX);
    const int z = at.bh * sp.nchunks + at.c;
    for (int x = 0; x < vb; ++x) {
      tma_load_3d(smem + L::SH + x * L::SBOX, &tmH, &s_full, at.c0 + x * 64, 0, z);
      tma_load_3d(smem + L::SL + x * L::SBOX, &tmL, &s_full, at.c0 + x * 64, 0, z);
      tma_load_4d(smem + L::V + x * RBOX, &tmV, &v_full, at.c0 + x * 64, at.t0, at.h, at.b);
    }
  }
  __syncwarp();
  if (warp == 0) {
    tmem_alloc(&tmem_slot, 512);
    tmem_relinquish();
  }
  const float lg = log2f((float)p.decay[at.h]);
  if (tid <= RT) power[tid] = exp2f(lg * tid);
  const __nv_bfloat16 *Q = (const __nv_bfloat16*)p.q + (long long)at.b * p.rows * p.ldq + at.h * p.Dk,
                      *K = (const __nv_bfloat16*)p.k + (long long)at.b * p.rows * p.ldk + at.h * p.Dk;
  const Turned both[2] = {{Q, p.ldq, smem + L::QH, smem + L::QL, 1.f, nullptr}, {K, p.ldk, smem + L::KH, smem + L::KL, 1.f / sqrtf((float)p.Dk), nullptr}};
  stage_turned(both, p.rot, p.rot_dims, at.t0, p.T, p.Dk, DKB, tid);
  fence_proxy_async_smem();
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = tmem_slot, base = smem_u32(smem);
  const uint32_t id_o = make_idesc(128, (at.ncol + 15) / 16 * 16, 1, 1, 0, 1);
  if (tid == 0) {
    const uint32_t id_s = make_idesc(128, 128, 1, 1, 0, 0);
    const int ks = (p.Dk + 15) / 16;
    for (int k = 0; k < ks; ++k) {
      const uint32_t off = (k >> 2) * RBOX + (k & 3) * 32;
      const uint64_t qh = make_smem_desc(base + L::QH + off, 16, 1024), kh = make_smem_desc(base + L::KH + off, 16, 1024);
      umma_bf16(tmem, qh, kh, id_s, k > 0);
      umma_bf16(tmem, qh, make_smem_desc(base + L::KL + off, 16, 1024), id_s, 1);
      umma_bf16(tmem, make_smem_desc(base + L::QL + off, 16, 1024), kh, id_s, 1);
    }
    umma_commit(&scored);
    if (mbar_wait(&s_full, 0)) {
      tc_fence_after_sync();
      for (int k = 0; k < ks; ++k) {
        const uint32_t off = (k >> 2) * RBOX + (k & 3) * 32;
        const uint64_t qh = make_smem_desc(base + L::QH + off, 16, 1024), sh = make_smem_desc(base + L::SH + k * 2048, L::SBOX, 1024);
        umma_bf16(tmem + 256, qh, sh, id_o, k > 0);
        umma_bf16(tmem + 256, qh, make_smem_desc(base + L::SL + k * 2048, L::SBOX, 1024), id_o, 1);
        umma_bf16(tmem + 256, make_smem_desc(base + L::QL + off, 16, 1024), sh, id_o, 1);
      }
    } else if (sp.status) {
      *sp.status = ST_TIMEOUT_FULL;
    }
  }
  __syncwarp();
  const int row = (warp & 3) * 32 + lane, col0 = (warp >> 2) * 32;
  const uint32_t lanes = tmem + ((uint32_t)((warp & 3) * 32) << 16);
  bool ok = mbar_wait(&scored, 0);
  if (!ok && sp.status) *sp.status = ST_TIMEOUT_TMEM;
  __syncwarp();
  tc_fence_after_sync();
  {  // decayed scores of 32 columns; columns past the row's token are zero
    uint32_t hi[16], lo[16];
    if (col0 <= (warp & 3) * 32 + 31) {  // some row of this warp sees them
      uint32_t s[32];
      tmem_ld_32x32b_x32(lanes + col0, s);
      tmem_ld_wait_regs(s);
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        const int n = row - col0 - 2 * i;
        const float a = n >= 0 ? __uint_as_float(s[2 * i]) * power[n] : 0.f, b = n >= 1 ? __uint_as_float(s[2 * i + 1]) * power[n - 1] : 0.f;
        split2(a, b, hi[i], lo[i]);
      }
    } else {
#pragma unroll
      for (int i = 0; i < 16; ++i) hi[i] = lo[i] = 0u;
    }
    tmem_st_32x32b_x16(lanes + 128 + col0 / 2, hi);
    tmem_st_32x32b_x16(lanes + 192 + col0 / 2, lo);
  }
  tmem_st_wait();
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  if (tid == 0) {
    if (mbar_wait(&v_full, 0)) {
      tc_fence_after_sync();
#pragma unroll
      for (int k = 0; k < RT / 16; ++k) {
        const uint64_t v = make_smem_desc(base + L::V + k * 2048, RBOX, 1024);
        umma_bf16_ts(tmem + 384, tmem + 128 + k * 8, v, id_o, k > 0);
        umma_bf16_ts(tmem + 384, tmem + 192 + k * 8, v, id_o, 1);
      }
    } else if (sp.status) {
      *sp.status = ST_TIMEOUT_FULL;
    }
    umma_commit(&done);
  }
  __syncwarp();
  ok = mbar_wait(&done, 0) && ok;
  if (!ok && sp.status) *sp.status = ST_TIMEOUT_TMEM;
  __syncwarp();
  tc_fence_after_sync();
  const int t = at.t0 + row;
  const float e = power[row + 1];
  __nv_bfloat16* O = (__nv_bfloat16*)p.out + ((long long)at.b * p.rows + t) * p.ldo + at.h * p.Dv + at.c0 + col0;
  uint32_t a[32], b[32];
  tmem_ld_32x32b_x32(lanes + 256 + col0, a);
  tmem_ld_32x32b_x32(lanes + 384 + col0, b);
  tmem_ld_wait_regs(a);
  tmem_ld_wait_regs(b);
  if (ok && t < p.T) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      float f[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] = e * __uint_as_float(a[8 * i + j]) + __uint_as_float(b[8 * i + j]);
      if (col0 + 8 * i < at.ncol) st8v(O + 8 * i, f);  // Dv is a multiple of eight
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  if (warp == 0) tmem_dealloc(tmem, 512);
}

template <int DKB>
void run_out(const CUtensorMap& tv, const RetParams& sp, int blocks, cudaStream_t s) {
  const RecurrentArgs& a = sp.a;
  const uint64_t planes = (uint64_t)a.B * a.H * sp.nchunks, row = a.Dv * 2ull, plane = (uint64_t)a.Dk * a.Dv * 2;
  const CUtensorMap th = make_tmap_3d(sp.hi, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a.Dv, a.Dk, planes, row, plane, 64, DKB * 64);
  const CUtensorMap tl = make_tmap_3d(sp.lo, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a.Dv, a.Dk, planes, row, plane, 64, DKB * 64);
  constexpr int smem = RetSmem<DKB>::END + 1024;
  static_assert(smem <= 227 * 1024, "shared memory of a block");
  cudaFuncSetAttribute(retention_out_kernel<DKB>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  retention_out_kernel<DKB><<<blocks, RTH, smem, s>>>(tv, th, tl, sp);
  check_launch("retention_out");
}

long long planes_of(const RecurrentArgs& a) { return (long long)a.B * a.H * ((a.T + RT - 1) / RT) * a.Dk * a.Dv; }

}  // namespace

bool retention_tc_supported(const RecurrentArgs& a) {
  return !a.f32 && a.kind == RK_RETENTION && a.T >= 64 && a.Dk <= 128 && a.Dk % 8 == 0 && a.Dv % 8 == 0 && a.rot_dims % 16 == 0 &&
         vec8_ok(a.q, a.ldq, false) && vec8_ok(a.k, a.ldk, false) && vec8_ok(a.v, a.ldv, false) && vec8_ok(a.out, a.ldo, false) &&
         vec8_ok(a.state, 4, true) && vec8_ok(a.rot, 4, true);
}

long long retention_tc_scratch(const RecurrentArgs& a) { return planes_of(a) * 8; }

void launch_retention_tc(const RecurrentArgs& a, void* scratch, int* status, cudaStream_t s) {
  if (a.B <= 0 || a.T <= 0) return;
  if (!retention_tc_supported(a)) throw std::runtime_error("retention_tc: unsupported shape");
  RetParams sp{};
  sp.a = a;
  sp.nchunks = (a.T + RT - 1) / RT;
  sp.own = (float*)scratch;
  sp.hi = (__nv_bfloat16*)(sp.own + planes_of(a));
  sp.lo = sp.hi + planes_of(a);
  sp.status = status;
  const CUtensorMap tv = make_tmap_4d_bf16(a.v, {(uint64_t)a.Dv, (uint64_t)a.T, (uint64_t)a.H, (uint64_t)a.B},
                                           {a.ldv * 2ull, a.Dv * 2ull, (uint64_t)a.rows * a.ldv * 2}, RT);
  const int blocks = a.B * a.H * sp.nchunks * ((a.Dv + RCOLS - 1) / RCOLS);
  cudaFuncSetAttribute(retention_states_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, RS_SMEM);
  retention_states_kernel<<<blocks, RTH, RS_SMEM, s>>>(tv, sp);
  check_launch("retention_states");
  retention_scan_kernel<<<dim3((unsigned)(((long long)a.Dk * a.Dv + 1023) / 1024), a.B * a.H), 256, 0, s>>>(sp);
  check_launch("retention_scan");
  if (a.Dk <= 64) run_out<1>(tv, sp, blocks, s);
  else run_out<2>(tv, sp, blocks, s);
}

}  // namespace tb
