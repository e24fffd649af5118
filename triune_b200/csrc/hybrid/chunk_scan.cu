// Chunk-parallel form of the matrix-state recurrences (Mamba-2 and gated delta rule) for prompts, bf16 inputs, with the
// arithmetic of the recurrence kept at 32-bit grade.
//
// With b_i the running sum of the log decays inside a chunk of 64 tokens and S_0 the state before it:
//   delta:   (I + L) U = R,  L_ij = beta_i e^{b_i-b_j} k_i.k_j (j < i),  R_i = beta_i (v_i - e^{b_i} S_0^T k_i)
//   mamba2:  u_j = dt_j x_j
//   out_i = e^{b_i} S_0^T q_i + sum_{j<=i} e^{b_i-b_j} (q_i.k_j) u_j,      S_64 = e^{b_64} S_0 + sum_j e^{b_64-b_j} k_j u_j^T
//
// Precision. Queries, keys and values are bf16 as stored (the unit-norm factors of the delta rule are applied as fp32
// scalars to the products), so they enter the tensor core exactly. Every other operand (state, decayed scores, the
// triangle's inverse, U) is fp32 and enters as the sum of two bf16 numbers; products of two such operands take three
// MMAs. Accumulators, decays and the carried state are fp32.
//
// Two kernels. (1) Scores, parallel over chunks: q k^T per key group (mamba2), or per head the decayed q k^T and the
// inverse of I + L (delta). They are written in the register order of the B operand they become, one 16-byte vector per
// lane. (2) The walk. Delta rule: a block owns 16 value columns of a head and walks the chunks; its eight warps split the tokens for
// the outputs and the key dimensions for the state, which stays in accumulator registers as S^T [columns, Dk] and is
// handed between warps as bf16 pairs in shared memory; Mamba-2: see below. A walk is one long dependent chain, so what can be formed ahead of
// it is: the per-token factors (decays, gates, unit norms) are written by the scores kernel or a small kernel before it. The products here are small, chained and
// re-split between steps, so they run on mma.sync register fragments: the accumulator layout of one product is the
// operand layout of the next, with no trip through TMEM or shared memory in between.
#include "../common/ptx.cuh"
#include "hybrid.cuh"
#include "tc_tiles.cuh"

namespace tb {
namespace {

__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p))
               : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p))
               : "memory");
}
// Rows [t0, t0 + 64) x [0, D) of a bf16 matrix into shared memory [64][pitch]; rows past T and columns past D are zero.
// `vec`: 16-byte asynchronous copies (D a multiple of 8, aligned rows), otherwise plain stores.
template <int COLS, int PITCH>
__device__ __forceinline__ void stage_rows(__nv_bfloat16* dst, const __nv_bfloat16* src, long long ld, int t0, int T, int D,
                                           bool vec, int tid, int nt) {
  if (vec) {
    for (int i = tid; i < CL * (COLS / 8); i += nt) {
      const int r = i / (COLS / 8), c = (i % (COLS / 8)) * 8;
      __nv_bfloat16* d = dst + r * PITCH + c;
      if (t0 + r < T && c < D)
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(d)), "l"(src + (long long)(t0 + r) * ld + c) : "memory");
      else
        *reinterpret_cast<uint4*>(d) = make_uint4(0u, 0u, 0u, 0u);
    }
  } else {
    for (int i = tid; i < CL * COLS; i += nt) {
      const int r = i / COLS, c = i % COLS;
      dst[r * PITCH + c] = t0 + r < T && c < D ? src[(long long)(t0 + r) * ld + c] : __float2bfloat16(0.f);
    }
  }
}
// Per-token factors of the walk, [B, H, nchunks][FACTORS][64] fp32 (b is the running log decay of the chunk):
//   mamba2:  0 b   1 dt   2 dt e^{b_end - b}   3 e^{b_end} in entry 0
//   delta:   0 beta   1 beta e^b / |k|   2 e^{b_end - b} / |k|   3 e^b Dk^-1/2 / |q|   4 e^{b_end} in entry 0
constexpr int FACTORS = 5;

struct ScanParams {
  RecurrentArgs a;
  int nchunks;
  bool vec_qk, vec_v;
  uint4* frag0;   // mamba2: [B, KG, nchunks][8][4][32] fp32 scores; delta: [B, H, nchunks][8][4][32] decayed q k^T (hi, lo)
  uint4* frag1;   // delta: the same of the inverse
  float* fac;
};

// ------------------------------------------------------------------------------------------------ scores
template <int KIND, int DK>
__global__ void __launch_bounds__(128) chunk_scores_kernel(const ScanParams sp) {
  constexpr int P = DK + 8;
  extern __shared__ __align__(16) uint8_t raw[];
  __nv_bfloat16 *sQ = reinterpret_cast<__nv_bfloat16*>(raw), *sK = sQ + CL * P;
  const RecurrentArgs& p = sp.a;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int heads = KIND == RK_DELTA ? p.H : p.KG;
  const int c = blockIdx.x % sp.nchunks, bh = blockIdx.x / sp.nchunks, h = bh % heads, b = bh / heads;
  const int kh = KIND == RK_DELTA ? h / (p.H / p.KG) : h, t0 = c * CL;
  const __nv_bfloat16 *Q = (const __nv_bfloat16*)p.q + (long long)b * p.rows * p.ldq + kh * p.Dk,
                      *K = (const __nv_bfloat16*)p.k + (long long)b * p.rows * p.ldk + kh * p.Dk;
  stage_rows<DK, P>(sQ, Q, p.ldq, t0, p.T, p.Dk, sp.vec_qk, tid, 128);
  stage_rows<DK, P>(sK, K, p.ldk, t0, p.T, p.Dk, sp.vec_qk, tid, 128);
  cp_commit();
  __shared__ float sb[CL], sgate[CL], srk[CL], srq[CL];
  if (KIND == RK_DELTA && warp == 0) {
    const __nv_bfloat16 *A = (const __nv_bfloat16*)p.a + (long long)b * p.rows * p.lda + h, *Bt = (const __nv_bfloat16*)p.b + (long long)b * p.rows * p.ldb + h;
    const int t = t0 + 2 * lane;
    chunk_scalars(p, load_or0(A, p.lda, t, p.T), load_or0(A, p.lda, t + 1, p.T), load_or0(Bt, p.ldb, t, p.T), load_or0(Bt, p.ldb, t + 1, p.T),
                  expf(p.A_log[h]), p.dt_bias[h], t0, sb, sgate);
  }
  cp_wait0();
  __syncthreads();
  if (KIND == RK_DELTA) {  // unit-norm factors: two threads per row
    const int r = tid >> 1;
    float kk = 0.f, qq = 0.f;
    for (int d = (tid & 1) * 2; d < DK; d += 4) {
      const uint32_t kv = *reinterpret_cast<const uint32_t*>(sK + r * P + d), qv = *reinterpret_cast<const uint32_t*>(sQ + r * P + d);
      kk += lo_f(kv) * lo_f(kv) + hi_f(kv) * hi_f(kv);
      qq += lo_f(qv) * lo_f(qv) + hi_f(qv) * hi_f(qv);
    }
    kk += __shfl_xor_sync(0xffffffffu, kk, 1);
    qq += __shfl_xor_sync(0xffffffffu, qq, 1);
    if ((tid & 1) == 0) {
      srk[r] = 1.f / sqrtf(kk + p.unit_eps);
      srq[r] = 1.f / (sqrtf(qq + p.unit_eps) * sqrtf((float)p.Dk));
      float* f = sp.fac + ((long long)bh * sp.nchunks + c) * FACTORS * CL;
      f[r] = sgate[r];
      f[CL + r] = sgate[r] * exp_neg(sb[r]) * srk[r];
      f[2 * CL + r] = exp_neg(sb[CL - 1] - sb[r]) * srk[r];
      f[3 * CL + r] = exp_neg(sb[r]) * srq[r];
      f[4 * CL + r] = exp_neg(sb[CL - 1]);
    }
    __syncthreads();
  }
  // warp w: rows i of tile w against all columns j up to the diagonal. As a B operand row i is n, column j is k, and the
  // accumulator of (A = K tile rows j, B = Q rows i) has rows j and columns i, so compute it transposed: A = rows i.
  float* sL = reinterpret_cast<float*>(sK + CL * P);  // delta: L, then its inverse, [64][65]
  uint32_t aq[4], ak[4], bk[4];
  float gq[8][4], gk[8][4];
#pragma unroll
  for (int n = 0; n < 8; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) gq[n][i] = gk[n][i] = 0.f;
#pragma unroll
  for (int ks = 0; ks < DK / 16; ++ks) {
    const int ar = warp * 16 + (lane & 15), ac = ks * 16 + (lane >> 4) * 8;
    ldsm4(aq, sQ + ar * P + ac);
    if (KIND == RK_DELTA) ldsm4(ak, sK + ar * P + ac);
#pragma unroll
    for (int nn = 0; nn < 4; ++nn) {  // 16 columns j at a time
      if (nn > warp) break;
      const int br = nn * 16 + (lane & 7) + ((lane >> 4) << 3), bc = ks * 16 + ((lane >> 3) & 1) * 8;
      ldsm4(bk, sK + br * P + bc);
      mma16816(gq[2 * nn], aq, bk[0], bk[1]);
      mma16816(gq[2 * nn + 1], aq, bk[2], bk[3]);
      if (KIND == RK_DELTA) {
        mma16816(gk[2 * nn], ak, bk[0], bk[1]);
        mma16816(gk[2 * nn + 1], ak, bk[2], bk[3]);
      }
    }
  }
  // accumulator [n][e]: row i = 16 warp + lane / 4 (+ 8 for e >= 2), column j = 8 n + 2 (lane % 4) + (e & 1).
  // Fragment of row tile it (8 rows), column step kt (16): lane l holds (i = l / 4, j = 2 (l % 4) + {0, 1}) and j + 8: the
  // rows of this lane are the same, so it owns whole fragments: row tile 2 warp from e = 0, 1 and 2 warp + 1 from e = 2, 3.
  const long long base = ((long long)bh * sp.nchunks + c) * 8 * 4 * 32;
  if constexpr (KIND == RK_MAMBA2) {
#pragma unroll
    for (int half = 0; half < 2; ++half)
#pragma unroll
      for (int kt = 0; kt < 4; ++kt) {
        if (kt > warp) break;
        uint4 v;
        v.x = __float_as_uint(gq[2 * kt][2 * half]);
        v.y = __float_as_uint(gq[2 * kt][2 * half + 1]);
        v.z = __float_as_uint(gq[2 * kt + 1][2 * half]);
        v.w = __float_as_uint(gq[2 * kt + 1][2 * half + 1]);
        sp.frag0[base + ((2 * warp + half) * 4 + kt) * 32 + lane] = v;
      }
  } else {
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int i = 16 * warp + 8 * half + (lane >> 2);
      const float bi = sb[i], si = srq[i], gi = sgate[i] * srk[i];
#pragma unroll
      for (int kt = 0; kt < 4; ++kt) {
        if (kt > warp) break;
        float pv[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int n = 2 * kt + (e >> 1), j = 8 * n + 2 * (lane & 3) + (e & 1);
          const float dec = j <= i ? exp_neg(bi - sb[j]) * srk[j] : 0.f;
          pv[e] = gq[n][2 * half + (e & 1)] * si * dec;
          sL[i * 65 + j] = j < i ? gk[n][2 * half + (e & 1)] * gi * dec : 0.f;
        }
        uint4 v;
        split2(pv[0], pv[1], v.x, v.z);
        split2(pv[2], pv[3], v.y, v.w);
        sp.frag0[base + ((2 * warp + half) * 4 + kt) * 32 + lane] = v;  // (hi b0, hi b1, lo b0, lo b1)
      }
    }
    __syncthreads();
    // inverse of I + L, a thread per column: T_ij = -sum_{j <= m < i} L_im T_mj, in 16-row blocks so that the running
    // column sits in registers while L is read as broadcasts
    float* sT = sL + CL * 65;
    if (tid < CL) {
      const int j = tid;
      for (int i = 0; i < CL; ++i) sT[i * 65 + j] = i == j ? 1.f : 0.f;
      for (int i0 = 0; i0 < CL; i0 += 16) {
        float acc[16];
#pragma unroll
        for (int r = 0; r < 16; ++r) acc[r] = 0.f;
        for (int m = 0; m < i0; ++m) {
          const float t = sT[m * 65 + j];
#pragma unroll
          for (int r = 0; r < 16; ++r) acc[r] += sL[(i0 + r) * 65 + m] * t;
        }
        float col[16];
#pragma unroll
        for (int r = 0; r < 16; ++r) {
          float s = acc[r];
#pragma unroll
          for (int m = 0; m < r; ++m) s += sL[(i0 + r) * 65 + i0 + m] * col[m];
          col[r] = i0 + r == j ? 1.f : (i0 + r > j ? -s : 0.f);
          sT[(i0 + r) * 65 + j] = col[r];
        }
      }
    }
    __syncthreads();
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int i = 16 * warp + 8 * half + (lane >> 2);
      for (int kt = 0; kt <= warp; ++kt) {
        const float* tr = sT + i * 65 + 16 * kt + 2 * (lane & 3);
        uint4 v;
        split2(tr[0], tr[1], v.x, v.z);
        split2(tr[8], tr[9], v.y, v.w);
        sp.frag1[base + ((2 * warp + half) * 4 + kt) * 32 + lane] = v;
      }
    }
  }
}

// Factors of mamba2, a warp per (batch, head, chunk).
__global__ void __launch_bounds__(128) chunk_factors_kernel(const ScanParams sp) {
  __shared__ float sb[4][CL], sg[4][CL];
  const RecurrentArgs& p = sp.a;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long id = (long long)blockIdx.x * 4 + warp;
  if (id >= (long long)p.B * p.H * sp.nchunks) return;
  const int c = (int)(id % sp.nchunks), bh = (int)(id / sp.nchunks), h = bh % p.H, b = bh / p.H, t = c * CL + 2 * lane;
  const __nv_bfloat16* A = (const __nv_bfloat16*)p.a + (long long)b * p.rows * p.lda + h;
  chunk_scalars(p, load_or0(A, p.lda, t, p.T), load_or0(A, p.lda, t + 1, p.T), 0.f, 0.f, expf(p.A_log[h]), p.dt_bias[h], c * CL, sb[warp], sg[warp]);
  __syncwarp();
  float* f = sp.fac + id * FACTORS * CL;
  const float bl = sb[warp][CL - 1];
#pragma unroll
  for (int i = lane; i < CL; i += 32) {
    f[i] = sb[warp][i];
    f[CL + i] = sg[warp][i];
    f[2 * CL + i] = sg[warp][i] * exp_neg(bl - sb[warp][i]);
    f[3 * CL + i] = exp_neg(bl);
  }
}

// ------------------------------------------------------------------------------------------------ delta rule: walk
constexpr int WW = 8, WCOLS = 16;  // warps and value columns of a block; a warp owns 8 tokens and DK / 8 key dimensions

template <int DK>
struct WalkSmem {
  static constexpr int P = DK + 8, PV = WCOLS + 8, PR = CL + 8;
  __nv_bfloat16 q[2][CL * P], k[2][CL * P], v[2][CL * PV];
  __nv_bfloat16 s[2][2][WCOLS * P];     // state buffer, hi / lo, [columns][Dk]
  __nv_bfloat16 r[3][2][WCOLS * PR];   // 0: weighted U of the state update, 1: R, 2: U; hi / lo, [columns][tokens]
  __nv_bfloat16 o[CL * PV];
  float f[2][FACTORS * CL];
};

__device__ __forceinline__ void ldsm2t(uint32_t& r0, uint32_t& r1, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(smem_u32(p)) : "memory");
}

template <int DK>
__global__ void __launch_bounds__(32 * WW) delta_walk_kernel(const ScanParams sp) {
  using Sm = WalkSmem<DK>;
  constexpr int P = Sm::P, PV = Sm::PV, PR = Sm::PR, NT = 32 * WW, KT = DK / 16, DW = DK / WW, NU = DW / 8;
  extern __shared__ __align__(16) uint8_t raw[];
  Sm& sm = *reinterpret_cast<Sm*>(raw);
  const RecurrentArgs& p = sp.a;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int slices = (p.Dv + WCOLS - 1) / WCOLS;
  const int slice = blockIdx.x % slices, bh = blockIdx.x / slices, h = bh % p.H, b = bh / p.H;
  const int kh = h / (p.H / p.KG), c0 = slice * WCOLS, ncol = min(WCOLS, p.Dv - c0);
  const __nv_bfloat16 *Q = (const __nv_bfloat16*)p.q + (long long)b * p.rows * p.ldq + kh * p.Dk,
                      *K = (const __nv_bfloat16*)p.k + (long long)b * p.rows * p.ldk + kh * p.Dk,
                      *V = (const __nv_bfloat16*)p.v + (long long)b * p.rows * p.ldv + h * p.Dv + c0;
  __nv_bfloat16* O = (__nv_bfloat16*)p.out + (long long)b * p.rows * p.ldo + h * p.Dv + c0;
  const uint4 *f0 = sp.frag0 + (long long)bh * sp.nchunks * 1024, *f1 = sp.frag1 + (long long)bh * sp.nchunks * 1024;
  const float* fac = sp.fac + (long long)bh * sp.nchunks * FACTORS * CL;

  auto stage = [&](int c) {
    const int t0 = c * CL, u = c & 1;
    stage_rows<DK, P>(sm.q[u], Q, p.ldq, t0, p.T, p.Dk, sp.vec_qk, tid, NT);
    stage_rows<DK, P>(sm.k[u], K, p.ldk, t0, p.T, p.Dk, sp.vec_qk, tid, NT);
    stage_rows<WCOLS, PV>(sm.v[u], V, p.ldv, t0, p.T, ncol, sp.vec_v, tid, NT);
    if (tid < FACTORS * CL / 4)
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(sm.f[u] + tid * 4)), "l"(fac + (long long)c * FACTORS * CL + tid * 4) : "memory");
    cp_commit();
  };

  // this warp's part of the state: columns lane / 4 and + 8, key dimensions warp DW + 8 n + 2 (lane % 4) + {0, 1}
  float S[NU][4];
  float* st = p.state + (long long)bh * p.Dk * p.Dv;
  const int col = lane >> 2, pair = 2 * (lane & 3), d_lo = warp * DW + pair;
#pragma unroll
  for (int n = 0; n < NU; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = d_lo + 8 * n + (e & 1), cc = col + (e >> 1) * 8;
      S[n][e] = d < p.Dk && cc < ncol ? st[(long long)d * p.Dv + c0 + cc] : 0.f;
    }
  auto publish = [&](int buf) {
#pragma unroll
    for (int n = 0; n < NU; ++n)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t hi, lo;
        split2(S[n][2 * half], S[n][2 * half + 1], hi, lo);
        const int at = (col + 8 * half) * P + d_lo + 8 * n;
        *reinterpret_cast<uint32_t*>(sm.s[buf][0] + at) = hi;
        *reinterpret_cast<uint32_t*>(sm.s[buf][1] + at) = lo;
      }
  };
  publish(0);
  stage(0);
  const int a_row = lane & 15, a_col = (lane >> 4) * 8;  // ldmatrix addresses of an A operand [column][k]
  const int tok0 = 8 * warp, wt = warp >> 1;             // this warp's tokens; their 16-token tile
  const int b_at = (tok0 + (lane & 7)) * P + (lane >> 3) * 8;  // B operand [token][k], two steps of 16 per load
  // a value pair of this lane's tokens, columns col and col + 8, as bf16 pairs into r[which]
  auto put = [&](int which, const float (&x)[4]) {
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      uint32_t hi, lo;
      split2(x[2 * half], x[2 * half + 1], hi, lo);
      const int at = (col + 8 * half) * PR + tok0 + pair;
      *reinterpret_cast<uint32_t*>(sm.r[which][0] + at) = hi;
      *reinterpret_cast<uint32_t*>(sm.r[which][1] + at) = lo;
    }
  };

  for (int c = 0; c < sp.nchunks; ++c) {
    const int u = c & 1, t0 = c * CL;
    cp_wait0();
    __syncthreads();  // tile c, its factors and the state before it are in place; every warp has left chunk c - 1
    if (c + 1 < sp.nchunks) stage(c + 1);
    const float* F = sm.f[u];
    // score fragments of this warp's row tile: issued early, used after the state products
    uint4 fr[4], ft[4];
#pragma unroll
    for (int kt = 0; kt < 4; ++kt)
      if (kt <= wt) {
        fr[kt] = f0[(long long)c * 1024 + (warp * 4 + kt) * 32 + lane];
        ft[kt] = f1[(long long)c * 1024 + (warp * 4 + kt) * 32 + lane];
      }
    float x[4];  // values of this lane's tokens: [column half][token of the pair]
#pragma unroll
    for (int e = 0; e < 4; ++e) x[e] = __bfloat162float(sm.v[u][(tok0 + pair + (e & 1)) * PV + col + (e >> 1) * 8]);
    // state products of this warp's tokens: S^T q and S^T k (hi and lo in separate accumulators)
    float oq[4] = {0.f, 0.f, 0.f, 0.f}, oq2[4] = {0.f, 0.f, 0.f, 0.f}, ok[4] = {0.f, 0.f, 0.f, 0.f}, ok2[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int ks = 0; ks < KT; ks += 2) {
      uint32_t ah[2][4], al[2][4], bq[4], bk[4];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        ldsm4(ah[i], sm.s[u][0] + a_row * P + (ks + i) * 16 + a_col);
        ldsm4(al[i], sm.s[u][1] + a_row * P + (ks + i) * 16 + a_col);
      }
      ldsm4(bq, sm.q[u] + b_at + ks * 16);
      ldsm4(bk, sm.k[u] + b_at + ks * 16);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        mma16816(oq, ah[i], bq[2 * i], bq[2 * i + 1]);
        mma16816(oq2, al[i], bq[2 * i], bq[2 * i + 1]);
        {
          mma16816(ok, ah[i], bk[2 * i], bk[2 * i + 1]);
          mma16816(ok2, al[i], bk[2 * i], bk[2 * i + 1]);
        }
      }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      oq[e] += oq2[e];
      ok[e] += ok2[e];
    }
    {
      float r[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = tok0 + pair + (e & 1);
        oq[e] *= F[3 * CL + i];
        r[e] = F[i] * x[e] - F[CL + i] * ok[e];
      }
      put(1, r);
      __syncthreads();
      float uu[4] = {0.f, 0.f, 0.f, 0.f}, u2[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int kt = 0; kt < 4; ++kt) {
        if (kt > wt) break;
        uint32_t ah[4], al[4];
        ldsm4(ah, sm.r[1][0] + a_row * PR + kt * 16 + a_col);
        ldsm4(al, sm.r[1][1] + a_row * PR + kt * 16 + a_col);
        mma16816(uu, ah, ft[kt].x, ft[kt].y);
        mma16816(u2, ah, ft[kt].z, ft[kt].w);
        mma16816(u2, al, ft[kt].x, ft[kt].y);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) uu[e] += u2[e];
      put(2, uu);
      const float w0 = F[2 * CL + tok0 + pair], w1 = F[2 * CL + tok0 + pair + 1];
      const float uw[4] = {uu[0] * w0, uu[1] * w1, uu[2] * w0, uu[3] * w1};
      put(0, uw);
      __syncthreads();
    }
    // decay the state and add this chunk's keys: A = weighted U (columns x tokens), B = key rows
    const float dl = F[4 * CL];
#pragma unroll
    for (int n = 0; n < NU; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) S[n][e] *= dl;
#pragma unroll
    for (int kt = 0; kt < 4; ++kt) {
      uint32_t ah[4], al[4];
      ldsm4(ah, sm.r[0][0] + a_row * PR + kt * 16 + a_col);
      ldsm4(al, sm.r[0][1] + a_row * PR + kt * 16 + a_col);
      const __nv_bfloat16* kr = sm.k[u] + (kt * 16 + (lane & 15)) * P + warp * DW;  // key rows, transposed into B fragments
      if constexpr (NU == 2) {
        uint32_t bk[4];
        ldsm4t(bk, kr + (lane >> 4) * 8);
        mma16816(S[0], ah, bk[0], bk[1]);
        mma16816(S[1], ah, bk[2], bk[3]);
        mma16816(S[0], al, bk[0], bk[1]);
        mma16816(S[1], al, bk[2], bk[3]);
      } else {
        uint32_t k0, k1;
        ldsm2t(k0, k1, kr);
        mma16816(S[0], ah, k0, k1);
        mma16816(S[0], al, k0, k1);
      }
    }
    publish(u ^ 1);
    {
      float o2[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int kt = 0; kt < 4; ++kt) {
        if (kt > wt) break;
        uint32_t ah[4], al[4];
        ldsm4(ah, sm.r[2][0] + a_row * PR + kt * 16 + a_col);
        ldsm4(al, sm.r[2][1] + a_row * PR + kt * 16 + a_col);
        mma16816(oq, ah, fr[kt].x, fr[kt].y);
        mma16816(o2, ah, fr[kt].z, fr[kt].w);
        mma16816(o2, al, fr[kt].x, fr[kt].y);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) oq[e] += o2[e];
    }
    // outputs: transpose through shared memory (this warp's tokens only), then 16-byte rows
#pragma unroll
    for (int e = 0; e < 4; ++e) sm.o[(tok0 + pair + (e & 1)) * PV + col + (e >> 1) * 8] = __float2bfloat16(oq[e]);
    __syncwarp();
    if (lane < 16) {
      const int i = tok0 + (lane >> 1), cc = (lane & 1) * 8, t = t0 + i;
      if (t < p.T) {
        const __nv_bfloat16* src = sm.o + i * PV + cc;
        __nv_bfloat16* dst = O + (long long)t * p.ldo + cc;
        if (sp.vec_v && cc + 8 <= ncol) *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(src);
        else
          for (int e = 0; e < 8 && cc + e < ncol; ++e) dst[e] = src[e];
      }
    }
  }
#pragma unroll
  for (int n = 0; n < NU; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = d_lo + 8 * n + (e & 1), cc = col + (e >> 1) * 8;
      if (d < p.Dk && cc < ncol) st[(long long)d * p.Dv + c0 + cc] = S[n][e];
    }
}

// ------------------------------------------------------------------------------------------------ Mamba-2
// The state's transition is a scalar per head, so a sequence is cut into segments that are walked independently: one pass
// leaves every segment's own contribution to its end state, a small scan turns these into the state before every segment,
// and the second pass walks the segments again for the outputs. A block owns 64 value columns of a head (two halves of
// four warps); as output tiles [tokens, columns] the decayed scores are the A operand, formed in registers once for 32
// columns, and values, weighted values and the state [Dk, columns] are B operands.
constexpr int SW = 8, SC = 64;  // warps, value columns

template <int DK, bool OUT>
struct SsdSmem {
  static constexpr int P = DK + 8, PC = SC + 8;
  __nv_bfloat16 k[CL * P], x[CL * PC], w[2][CL * PC];
  __nv_bfloat16 q[OUT ? CL * P : 8], s[2][OUT ? DK * PC : 8];
  float f[4 * CL];
};

template <int DK, bool OUT>
__global__ void __launch_bounds__(32 * SW, 2) ssd_kernel(const ScanParams sp, float* seg_state, int seg_chunks, int nseg) {
  using Sm = SsdSmem<DK, OUT>;
  constexpr int P = Sm::P, PC = Sm::PC, NT = 32 * SW, KT = DK / 16, MU = DK / 64;  // MU: 16-row tiles of this warp's key dimensions
  extern __shared__ __align__(16) uint8_t raw[];
  Sm& sm = *reinterpret_cast<Sm*>(raw);
  const RecurrentArgs& p = sp.a;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, wt = warp & 3, wc = (warp >> 2) * 32;
  const int slices = (p.Dv + SC - 1) / SC;
  const int slice = blockIdx.x % slices, bh = blockIdx.x / slices, h = bh % p.H, b = bh / p.H, seg = blockIdx.y;
  const int kh = h / (p.H / p.KG), c0 = slice * SC, ncol = min(SC, p.Dv - c0);
  const __nv_bfloat16 *Q = (const __nv_bfloat16*)p.q + (long long)b * p.rows * p.ldq + kh * p.Dk,
                      *K = (const __nv_bfloat16*)p.k + (long long)b * p.rows * p.ldk + kh * p.Dk,
                      *V = (const __nv_bfloat16*)p.v + (long long)b * p.rows * p.ldv + h * p.Dv + c0;
  __nv_bfloat16* O = (__nv_bfloat16*)p.out + (long long)b * p.rows * p.ldo + h * p.Dv + c0;
  const float Dh = p.D[h];
  const float4* f0 = reinterpret_cast<const float4*>(sp.frag0) + ((long long)b * p.KG + kh) * sp.nchunks * 1024;
  const float* fac = sp.fac + (long long)bh * sp.nchunks * FACTORS * CL;
  const int first = seg * seg_chunks, last = min(first + seg_chunks, sp.nchunks);

  // accumulators of this warp's part of the state: key dimensions wt DK / 4 + 16 m + {lane / 4, + 8}, columns
  // wc + 8 n + 2 (lane % 4) + {0, 1}
  const int rl = lane >> 2, pair = 2 * (lane & 3), d0 = wt * (DK / 4);
  float S[MU][4][4];
  const long long plane = (long long)p.Dk * p.Dv;
  float* mine = nseg > 1 ? seg_state + ((long long)seg * p.B * p.H + bh) * plane : p.state + (long long)bh * plane;
#pragma unroll
  for (int m = 0; m < MU; ++m)
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = d0 + 16 * m + rl + (e >> 1) * 8, cc = wc + 8 * n + pair + (e & 1);
        S[m][n][e] = OUT && d < p.Dk && cc < ncol ? mine[(long long)d * p.Dv + c0 + cc] : 0.f;
      }
  auto publish = [&]() {
#pragma unroll
    for (int m = 0; m < MU; ++m)
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          uint32_t hi, lo;
          split2(S[m][n][2 * half], S[m][n][2 * half + 1], hi, lo);
          const int at = (d0 + 16 * m + rl + 8 * half) * PC + wc + 8 * n + pair;
          *reinterpret_cast<uint32_t*>(sm.s[0] + at) = hi;
          *reinterpret_cast<uint32_t*>(sm.s[1] + at) = lo;
        }
  };
  auto stage_kx = [&](int c) {
    stage_rows<DK, P>(sm.k, K, p.ldk, c * CL, p.T, p.Dk, sp.vec_qk, tid, NT);
    stage_rows<SC, PC>(sm.x, V, p.ldv, c * CL, p.T, ncol, sp.vec_v, tid, NT);
    if (tid < CL)
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(sm.f + tid * 4)), "l"(fac + (long long)c * FACTORS * CL + tid * 4) : "memory");
  };
  auto stage_q = [&](int c) {
    if constexpr (OUT) stage_rows<DK, P>(sm.q, Q, p.ldq, c * CL, p.T, p.Dk, sp.vec_qk, tid, NT);
  };
  if (first < last) {
    stage_q(first);
    stage_kx(first);
    cp_commit();
  }
  if constexpr (OUT) publish();
  float decay = 1.f;  // of the whole segment
  const int nt_row = (lane & 7) + ((lane >> 4) << 3), nt_col = ((lane >> 3) & 1) * 8;  // transposed A: stored [k][row]
  const int tr_row = lane & 15, tr_col = (lane >> 4) * 8;                              // A [row][k]; transposed B: stored [k][n]

  for (int c = first; c < last; ++c) {
    const int t0 = c * CL;
    float4 fr[2][OUT ? 4 : 1];
    if constexpr (OUT) {
#pragma unroll
      for (int kt = 0; kt < 4; ++kt)
        if (kt <= wt)
#pragma unroll
          for (int i = 0; i < 2; ++i) fr[i][kt] = f0[(long long)c * 1024 + ((2 * wt + i) * 4 + kt) * 32 + lane];
    }
    cp_wait0();
    __syncthreads();  // the chunk's tiles and the state before it
    const float* F = sm.f;
    {  // weighted values of 16 tokens x 32 columns: a lane has 16 columns of one token
      const int t = 16 * wt + (lane >> 1), at = t * PC + wc + (lane & 1) * 16;
      const float w = F[2 * CL + t];
#pragma unroll
      for (int g = 0; g < 2; ++g) {
        const uint4 v = *reinterpret_cast<const uint4*>(sm.x + at + 8 * g);
        uint4 hi, lo;
        split2(lo_f(v.x) * w, hi_f(v.x) * w, hi.x, lo.x);
        split2(lo_f(v.y) * w, hi_f(v.y) * w, hi.y, lo.y);
        split2(lo_f(v.z) * w, hi_f(v.z) * w, hi.z, lo.z);
        split2(lo_f(v.w) * w, hi_f(v.w) * w, hi.w, lo.w);
        *reinterpret_cast<uint4*>(sm.w[0] + at + 8 * g) = hi;
        *reinterpret_cast<uint4*>(sm.w[1] + at + 8 * g) = lo;
      }
    }
    if constexpr (OUT) {
      float o[4][4];
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[n][e] = 0.f;
#pragma unroll
      for (int ks = 0; ks < KT; ++ks) {
        uint32_t aq[4];
        ldsm4(aq, sm.q + (16 * wt + tr_row) * P + ks * 16 + tr_col);
#pragma unroll
        for (int n2 = 0; n2 < 2; ++n2) {
          uint32_t bh4[4], bl4[4];
          const int at = (ks * 16 + tr_row) * PC + wc + n2 * 16 + tr_col;
          ldsm4t(bh4, sm.s[0] + at);
          ldsm4t(bl4, sm.s[1] + at);
          mma16816(o[2 * n2], aq, bh4[0], bh4[1]);
          mma16816(o[2 * n2 + 1], aq, bh4[2], bh4[3]);
          mma16816(o[2 * n2], aq, bl4[0], bl4[1]);
          mma16816(o[2 * n2 + 1], aq, bl4[2], bl4[3]);
        }
      }
      // e^{b_i - b_j} = e^{b_i - b_ref} e^{b_ref - b_j} for tokens j before this tile, the tile's first token as reference:
      // both factors are at most 1, and the first is applied once to the whole sum; within the tile, pair by pair
      const float br = F[16 * wt], er = exp_neg(br), bi0 = F[16 * wt + rl], bi1 = F[16 * wt + rl + 8];
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[n][e] *= er;
#pragma unroll
      for (int kt = 0; kt < 4; ++kt) {
        if (kt > wt) break;
        const int j = kt * 16 + pair;
        const float2 b0 = *reinterpret_cast<const float2*>(F + j), b8 = *reinterpret_cast<const float2*>(F + j + 8);
        const float2 g0 = *reinterpret_cast<const float2*>(F + CL + j), g8 = *reinterpret_cast<const float2*>(F + CL + j + 8);
        uint32_t ah[4], al[4];
        if (kt < wt) {
          const float w0 = g0.x * exp_neg(br - b0.x), w1 = g0.y * exp_neg(br - b0.y), w8 = g8.x * exp_neg(br - b8.x), w9 = g8.y * exp_neg(br - b8.y);
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            split2(fr[i][kt].x * w0, fr[i][kt].y * w1, ah[i], al[i]);
            split2(fr[i][kt].z * w8, fr[i][kt].w * w9, ah[2 + i], al[2 + i]);
          }
        } else {
          const float s0 = exp_neg(bi0 - br), s1 = exp_neg(bi1 - br);
#pragma unroll
          for (int n = 0; n < 4; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) o[n][e] *= e < 2 ? s0 : s1;
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const int row = 16 * wt + rl + 8 * i;
            const float bi = i == 0 ? bi0 : bi1;
            const float m0 = j <= row ? fr[i][kt].x * g0.x * exp_neg(bi - b0.x) : 0.f, m1 = j + 1 <= row ? fr[i][kt].y * g0.y * exp_neg(bi - b0.y) : 0.f;
            const float m8 = j + 8 <= row ? fr[i][kt].z * g8.x * exp_neg(bi - b8.x) : 0.f, m9 = j + 9 <= row ? fr[i][kt].w * g8.y * exp_neg(bi - b8.y) : 0.f;
            split2(m0, m1, ah[i], al[i]);
            split2(m8, m9, ah[2 + i], al[2 + i]);
          }
        }
#pragma unroll
        for (int n2 = 0; n2 < 2; ++n2) {
          uint32_t bx[4];
          ldsm4t(bx, sm.x + (kt * 16 + tr_row) * PC + wc + n2 * 16 + tr_col);
          mma16816(o[2 * n2], ah, bx[0], bx[1]);
          mma16816(o[2 * n2 + 1], ah, bx[2], bx[3]);
          mma16816(o[2 * n2], al, bx[0], bx[1]);
          mma16816(o[2 * n2 + 1], al, bx[2], bx[3]);
        }
      }
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int i = 16 * wt + rl + 8 * half, t = t0 + i;
        if (t < p.T) {
          __nv_bfloat16* dst = O + (long long)t * p.ldo;
#pragma unroll
          for (int n = 0; n < 4; ++n) {
            const int cc = wc + 8 * n + pair;
            const uint32_t xv = *reinterpret_cast<const uint32_t*>(sm.x + i * PC + cc);
            const uint32_t y = pack_bf16x2(o[n][2 * half] + Dh * lo_f(xv), o[n][2 * half + 1] + Dh * hi_f(xv));
            if (sp.vec_v && cc < ncol) *reinterpret_cast<uint32_t*>(dst + cc) = y;
            else {
              if (cc < ncol) dst[cc] = __float2bfloat16(lo_f(y));
              if (cc + 1 < ncol) dst[cc + 1] = __float2bfloat16(hi_f(y));
            }
          }
        }
      }
    }
    __syncthreads();  // every warp's weighted values are there; queries and the published state have been read
    const bool more = c + 1 < last;
    if (more) stage_q(c + 1);
    const float dl = F[3 * CL];
    decay *= dl;
#pragma unroll
    for (int m = 0; m < MU; ++m)
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[m][n][e] *= dl;
#pragma unroll
    for (int kt = 0; kt < 4; ++kt) {
      uint32_t ak[MU][4];
#pragma unroll
      for (int m = 0; m < MU; ++m) ldsm4t(ak[m], sm.k + (kt * 16 + nt_row) * P + d0 + 16 * m + nt_col);
#pragma unroll
      for (int n2 = 0; n2 < 2; ++n2) {
        uint32_t wh[4], wl[4];
        const int at = (kt * 16 + tr_row) * PC + wc + n2 * 16 + tr_col;
        ldsm4t(wh, sm.w[0] + at);
        ldsm4t(wl, sm.w[1] + at);
#pragma unroll
        for (int m = 0; m < MU; ++m) {
          mma16816(S[m][2 * n2], ak[m], wh[0], wh[1]);
          mma16816(S[m][2 * n2 + 1], ak[m], wh[2], wh[3]);
          mma16816(S[m][2 * n2], ak[m], wl[0], wl[1]);
          mma16816(S[m][2 * n2 + 1], ak[m], wl[2], wl[3]);
        }
      }
    }
    if constexpr (OUT) publish();
    if (more) {
      __syncthreads();  // keys, values and factors have been read
      stage_kx(c + 1);
      cp_commit();
    }
  }
  if (!OUT || seg == nseg - 1) {
    float* dst = OUT ? p.state + (long long)bh * plane : mine;
#pragma unroll
    for (int m = 0; m < MU; ++m)
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int d = d0 + 16 * m + rl + (e >> 1) * 8, cc = wc + 8 * n + pair + (e & 1);
          if (d < p.Dk && cc < ncol) dst[(long long)d * p.Dv + c0 + cc] = S[m][n][e];
        }
    if (!OUT && slice == 0 && tid == 0) seg_state[(long long)nseg * p.B * p.H * plane + (long long)seg * p.B * p.H + bh] = decay;
  }
}

// seg_state: own contribution of every segment but the last -> state before every segment; the segments' decays follow
// the states. grid (ceil(plane / 256), B H)
__global__ void ssd_scan_kernel(const RecurrentArgs p, float* seg_state, int nseg) {
  const long long plane = (long long)p.Dk * p.Dv, bh = blockIdx.y, heads = (long long)p.B * p.H;
  const float* dec = seg_state + nseg * heads * plane + bh;
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= plane) return;
  float run = p.state[bh * plane + i];
  float* at = seg_state + bh * plane + i;
  for (int g0 = 0; g0 < nseg - 1; g0 += 8) {  // loads first: they do not wait for one another
    float own[8], d[8];
#pragma unroll
    for (int g = 0; g < 8; ++g)
      if (g0 + g < nseg - 1) {
        own[g] = at[(g0 + g) * heads * plane];
        d[g] = dec[(g0 + g) * heads];
      }
#pragma unroll
    for (int g = 0; g < 8; ++g)
      if (g0 + g < nseg - 1) {
        at[(g0 + g) * heads * plane] = run;
        run = d[g] * run + own[g];
      }
  }
  at[(nseg - 1) * heads * plane] = run;
}

// Segments so that about two blocks per SM walk; none where the heads alone fill the machine.
int ssd_segments(const RecurrentArgs& a) {
  const int blocks = a.B * a.H * ((a.Dv + SC - 1) / SC), n = (a.T + CL - 1) / CL;
  int s = (2 * 148) / blocks;
  s = s > n / 4 ? n / 4 : s;
  s = s > 64 ? 64 : s;
  return s < 2 ? 1 : s;
}

template <int KIND, int DK>
void run_scores(const ScanParams& sp, cudaStream_t s) {
  const RecurrentArgs& a = sp.a;
  auto kern = chunk_scores_kernel<KIND, DK>;
  constexpr int smem = 2 * CL * (DK + 8) * 2 + (KIND == RK_DELTA ? 2 * CL * 65 * 4 : 0);
  cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  kern<<<a.B * (KIND == RK_DELTA ? a.H : a.KG) * sp.nchunks, 128, smem, s>>>(sp);
  check_launch("chunk_scores");
}

template <int DK>
void run_delta(const ScanParams& sp, cudaStream_t s) {
  const RecurrentArgs& a = sp.a;
  run_scores<RK_DELTA, DK>(sp, s);
  auto walk = delta_walk_kernel<DK>;
  constexpr int smem = (int)sizeof(WalkSmem<DK>);
  cudaFuncSetAttribute(walk, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  walk<<<a.B * a.H * ((a.Dv + WCOLS - 1) / WCOLS), 32 * WW, smem, s>>>(sp);
  check_launch("delta_walk");
}

template <int DK>
void run_ssd(const ScanParams& sp, float* seg_state, cudaStream_t s) {
  const RecurrentArgs& a = sp.a;
  run_scores<RK_MAMBA2, DK>(sp, s);
  const long long n = (long long)a.B * a.H * sp.nchunks;
  chunk_factors_kernel<<<(unsigned)((n + 3) / 4), 128, 0, s>>>(sp);
  check_launch("chunk_factors");
  const int want = ssd_segments(a), per = (sp.nchunks + want - 1) / want, nseg = (sp.nchunks + per - 1) / per;
  const dim3 grid(a.B * a.H * ((a.Dv + SC - 1) / SC), nseg);
  if (nseg > 1) {
    auto own = ssd_kernel<DK, false>;
    constexpr int smem = (int)sizeof(SsdSmem<DK, false>);
    cudaFuncSetAttribute(own, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    own<<<dim3(grid.x, nseg - 1), 32 * SW, smem, s>>>(sp, seg_state, per, nseg);
    check_launch("ssd_states");
    launch_ssd_scan(a, seg_state, nseg, s);
  }
  auto out = ssd_kernel<DK, true>;
  constexpr int smem = (int)sizeof(SsdSmem<DK, true>);
  cudaFuncSetAttribute(out, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  out<<<grid, 32 * SW, smem, s>>>(sp, seg_state, per, nseg);
  check_launch("ssd_out");
}

}  // namespace

void launch_ssd_scan(const RecurrentArgs& a, float* seg_state, int nseg, cudaStream_t s) {
  ssd_scan_kernel<<<dim3((unsigned)(((long long)a.Dk * a.Dv + 255) / 256), a.B * a.H), 256, 0, s>>>(a, seg_state, nseg);
  check_launch("ssd_scan");
}

bool chunk_scan_supported(const RecurrentArgs& a) { return a.kind != RK_RETENTION && !a.f32 && a.Dk <= 128 && a.T >= 32; }

long long chunk_scan_scratch(const RecurrentArgs& a) {
  const long long n = (a.T + CL - 1) / CL;
  const long long chunks = (long long)a.B * n * (a.H * FACTORS * CL * 4ll + (a.kind == RK_DELTA ? a.H * 2 * 16384ll : a.KG * 16384ll));
  return chunks + (a.kind == RK_DELTA ? 0 : (long long)ssd_segments(a) * a.B * a.H * ((long long)a.Dk * a.Dv + 1) * 4);
}

void launch_chunk_scan(const RecurrentArgs& a, void* scratch, cudaStream_t s) {
  if (a.B <= 0 || a.T <= 0) return;
  if (!chunk_scan_supported(a)) throw std::runtime_error("chunk_scan: unsupported shape");
  ScanParams sp{};
  sp.a = a;
  sp.nchunks = (a.T + CL - 1) / CL;
  sp.vec_qk = a.Dk % 8 == 0 && vec8_ok(a.q, a.ldq, false) && vec8_ok(a.k, a.ldk, false);
  sp.vec_v = a.Dv % 8 == 0 && vec8_ok(a.v, a.ldv, false) && vec8_ok(a.out, a.ldo, false);
  sp.frag0 = (uint4*)scratch;
  if (a.kind == RK_DELTA) {
    sp.frag1 = sp.frag0 + (long long)a.B * a.H * sp.nchunks * 1024;
    sp.fac = (float*)(sp.frag1 + (long long)a.B * a.H * sp.nchunks * 1024);
    if (a.Dk <= 64) run_delta<64>(sp, s);
    else run_delta<128>(sp, s);
  } else {
    sp.fac = (float*)(sp.frag0 + (long long)a.B * a.KG * sp.nchunks * 1024);
    float* seg = sp.fac + (long long)a.B * a.H * sp.nchunks * FACTORS * CL;
    if (a.Dk <= 64) run_ssd<64>(sp, seg, s);
    else run_ssd<128>(sp, seg, s);
  }
}

}  // namespace tb
