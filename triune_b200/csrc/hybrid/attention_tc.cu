// Causal softmax attention with a sink on the tensor cores (bf16 operands, fp32 scores, softmax and accumulators).
//
// A CTA owns 256 consecutive queries of one head as two tiles of 128 and walks the keys in tiles of 128. Warp roles:
//   warp 0      TMA producer: the two query tiles once, then a two-stage ring of key and value tiles
//   warp 1      issues tcgen05.mma: S_w = Q_w K^T into TMEM, and O_w += P_w V with P_w read from TMEM
//   warps 4-7   softmax of query tile 0, one row per thread (TMEM lane = row)
//   warps 8-11  softmax of query tile 1
// The tiles alternate: while one tile's scores are being exponentiated the tensor core works on the other. P (bf16)
// overwrites the first half of its S columns; MMAs of one thread complete in issue order, so S_w of the next key tile
// may be issued right behind the product that reads P_w. The running maximum is lazy: the accumulator is rescaled (by
// the softmax warps, in TMEM) only when the maximum has grown by more than 2^8, otherwise the old reference stays and
// the weights are at most 256 times larger, which fp32 sums and bf16 weights carry without loss. The sink starts the
// row's maximum and sum: it has no key and no value. A second part of queries and keys (the turned part of latent
// attention, one for all heads) is a further box of the same tiles; with three boxes and wide values, values have one stage.
// TMEM: columns 0-127 S_0, 128-255 S_1, 256-383 O_0, 384-511 O_1.
#include "../common/ptx.cuh"
#include "../common/tma_desc.h"
#include "hybrid.cuh"
#include "tc_tiles.cuh"

namespace tb {
namespace {

constexpr int FA_BM = 128, FA_BN = 128, FA_THREADS = 384, FA_BOX = 128 * 128;  // bytes of a 128 x 64 bf16 box
constexpr float FA_LAZY = 8.f;

struct FaParams {
  const float* sink;
  const __nv_bfloat16* gate;
  long long ldg;
  __nv_bfloat16* out;
  long long ldo;
  int T, H, G, D, E, R;
  float scale2;  // scale * log2(e)
  float out_scale;
  Pos pos;
  int* status;
};

template <int KB, int EVB>
constexpr int fa_value_stages() {  // what 227 KB hold beside two query tiles and two key stages
  return 4 * KB + 2 * EVB <= 14 ? 2 : 1;
}

template <int DKB, int RKB, int EVB>  // 64-wide boxes of the key (first and second part) and value head sizes
__global__ void __launch_bounds__(FA_THREADS, 1) attn_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                                                                const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmQ2,
                                                                const __grid_constant__ CUtensorMap tmK2, const FaParams p) {
  constexpr int KB = DKB + RKB, VS = fa_value_stages<KB, EVB>();
  extern __shared__ uint8_t raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(raw) + 1023) & ~uintptr_t(1023));
  uint8_t *sQ = smem, *sK = sQ + 2 * KB * FA_BOX, *sV = sK + 2 * KB * FA_BOX;
  __shared__ __align__(8) uint64_t bars[13];
  uint64_t *q_full = bars, *k_full = bars + 1, *k_empty = bars + 3, *v_full = bars + 5, *v_empty = bars + 7, *s_full = bars + 9,
           *p_ready = bars + 11;
  __shared__ __align__(8) uint64_t o_full[2];
  __shared__ uint32_t tmem_slot;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int bh = blockIdx.x, h = bh % p.H, b = bh / p.H;
  const int kvh = h / (p.H / p.G);
  const int q0 = (gridDim.y - 1 - blockIdx.y) * 2 * FA_BM;  // the longest rows start first
  const long long p0l = pos_of(p.pos);
  const int p0 = (int)p0l;
  int n[2];
#pragma unroll
  for (int w = 0; w < 2; ++w) {
    const int first = q0 + w * FA_BM, last = min(p.T, first + FA_BM) - 1;
    n[w] = first < p.T ? (p0 + last) / FA_BN + 1 : 0;
  }
  const int nt = max(n[0], n[1]);

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(k_full + i, 1);
      mbar_init(k_empty + i, 1);
      mbar_init(v_full + i, 1);
      mbar_init(v_empty + i, 1);
      mbar_init(s_full + i, 1);
      mbar_init(p_ready + i, 128);
      mbar_init(o_full + i, 1);
    }
    mbar_fence_init();
  }
  if (warp == 2) {
    tmem_alloc(&tmem_slot, 512);
    tmem_relinquish();
  }
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = tmem_slot;

  if (warp == 0) {
    if (lane == 0) {
      prefetch_tmap(&tmQ);
      prefetch_tmap(&tmK);
      prefetch_tmap(&tmV);
      const int tiles = n[1] > 0 ? 2 : 1;
      mbar_expect_tx(q_full, tiles * KB * FA_BOX);
      for (int w = 0; w < tiles; ++w) {
        for (int d = 0; d < DKB; ++d) tma_load_4d(sQ + (w * KB + d) * FA_BOX, &tmQ, q_full, d * 64, q0 + w * FA_BM, h, b);
        for (int d = 0; d < RKB; ++d) tma_load_4d(sQ + (w * KB + DKB + d) * FA_BOX, &tmQ2, q_full, d * 64, q0 + w * FA_BM, h, b);
      }
      bool ok = true;
      // keys run one tile ahead of values: the scores of the next tile are issued before the use of these values ends
      for (int j = 0; j <= nt && ok; ++j) {
        if (j < nt) {
          const int s = j & 1;
          if (j >= 2) ok = mbar_wait(k_empty + s, ((j >> 1) & 1) ^ 1);
          if (!ok) break;
          mbar_expect_tx(k_full + s, KB * FA_BOX);
          for (int d = 0; d < DKB; ++d) tma_load_4d(sK + (s * KB + d) * FA_BOX, &tmK, k_full + s, d * 64, j * FA_BN, kvh, b);
          for (int d = 0; d < RKB; ++d) tma_load_4d(sK + (s * KB + DKB + d) * FA_BOX, &tmK2, k_full + s, d * 64, j * FA_BN, 0, b);
        }
        if (j > 0) {
          const int i = j - 1, s = i % VS;
          if (i >= VS) ok = mbar_wait(v_empty + s, ((i / VS) & 1) ^ 1);
          if (!ok) break;
          mbar_expect_tx(v_full + s, EVB * FA_BOX);
          for (int d = 0; d < EVB; ++d) tma_load_4d(sV + (s * EVB + d) * FA_BOX, &tmV, v_full + s, d * 64, i * FA_BN, kvh, b);
        }
      }
      if (!ok && p.status) *p.status = ST_TIMEOUT_EMPTY;
    }
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t id_s = make_idesc(128, 128, 1, 1, 0, 0), id_o = make_idesc(128, (p.E + 15) / 16 * 16, 1, 1, 0, 1);
      const int ks = (p.D + 15) / 16, rs = RKB > 0 ? (p.R + 15) / 16 : 0;
      auto scores = [&](int w, int j) {
        const uint32_t qa = smem_u32(sQ + w * KB * FA_BOX), ka = smem_u32(sK + (j & 1) * KB * FA_BOX);
        for (int k = 0; k < ks; ++k) {
          const uint32_t off = (k >> 2) * FA_BOX + (k & 3) * 32;
          umma_bf16(tmem + w * 128, make_smem_desc(qa + off, 16, 1024), make_smem_desc(ka + off, 16, 1024), id_s, k > 0);
        }
        for (int k = 0; k < rs; ++k) {
          const uint32_t off = (DKB + (k >> 2)) * FA_BOX + (k & 3) * 32;
          umma_bf16(tmem + w * 128, make_smem_desc(qa + off, 16, 1024), make_smem_desc(ka + off, 16, 1024), id_s, 1);
        }
        umma_commit(s_full + w);
      };
      auto values = [&](int w, int j) {
        const uint32_t va = smem_u32(sV + (j % VS) * EVB * FA_BOX);
#pragma unroll
        for (int k = 0; k < FA_BN / 16; ++k)
          umma_bf16_ts(tmem + 256 + w * 128, tmem + w * 128 + k * 8, make_smem_desc(va + k * 2048, FA_BOX, 1024), id_o, j > 0 || k > 0);
      };
      bool ok = mbar_wait(q_full, 0) && mbar_wait(k_full, 0);
      if (ok) {
        tc_fence_after_sync();
        for (int w = 0; w < 2; ++w)
          if (n[w] > 0) scores(w, 0);
        umma_commit(k_empty);
        for (int j = 0; j < nt && ok; ++j) {
          ok = mbar_wait(v_full + j % VS, (j / VS) & 1);
          if (ok && j + 1 < nt) ok = mbar_wait(k_full + ((j + 1) & 1), ((j + 1) >> 1) & 1);
          for (int w = 0; w < 2 && ok; ++w) {
            if (j >= n[w]) continue;
            ok = mbar_wait(p_ready + w, j & 1);
            if (!ok) break;
            tc_fence_after_sync();
            values(w, j);
            if (j + 1 == n[w]) umma_commit(o_full + w);
            else scores(w, j + 1);
          }
          if (!ok) break;
          umma_commit(v_empty + j % VS);
          if (j + 1 < nt) umma_commit(k_empty + ((j + 1) & 1));
        }
      }
      if (!ok && p.status) *p.status = ST_TIMEOUT_FULL;
    }
  } else if (warp >= 4) {
    const int w = (warp - 4) >> 2, quarter = warp & 3, row = quarter * 32 + lane;
    const int t = q0 + w * FA_BM + row;  // query of this thread
    const int qpos = p0 + t;
    const uint32_t lane_base = (uint32_t)(quarter * 32) << 16;
    const uint32_t tS = tmem + lane_base + w * 128, tO = tmem + lane_base + 256 + w * 128;
    const float c2 = p.scale2;
    float m = p.sink != nullptr ? p.sink[h] * 1.4426950408889634f : -INFINITY, l = p.sink != nullptr ? 1.f : 0.f;
    bool ok = true;
    const int first = p0 + q0 + w * FA_BM;
    for (int j = 0; j < n[w]; ++j) {
      ok = mbar_wait(s_full + w, j & 1);
      if (!ok) break;
      tc_fence_after_sync();
      const bool masked = j * FA_BN + FA_BN - 1 > first;
      const int lim = qpos - j * FA_BN;  // columns up to this one are visible
      uint32_t ra[32], rb[32];
      float mx = -INFINITY;
      auto row_max = [&](uint32_t (&r)[32], int c0) {
        if (masked) {
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (c0 + i <= lim) mx = fmaxf(mx, __uint_as_float(r[i]));
        } else {
          float x0 = __uint_as_float(r[0]), x1 = __uint_as_float(r[1]), x2 = __uint_as_float(r[2]), x3 = __uint_as_float(r[3]);
#pragma unroll
          for (int i = 4; i < 32; i += 4) {
            x0 = fmaxf(x0, __uint_as_float(r[i]));
            x1 = fmaxf(x1, __uint_as_float(r[i + 1]));
            x2 = fmaxf(x2, __uint_as_float(r[i + 2]));
            x3 = fmaxf(x3, __uint_as_float(r[i + 3]));
          }
          mx = fmaxf(mx, fmaxf(fmaxf(x0, x1), fmaxf(x2, x3)));
        }
      };
      tmem_ld_32x32b_x32(tS, ra);
      tmem_ld_wait_regs(ra);
      tmem_ld_32x32b_x32(tS + 32, rb);
      row_max(ra, 0);
      tmem_ld_wait_regs(rb);
      tmem_ld_32x32b_x32(tS + 64, ra);
      row_max(rb, 32);
      tmem_ld_wait_regs(ra);
      tmem_ld_32x32b_x32(tS + 96, rb);
      row_max(ra, 64);
      tmem_ld_wait_regs(rb);
      tmem_ld_32x32b_x32(tS, ra);  // the first columns again, for the exponentials
      row_max(rb, 96);
      const float mn = fmaxf(m, mx * c2);
      const bool grow = j == 0 || mn - m > FA_LAZY;
      float f = 1.f;
      if (grow) {
        f = ex2(m - mn);  // m = -inf at the first tile of a row without a sink gives 0
        m = mn;
        l *= f;
      }
      tmem_ld_wait_regs(ra);
      if (j > 0 && __any_sync(0xffffffffu, grow)) {
        for (int c = 0; c < p.E; c += 16) {
          uint32_t o[16];
          tmem_ld_32x32b_x16(tO + c, o);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * f);
          tmem_st_32x32b_x16(tO + c, o);
        }
        tmem_st_wait();
      }
      const uint64_t cc = pack_f2(c2, c2), mm = pack_f2(-m, -m);
      uint64_t sum2 = pack_f2(0.f, 0.f);
      auto weights = [&](uint32_t (&r)[32], int c0) {
        uint32_t q[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          float a, e;
          unpack_f2(fma2(pack_f2(__uint_as_float(r[2 * i]), __uint_as_float(r[2 * i + 1])), cc, mm), a, e);
          a = ex2(a);
          e = ex2(e);
          if (masked) {
            a = c0 + 2 * i <= lim ? a : 0.f;
            e = c0 + 2 * i + 1 <= lim ? e : 0.f;
          }
          sum2 = add2(sum2, pack_f2(a, e));
          q[i] = pack_bf16x2(a, e);
        }
        tmem_st_32x32b_x16(tS + c0 / 2, q);  // lands in columns whose scores this thread has already read
      };
      tmem_ld_32x32b_x32(tS + 32, rb);
      weights(ra, 0);
      tmem_ld_wait_regs(rb);
      tmem_ld_32x32b_x32(tS + 64, ra);
      weights(rb, 32);
      tmem_ld_wait_regs(ra);
      tmem_ld_32x32b_x32(tS + 96, rb);
      weights(ra, 64);
      tmem_ld_wait_regs(rb);
      weights(rb, 96);
      float s0, s1;
      unpack_f2(sum2, s0, s1);
      l += s0 + s1;
      tmem_st_wait();
      tc_fence_before_sync();
      mbar_arrive(p_ready + w);
    }
    if (ok && n[w] > 0) {
      ok = mbar_wait(o_full + w, 0);
      if (ok) {
        tc_fence_after_sync();
        float r = p.out_scale / l;
        if (p.gate != nullptr && t < p.T) r *= sigmoid_f(__bfloat162float(p.gate[((long long)b * p.T + t) * p.ldg + h]));
        __nv_bfloat16* o = p.out + ((long long)b * p.T + t) * p.ldo + (long long)h * p.E;
        const bool vec = (p.E & 7) == 0 && (p.ldo & 7) == 0 && (reinterpret_cast<uintptr_t>(p.out) & 15) == 0;
        for (int c = 0; c < p.E; c += 16) {
          uint32_t v[16];
          tmem_ld_32x32b_x16(tO + c, v);
          tmem_ld_wait();
          if (t < p.T) {
            if (vec) {
#pragma unroll
              for (int g = 0; g < 2; ++g)
                if (c + 8 * g < p.E) {
                  uint4 u;
                  uint32_t* up = &u.x;
#pragma unroll
                  for (int i = 0; i < 4; ++i)
                    up[i] = pack_bf16x2(__uint_as_float(v[8 * g + 2 * i]) * r, __uint_as_float(v[8 * g + 2 * i + 1]) * r);
                  *reinterpret_cast<uint4*>(o + c + 8 * g) = u;
                }
            } else {
#pragma unroll
              for (int i = 0; i < 16; ++i)
                if (c + i < p.E) o[c + i] = __float2bfloat16(__uint_as_float(v[i]) * r);
            }
          }
        }
      }
    }
    if (!ok && p.status) *p.status = ST_TIMEOUT_TMEM;
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  if (warp == 2) tmem_dealloc(tmem, 512);
}

CUtensorMap operand_map(const AttnOperand& o, int d, int rows, int heads, int batch) {
  return make_tmap_4d_bf16(o.p, {(uint64_t)d, (uint64_t)rows, (uint64_t)heads, (uint64_t)batch},
                           {(uint64_t)o.sr * 2, (uint64_t)o.sh * 2, (uint64_t)o.sb * 2}, 128);
}

template <int DKB, int RKB, int EVB>
void run(const AttnArgs& a, int* status, cudaStream_t s) {
  const CUtensorMap tq = operand_map(a.q, a.D, a.T, a.H, a.B), tk = operand_map(a.k, a.D, a.rows, a.G, a.B), tv = operand_map(a.v, a.E, a.rows, a.G, a.B);
  const CUtensorMap tq2 = RKB > 0 ? operand_map(a.q2, a.R, a.T, a.H, a.B) : tq, tk2 = RKB > 0 ? operand_map(a.k2, a.R, a.rows, 1, a.B) : tk;
  FaParams p{a.sink, (const __nv_bfloat16*)a.gate, a.ldg, (__nv_bfloat16*)a.out, a.ldo, a.T, a.H, a.G, a.D, a.E, a.R,
             a.scale * 1.4426950408889634f, a.out_scale, a.pos, status};
  constexpr int KB = DKB + RKB;
  constexpr int smem = (4 * KB + fa_value_stages<KB, EVB>() * EVB) * FA_BOX + 1024;
  static_assert(smem <= 227 * 1024, "shared memory of a block");
  auto kern = attn_tc_kernel<DKB, RKB, EVB>;
  cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  kern<<<dim3(a.B * a.H, (a.T + 2 * FA_BM - 1) / (2 * FA_BM)), FA_THREADS, smem, s>>>(tq, tk, tv, tq2, tk2, p);
}

template <int DKB, int RKB>
void run_values(const AttnArgs& a, int* status, cudaStream_t s) {
  if (a.E <= 64) run<DKB, RKB, 1>(a, status, s);
  else run<DKB, RKB, 2>(a, status, s);
}

}  // namespace

bool attn_tc_supported(const AttnArgs& a) {
  auto fits = [](const AttnOperand& o) {
    return (reinterpret_cast<uintptr_t>(o.p) & 15) == 0 && o.sr % 8 == 0 && o.sh % 8 == 0 && o.sb % 8 == 0;
  };
  return !a.f32 && a.D <= 128 && a.E <= 128 && a.R <= 64 && a.scale > 0.f && a.T > 0 && fits(a.q) && fits(a.k) && fits(a.v) &&
         (a.R == 0 || (fits(a.q2) && fits(a.k2)));
}

void launch_attn_tc(const AttnArgs& a, int* status, cudaStream_t s) {
  if (a.B <= 0 || a.T <= 0) return;
  if (!attn_tc_supported(a)) throw std::runtime_error("attn_tc: unsupported shape");
  if (a.R > 0) {
    if (a.D <= 64) run_values<1, 1>(a, status, s);
    else run_values<2, 1>(a, status, s);
  } else {
    if (a.D <= 64) run_values<1, 0>(a, status, s);
    else run_values<2, 0>(a, status, s);
  }
  check_launch("attn_tc");
}

}  // namespace tb
