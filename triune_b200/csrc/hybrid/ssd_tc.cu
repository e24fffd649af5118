// Mamba-2 prompts on the tcgen05 tensor cores: the segment scheme of chunk_scan.cu with chunks of 128 tokens, for aligned
// bf16 inputs and key sizes of 65 to 128.
//
// Per chunk, with C the queries, K the keys and x the values (exact bf16), b the running log decay, w_j = dt_j e^{b_end-b_j}:
//   G  = C K^T                                     -> M_ij = G_ij dt_j e^{b_i-b_j} (j <= i), two bf16 numbers each, in TMEM
//   Y  = e^{b_i} (C S) + M x + D x                  S as two bf16 numbers in shared memory, M as the A operand from TMEM
//   S <- e^{b_end} S + K^T (w x)                    w x as two bf16 numbers; the sum in fp32 registers
// A block owns 64 value columns of a head and a segment of the sequence. 256 of its threads are two halves of 128 rows: a
// thread has row r = its TMEM lane (a token for G, M and Y; a key dimension for the state) and half of the columns, so every
// pass between the products stays in its registers. Shared-memory tiles are 128 rows of 128 bytes in the 128B-swizzled
// layout; a ninth warp issues the MMAs (issuing blocks while the tensor pipe is busy): K and C are K-major operands for G, K is read again as the transposed A operand of the update.
// TMEM columns: 0 G (128), 128 and 448 C S of alternating chunks (64 each), 192 M x (64), 256 K^T (w x) (64), 320 low halves
// of M (64), 384 high halves (64).
#include "../common/ptx.cuh"
#include "hybrid.cuh"
#include "tc_tiles.cuh"

namespace tb {
namespace {

constexpr int TL = 128, TT = 256, TCOLS = 64, TBOX = 128 * 128;  // tokens, threads, value columns, bytes of a tile
constexpr int TF = 5;  // factor rows: 0 b, 1 dt, 2 w, 3 dt e^{b_ref - b} with the last token of each 32 as reference, 4 e^{b_end}

struct SsdTcParams {
  RecurrentArgs a;
  int nchunks, seg_chunks, nseg;
  float* fac;        // [B, H, nchunks][TF][128]
  float* seg_state;  // as in chunk_scan.cu
  int* status;
};

__global__ void __launch_bounds__(128) ssd_tc_factors_kernel(const SsdTcParams sp) {
  __shared__ float sb[4][TL], sg[4][TL];
  const RecurrentArgs& p = sp.a;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long id = (long long)blockIdx.x * 4 + warp;
  if (id >= (long long)p.B * p.H * sp.nchunks) return;
  const int c = (int)(id % sp.nchunks), bh = (int)(id / sp.nchunks), h = bh % p.H, b = bh / p.H;
  const __nv_bfloat16* A = (const __nv_bfloat16*)p.a + (long long)b * p.rows * p.lda + h;
  const float ea = expf(p.A_log[h]), bias = p.dt_bias[h];
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int t0 = c * TL + half * CL, t = t0 + 2 * lane;
    chunk_scalars(p, load_or0(A, p.lda, t, p.T), load_or0(A, p.lda, t + 1, p.T), 0.f, 0.f, ea, bias, t0, sb[warp] + half * CL, sg[warp] + half * CL);
  }
  __syncwarp();
  const float first = sb[warp][CL - 1];
  for (int i = CL + lane; i < TL; i += 32) sb[warp][i] += first;
  __syncwarp();
  float* f = sp.fac + id * TF * TL;
  const float bl = sb[warp][TL - 1];
  for (int i = lane; i < TL; i += 32) {
    f[i] = sb[warp][i];
    f[TL + i] = sg[warp][i];
    f[2 * TL + i] = sg[warp][i] * exp_neg(bl - sb[warp][i]);
    f[3 * TL + i] = sg[warp][i] * exp_neg(sb[warp][i | 31] - sb[warp][i]);
    f[4 * TL + i] = exp_neg(bl);
  }
}

// Rows t0 .. t0 + 127 and `boxes` tiles of 64 columns into swizzled tiles; rows past T and columns past D become zero.
__device__ __forceinline__ void stage_tile(uint8_t* dst, const __nv_bfloat16* src, long long ld, int t0, int T, int D, int boxes, int tid) {
  const int ch = tid & 7, r0 = tid >> 3;
  for (int x = 0; x < boxes; ++x) {
    const int c = x * 64 + ch * 8;
#pragma unroll
    for (int i = 0; i < TL / (TT / 8); ++i) {
      const int r = r0 + i * (TT / 8);
      const bool ok = t0 + r < T && c < D;
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst + x * TBOX + sw(r, ch))),
                   "l"(ok ? src + (long long)(t0 + r) * ld + c : src), "r"(ok ? 16 : 0)
                   : "memory");
    }
  }
}

template <bool OUT>
struct SsdTcSmem {  // after alignment to 1024 bytes
  static constexpr int NK = OUT ? 2 : 3, NX = 3;  // chunks of keys, and of values and factors, in shared memory
  static constexpr int K = 0, X = K + NK * 2 * TBOX, WH = X + NX * TBOX, WL = WH + TBOX, F = WL + TBOX;
  static constexpr int C = (F + NX * TF * TL * 4 + 1023) / 1024 * 1024, SH = C + (OUT ? 2 * TBOX : 0), SL = SH + (OUT ? TBOX : 0), END = SL + (OUT ? TBOX : 0);
  static_assert(F % 1024 == 0 && C % 1024 == 0, "tiles start on 1024 bytes");
};

template <bool OUT>
__global__ void __launch_bounds__(TT + 32, 1) ssd_tc_kernel(const SsdTcParams sp) {
  using L = SsdTcSmem<OUT>;
  extern __shared__ uint8_t raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(raw) + 1023) & ~uintptr_t(1023));
  __shared__ __align__(8) uint64_t bars[4];   // products done: G, C S, M x, update
  __shared__ __align__(8) uint64_t ready[3];  // operands in place: tiles and state, weighted values, M
  __shared__ uint32_t tmem_slot;
  __shared__ int dead;
  const RecurrentArgs& p = sp.a;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, half = warp >> 2, row = (warp & 3) * 32 + lane;
  const int slices = (p.Dv + TCOLS - 1) / TCOLS;
  const int slice = blockIdx.x % slices, bh = blockIdx.x / slices, h = bh % p.H, b = bh / p.H, seg = blockIdx.y;
  const int kh = h / (p.H / p.KG), c0 = slice * TCOLS, ncol = min(TCOLS, p.Dv - c0), col0 = half * 32;
  const __nv_bfloat16 *Q = (const __nv_bfloat16*)p.q + (long long)b * p.rows * p.ldq + kh * p.Dk,
                      *K = (const __nv_bfloat16*)p.k + (long long)b * p.rows * p.ldk + kh * p.Dk,
                      *V = (const __nv_bfloat16*)p.v + (long long)b * p.rows * p.ldv + h * p.Dv + c0;
  __nv_bfloat16* O = (__nv_bfloat16*)p.out + (long long)b * p.rows * p.ldo + h * p.Dv + c0;
  const float Dh = p.D[h];
  const float* fac = sp.fac + (long long)bh * sp.nchunks * TF * TL;
  const int first = seg * sp.seg_chunks, last = min(first + sp.seg_chunks, sp.nchunks);

  if (tid == 0) {
    for (int i = 0; i < 4; ++i) mbar_init(bars + i, 1);
    for (int i = 0; i < 3; ++i) mbar_init(ready + i, TT);
    mbar_fence_init();
    dead = 0;
  }
  __syncwarp();
  if (warp == 8) {
    tmem_alloc(&tmem_slot, 512);
    tmem_relinquish();
  }
  // state: key dimension `row`, value columns col0 .. col0 + 31
  float S[32];
  const long long plane = (long long)p.Dk * p.Dv;
  float* mine = sp.nseg > 1 ? sp.seg_state + ((long long)seg * p.B * p.H + bh) * plane : p.state + (long long)bh * plane;
#pragma unroll
  for (int g = 0; g < 4; ++g) {
    float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (OUT && warp < 8 && row < p.Dk && col0 + 8 * g < ncol) ld8v(mine + (long long)row * p.Dv + c0 + col0 + 8 * g, f);
#pragma unroll
    for (int i = 0; i < 8; ++i) S[8 * g + i] = f[i];
  }
  // 32 fp32 values of this thread's row as two bf16 tiles
  auto put = [&](int hi_at, int lo_at, const float (&v)[32]) {
#pragma unroll
    for (int g = 0; g < 4; ++g) {
      uint4 hi, lo;
      split2(v[8 * g], v[8 * g + 1], hi.x, lo.x);
      split2(v[8 * g + 2], v[8 * g + 3], hi.y, lo.y);
      split2(v[8 * g + 4], v[8 * g + 5], hi.z, lo.z);
      split2(v[8 * g + 6], v[8 * g + 7], hi.w, lo.w);
      const uint32_t at = sw(row, half * 4 + g);
      *reinterpret_cast<uint4*>(smem + hi_at + at) = hi;
      *reinterpret_cast<uint4*>(smem + lo_at + at) = lo;
    }
  };
  auto stage_kx = [&](int c) {
    const int u = (c - first) % L::NX;
    stage_tile(smem + L::K + (c - first) % L::NK * 2 * TBOX, K, p.ldk, c * TL, p.T, p.Dk, 2, tid);
    stage_tile(smem + L::X + u * TBOX, V, p.ldv, c * TL, p.T, ncol, 1, tid);
    if (tid < TF * TL / 4)
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem + L::F + u * TF * TL * 4 + tid * 16)),
                   "l"(fac + (long long)c * TF * TL + tid * 4)
                   : "memory");
  };
  auto stage_c = [&](int c) {
    if constexpr (OUT) stage_tile(smem + L::C, Q, p.ldq, c * TL, p.T, p.Dk, 2, tid);
  };
  if (first < last && warp < 8) {
    stage_c(first);
    stage_kx(first);
    cp_commit();
    if constexpr (!OUT) {
      if (first + 1 < last) stage_kx(first + 1);
      cp_commit();
    }
  }
  if (OUT && warp < 8) put(L::SH, L::SL, S);
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = tmem_slot, lanes = tmem + ((uint32_t)((warp & 3) * 32) << 16);
  const uint32_t base = smem_u32(smem);
  auto wait_on = [&](uint64_t* bar, uint32_t parity) {
    if (*(volatile int*)&dead == 0 && !mbar_wait(bar, parity)) {
      dead = 1;
      if (sp.status) *sp.status = ST_TIMEOUT_TMEM;
    }
  };
  auto wait_bar = [&](int i, uint32_t parity) {
    wait_on(bars + i, parity);
    __syncwarp();
    tc_fence_after_sync();
  };
  auto rows_sync = [&]() { asm volatile("bar.sync 1, 256;" ::: "memory"); };
  if (warp == 8) {
    if (lane == 0) {
      constexpr uint32_t id_g = make_idesc(128, 128, 1, 1, 0, 0), id_s = make_idesc(128, 64, 1, 1, 0, 1), id_u = make_idesc(128, 64, 1, 1, 1, 1);
      for (int c = first; c < last; ++c) {
        const uint32_t u = (c - first) & 1, ka = base + L::K + (c - first) % L::NK * 2 * TBOX, xa = base + L::X + (c - first) % L::NX * TBOX, ca = base + L::C;
        wait_on(ready + 0, u);
        tc_fence_after_sync();
        if constexpr (OUT) {
#pragma unroll
          for (int k = 0; k < 8; ++k) {
            const uint32_t off = (k >> 2) * TBOX + (k & 3) * 32;
            umma_bf16(tmem, make_smem_desc(ca + off, 16, 1024), make_smem_desc(ka + off, 16, 1024), id_g, k > 0);
          }
          umma_commit(bars + 0);
          const uint32_t cs = tmem + (u == 0 ? 128 : 448);
#pragma unroll
          for (int k = 0; k < 8; ++k) {
            const uint64_t a = make_smem_desc(ca + (k >> 2) * TBOX + (k & 3) * 32, 16, 1024);
            umma_bf16(cs, a, make_smem_desc(base + L::SH + k * 2048, TBOX, 1024), id_s, k > 0);
            umma_bf16(cs, a, make_smem_desc(base + L::SL + k * 2048, TBOX, 1024), id_s, 1);
          }
          umma_commit(bars + 1);
        }
        wait_on(ready + 1, u);
        tc_fence_after_sync();
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          const uint64_t a = make_smem_desc(ka + k * 2048, TBOX, 1024);
          umma_bf16(tmem + 256, a, make_smem_desc(base + L::WH + k * 2048, TBOX, 1024), id_u, k > 0);
          umma_bf16(tmem + 256, a, make_smem_desc(base + L::WL + k * 2048, TBOX, 1024), id_u, 1);
        }
        umma_commit(bars + 3);
        if constexpr (OUT) {
          wait_on(ready + 2, u);
          tc_fence_after_sync();
#pragma unroll
          for (int k = 0; k < 8; ++k) {
            const uint64_t x = make_smem_desc(xa + k * 2048, TBOX, 1024);
            umma_bf16_ts(tmem + 192, tmem + 384 + k * 8, x, id_s, k > 0);
            umma_bf16_ts(tmem + 192, tmem + 320 + k * 8, x, id_s, 1);
          }
          umma_commit(bars + 2);
        }
      }
    }
    __syncwarp();
  } else {
  float decay = 1.f;

  // outputs of chunk c: e^{b_i} (C S) + M x + D x
  auto outputs = [&](int c) {
    const int u = (c - first) & 1, slot = (c - first) % L::NX, t = c * TL + row;
    const uint8_t* X = smem + L::X + slot * TBOX;
    const float e = exp_neg(reinterpret_cast<const float*>(smem + L::F)[slot * TF * TL + row]);
    wait_bar(2, u);
    uint32_t cs[32], mx[32];
    tmem_ld_32x32b_x32(lanes + (u == 0 ? 128 : 448) + col0, cs);
    tmem_ld_32x32b_x32(lanes + 192 + col0, mx);
    tmem_ld_wait_regs(cs);
    tmem_ld_wait_regs(mx);
    if (t < p.T) {
      __nv_bfloat16* dst = O + (long long)t * p.ldo + col0;
#pragma unroll
      for (int g = 0; g < 4; ++g) {
        const uint4 q = *reinterpret_cast<const uint4*>(X + sw(row, half * 4 + g));
        const uint32_t xs[4] = {q.x, q.y, q.z, q.w};
        uint4 y;
        uint32_t* ys = &y.x;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int k = 8 * g + 2 * i;
          ys[i] = pack_bf16x2(e * __uint_as_float(cs[k]) + __uint_as_float(mx[k]) + Dh * lo_f(xs[i]),
                              e * __uint_as_float(cs[k + 1]) + __uint_as_float(mx[k + 1]) + Dh * hi_f(xs[i]));
        }
        if (col0 + 8 * g < ncol) *reinterpret_cast<uint4*>(dst + 8 * g) = y;  // Dv is a multiple of eight
      }
    }
  };

  // Order within a chunk: scores and state products are issued first; the previous chunk's outputs are written under them;
  // the update is issued as soon as the weighted values are there and runs under the decay of the scores; the state is
  // updated and published under the last product.
  for (int c = first; c < last; ++c) {
    const int slot = (c - first) % L::NX;
    const uint32_t par = (c - first) & 1;
    const float* F = reinterpret_cast<const float*>(smem + L::F) + slot * TF * TL;
    const uint8_t* X = smem + L::X + slot * TBOX;
    if constexpr (OUT) cp_wait0();
    else asm volatile("cp.async.wait_group 1;" ::: "memory");
    fence_proxy_async_smem();
    tc_fence_before_sync();
    rows_sync();  // this chunk's tiles and the state before it
    mbar_arrive(ready + 0);
    const bool more = c + 1 < last;
    if (OUT && more) stage_kx(c + 1);  // its keys' slot is free: every update so far has been waited for
    if (OUT && c > first) outputs(c - 1);
    {
      const float w = F[2 * TL + row];
      float v[32];
#pragma unroll
      for (int g = 0; g < 4; ++g) {
        const uint4 q = *reinterpret_cast<const uint4*>(X + sw(row, half * 4 + g));
        v[8 * g] = lo_f(q.x) * w; v[8 * g + 1] = hi_f(q.x) * w; v[8 * g + 2] = lo_f(q.y) * w; v[8 * g + 3] = hi_f(q.y) * w;
        v[8 * g + 4] = lo_f(q.z) * w; v[8 * g + 5] = hi_f(q.z) * w; v[8 * g + 6] = lo_f(q.w) * w; v[8 * g + 7] = hi_f(q.w) * w;
      }
      put(L::WH, L::WL, v);
    }
    fence_proxy_async_smem();
    tc_fence_before_sync();
    rows_sync();  // every thread has read what it needs of chunk c - 1
    mbar_arrive(ready + 1);
    if constexpr (!OUT) {  // one commit per chunk, empty at the end
      if (c + 2 < last) stage_kx(c + 2);
      cp_commit();
    }
    if constexpr (OUT) {
      // decayed scores: blocks of 32 tokens before this warp's rows factor through the block's last token, the block of
      // the rows themselves goes pair by pair, later blocks are zero
      const float bi = F[row];
      wait_bar(0, par);
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const int jb = half * 2 + k, q = warp & 3;
        uint32_t hi[16], lo[16];
        if (jb <= q) {
          uint32_t g[32];
          tmem_ld_32x32b_x32(lanes + jb * 32, g);
          tmem_ld_wait_regs(g);
          if (jb < q) {
            const float e = exp_neg(bi - F[jb * 32 + 31]);
            const float4* cf = reinterpret_cast<const float4*>(F + 3 * TL + jb * 32);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
              const float4 f = cf[i];
              split2(__uint_as_float(g[4 * i]) * (f.x * e), __uint_as_float(g[4 * i + 1]) * (f.y * e), hi[2 * i], lo[2 * i]);
              split2(__uint_as_float(g[4 * i + 2]) * (f.z * e), __uint_as_float(g[4 * i + 3]) * (f.w * e), hi[2 * i + 1], lo[2 * i + 1]);
            }
          } else {
            const float4 *bj = reinterpret_cast<const float4*>(F + jb * 32), *dt = reinterpret_cast<const float4*>(F + TL + jb * 32);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
              const float4 f = bj[i], d = dt[i];
              const float m0 = 4 * i <= lane ? __uint_as_float(g[4 * i]) * d.x * exp_neg(bi - f.x) : 0.f;
              const float m1 = 4 * i + 1 <= lane ? __uint_as_float(g[4 * i + 1]) * d.y * exp_neg(bi - f.y) : 0.f;
              const float m2 = 4 * i + 2 <= lane ? __uint_as_float(g[4 * i + 2]) * d.z * exp_neg(bi - f.z) : 0.f;
              const float m3 = 4 * i + 3 <= lane ? __uint_as_float(g[4 * i + 3]) * d.w * exp_neg(bi - f.w) : 0.f;
              split2(m0, m1, hi[2 * i], lo[2 * i]);
              split2(m2, m3, hi[2 * i + 1], lo[2 * i + 1]);
            }
          }
        } else {
#pragma unroll
          for (int i = 0; i < 16; ++i) hi[i] = lo[i] = 0u;
        }
        tmem_st_32x32b_x16(lanes + 384 + jb * 16, hi);
        tmem_st_32x32b_x16(lanes + 320 + jb * 16, lo);
        if (k == 0) {
          wait_bar(1, par);  // the queries and the published state have been read
          if (more) {
            stage_c(c + 1);
            cp_commit();
          }
        }
      }
      tmem_st_wait();
      tc_fence_before_sync();
      mbar_arrive(ready + 2);
    }
    const float dl = F[4 * TL];
    decay *= dl;
    wait_bar(3, par);
    uint32_t kv[32];
    tmem_ld_32x32b_x32(lanes + 256 + col0, kv);
    tmem_ld_wait_regs(kv);
#pragma unroll
    for (int i = 0; i < 32; ++i) S[i] = dl * S[i] + __uint_as_float(kv[i]);
    if constexpr (OUT) put(L::SH, L::SL, S);
  }
  if (OUT && first < last) outputs(last - 1);
  if (!OUT || seg == sp.nseg - 1) {
    float* dst = OUT ? p.state + (long long)bh * plane : mine;
#pragma unroll
    for (int g = 0; g < 4; ++g) {
      float f[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] = S[8 * g + i];
      if (row < p.Dk && col0 + 8 * g < ncol) st8v(dst + (long long)row * p.Dv + c0 + col0 + 8 * g, f);
    }
    if (!OUT && slice == 0 && tid == 0) sp.seg_state[(long long)sp.nseg * p.B * p.H * plane + (long long)seg * p.B * p.H + bh] = decay;
  }
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  if (warp == 8) tmem_dealloc(tmem, 512);
}

}  // namespace

bool ssd_tc_supported(const RecurrentArgs& a) {
  return !a.f32 && a.kind == RK_MAMBA2 && a.T >= 64 && a.Dk > 64 && a.Dk <= 128 && a.Dk % 8 == 0 && a.Dv % 8 == 0 && vec8_ok(a.q, a.ldq, false) &&
         vec8_ok(a.k, a.ldk, false) && vec8_ok(a.v, a.ldv, false) && vec8_ok(a.out, a.ldo, false) && vec8_ok(a.state, 4, true);
}

// About one block per SM; at least two chunks per segment.
int ssd_tc_segments(const RecurrentArgs& a) {
  const int blocks = a.B * a.H * ((a.Dv + TCOLS - 1) / TCOLS), n = (a.T + TL - 1) / TL;
  int s = 148 / blocks;
  s = s > n / 2 ? n / 2 : s;
  s = s > 64 ? 64 : s;
  return s < 2 ? 1 : s;
}

long long ssd_tc_scratch(const RecurrentArgs& a) {
  const long long n = (a.T + TL - 1) / TL;
  return a.B * a.H * n * TF * TL * 4 + (long long)ssd_tc_segments(a) * a.B * a.H * ((long long)a.Dk * a.Dv + 1) * 4;
}

void launch_ssd_tc(const RecurrentArgs& a, void* scratch, int* status, cudaStream_t s) {
  if (a.B <= 0 || a.T <= 0) return;
  if (!ssd_tc_supported(a)) throw std::runtime_error("ssd_tc: unsupported shape");
  SsdTcParams sp{};
  sp.a = a;
  sp.nchunks = (a.T + TL - 1) / TL;
  const int want = ssd_tc_segments(a);
  sp.seg_chunks = (sp.nchunks + want - 1) / want;
  sp.nseg = (sp.nchunks + sp.seg_chunks - 1) / sp.seg_chunks;
  sp.fac = (float*)scratch;
  sp.seg_state = sp.fac + (long long)a.B * a.H * sp.nchunks * TF * TL;
  sp.status = status;
  const long long n = (long long)a.B * a.H * sp.nchunks;
  ssd_tc_factors_kernel<<<(unsigned)((n + 3) / 4), 128, 0, s>>>(sp);
  check_launch("ssd_tc_factors");
  const int blocks = a.B * a.H * ((a.Dv + TCOLS - 1) / TCOLS);
  if (sp.nseg > 1) {
    constexpr int smem = SsdTcSmem<false>::END + 1024;
    cudaFuncSetAttribute(ssd_tc_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    ssd_tc_kernel<false><<<dim3(blocks, sp.nseg - 1), TT + 32, smem, s>>>(sp);
    check_launch("ssd_tc_states");
    launch_ssd_scan(a, sp.seg_state, sp.nseg, s);
  }
  constexpr int smem = SsdTcSmem<true>::END + 1024;
  static_assert(smem <= 227 * 1024, "shared memory of a block");
  cudaFuncSetAttribute(ssd_tc_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  ssd_tc_kernel<true><<<dim3(blocks, sp.nseg), TT + 32, smem, s>>>(sp);
  check_launch("ssd_tc_out");
}

}  // namespace tb
