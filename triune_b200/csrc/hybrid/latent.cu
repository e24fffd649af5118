// Multi-head latent attention beside its prompt attention (attention.cu, attention_tc.cu): preparation of a prompt's
// queries and cached rows, and the one-token step in the latent space.
//
// A cached row is [normed latent (rank) | turned key part (R)]. With k_h = W_uk,h c and v_h = W_uv,h c:
//   q_h . k_h = (W_uk,h^T q_h) . c        sum_j p_j v_hj = W_uv,h (sum_j p_j c_j)
// so a step never forms keys or values: every head attends to the cached rows themselves with a query of rank + R
// entries, and one row of the cache serves all heads.
#include "../common/ptx.cuh"
#include "hybrid.cuh"
#include "step_common.cuh"

namespace tb {
namespace {

// ------------------------------------------------------------------------------------------------ prompts
constexpr int LP_THREADS = 128;

// block: one token of one sequence
template <class T>
__global__ void __launch_bounds__(LP_THREADS) latent_prep_kernel(const LatentPrepArgs p, bool vec) {
  __shared__ float red[33];
  const int t = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, half = p.R / 2;
  T* pr = (T*)p.proj + ((long long)b * p.T + t) * p.ld;
  const float *cs = p.rot + (long long)t * p.R, *sn = cs + half;
  if (vec) {  // halves in pieces of eight
    const int n = half / 8;
    for (int i = tid; i < p.H * n; i += LP_THREADS) {
      const int h = i / n, d = (i % n) * 8;
      T* q = pr + p.col_q + h * (p.Dp + p.Rp) + p.Dp;
      float u[8], v[8], c[8], s[8], a[8], o[8];
      ld8v(q + d, u);
      ld8v(q + half + d, v);
      ld8v(cs + d, c);
      ld8v(sn + d, s);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        a[e] = u[e] * c[e] - v[e] * s[e];
        o[e] = v[e] * c[e] + u[e] * s[e];
      }
      st8v(q + d, a);
      st8v(q + half + d, o);
    }
  } else {
    for (int i = tid; i < p.H * half; i += LP_THREADS) {
      const int h = i / half, d = i % half;
      T* q = pr + p.col_q + h * (p.Dp + p.Rp) + p.Dp;
      const float u = ldf(q + d), v = ldf(q + half + d), c = cs[d], s = sn[d];
      stf(q + d, u * c - v * s);
      stf(q + half + d, v * c + u * s);
    }
  }
  const long long pos = pos_of(p.pos) + t;
  if (p.col_c < 0 || pos < 0 || pos >= p.cap) return;  // the host reserves before every call
  const T* z = pr + p.col_c;
  T* dst = (T*)p.cache + ((long long)b * p.cap + pos) * (p.rank_p + p.Rp);
  float ss = 0.f;
  if (vec && p.rank % 8 == 0 && p.rank <= LP_THREADS * 8) {
    float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    const bool on = tid * 8 < p.rank;
    if (on) ld8v(z + tid * 8, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) ss += f[e] * f[e];
    const float r = 1.f / sqrtf(block_sum(ss, red) / p.rank + p.eps);
    if (on) {
      float w[8];
      ld8v(p.norm_w + tid * 8, w);
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] *= r * w[e];
      st8v(dst + tid * 8, f);
    }
  } else {
    for (int i = tid; i < p.rank; i += LP_THREADS) ss += ldf(z + i) * ldf(z + i);
    const float r = 1.f / sqrtf(block_sum(ss, red) / p.rank + p.eps);
    for (int i = tid; i < p.rank_p; i += LP_THREADS) stf(dst + i, i < p.rank ? ldf(z + i) * r * p.norm_w[i] : 0.f);
  }
  for (int i = tid; i < p.Rp; i += LP_THREADS) {
    float v = 0.f;
    if (i < p.R) {
      const int d = i < half ? i : i - half;
      const float x = ldf(z + p.rank_p + i), o = ldf(z + p.rank_p + (i < half ? i + half : i - half));
      v = i < half ? x * cs[d] - o * sn[d] : x * cs[d] + o * sn[d];
    }
    stf(dst + p.rank_p + i, v);
  }
}

// ------------------------------------------------------------------------------------------------ step: queries
constexpr int LQ_THREADS = 256, LQ_COLS = 64;

// Entry i of a turned part x at the step's position.
__device__ __forceinline__ float turn_part(const LatentStepArgs& p, const float* x, int i, long long pos) {
  const int half = p.R / 2, d = i < half ? i : i - half;
  float s, c;
  rotation(pos, p.freqs[d], &s, &c);
  s *= p.amplitude;
  c *= p.amplitude;
  return i < half ? x[i] * c - x[i + half] * s : x[i] * c + x[i - half] * s;
}

// blocks (slice of 64 latent columns, head, sequence): W_uk^T q, a thread per 16 bytes of columns and group of key rows;
// one more slice of head 0 appends the position's row to the cache
template <class T>
__global__ void __launch_bounds__(LQ_THREADS) latent_query_kernel(const LatentStepArgs p, int slices) {
  constexpr int VEC = 16 / sizeof(T), TX = LQ_COLS / VEC, GR = LQ_THREADS / TX;
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[33];
  const int tid = threadIdx.x, unit = blockIdx.x, b = unit / (slices * p.H + 1), w = unit % (slices * p.H + 1);
  const int pitch = p.rank_p + p.Rp, h = w / slices, c0 = (w % slices) * LQ_COLS;
  const int tx = tid % TX, gr = tid / TX, col = c0 + tx * VEC;
  const bool work = h < p.H && col < p.rank_p;  // rank_p is a multiple of eight
  const T* up = (const T*)p.up + (long long)h * (p.Dp + p.Ep) * p.rank_p + col;
  constexpr int PRE = 4;  // weights fetched before the wait: they do not depend on the previous kernel
  uint4 pre[PRE];
#pragma unroll
  for (int i = 0; i < PRE; ++i)
    if (work && gr + i * GR < p.D) pre[i] = *reinterpret_cast<const uint4*>(up + (long long)(gr + i * GR) * p.rank_p);
  launch_dependents();
  wait_for_previous();
  const long long pos = pos_of(p.pos);
  const float* pr = p.proj + (long long)b * p.ld;
  if (w == slices * p.H) {
    if (p.col_c < 0 || pos < 0 || pos >= p.cap) return;
    const float* z = pr + p.col_c;
    T* dst = (T*)p.cache + ((long long)b * p.cap + pos) * pitch;
    float ss = 0.f;
    for (int i = tid; i < p.rank; i += LQ_THREADS) ss += z[i] * z[i];
    const float r = 1.f / sqrtf(block_sum(ss, red) / p.rank + p.eps);
    for (int i = tid; i < p.rank_p; i += LQ_THREADS) stf(dst + i, i < p.rank ? z[i] * r * p.norm_w[i] : 0.f);
    for (int i = tid; i < p.Rp; i += LQ_THREADS) stf(dst + p.rank_p + i, i < p.R ? turn_part(p, z + p.rank_p, i, pos) : 0.f);
    return;
  }
  const float* q = pr + p.col_q + h * (p.Dp + p.Rp);
  float* qa = p.qa + ((long long)b * p.H + h) * pitch;
  float *sq = sm, *acc = sm + p.Dp;
  for (int i = tid; i < p.D; i += LQ_THREADS) sq[i] = q[i];
  if (c0 == 0)
    for (int i = tid; i < p.Rp; i += LQ_THREADS) qa[p.rank_p + i] = i < p.R ? turn_part(p, q + p.Dp, i, pos) : 0.f;
  __syncthreads();
  float a[VEC];
#pragma unroll
  for (int i = 0; i < VEC; ++i) a[i] = 0.f;
  if (work) {
    auto take = [&](const uint4& u, int d) {
      float f[VEC];
      unpack_vec<T>(u, f);
#pragma unroll
      for (int i = 0; i < VEC; ++i) a[i] += f[i] * sq[d];
    };
#pragma unroll
    for (int i = 0; i < PRE; ++i)
      if (gr + i * GR < p.D) take(pre[i], gr + i * GR);
#pragma unroll 4
    for (int d = gr + PRE * GR; d < p.D; d += GR) take(*reinterpret_cast<const uint4*>(up + (long long)d * p.rank_p), d);
  }
  // key rows of a warp's lanes, then of the warps
#pragma unroll
  for (int o = TX; o < 32; o <<= 1)
#pragma unroll
    for (int i = 0; i < VEC; ++i) a[i] += __shfl_xor_sync(0xffffffffu, a[i], o);
  if ((tid & 31) < TX) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) acc[(tid >> 5) * LQ_COLS + tx * VEC + i] = a[i];
  }
  __syncthreads();
  if (tid < LQ_COLS && c0 + tid < p.rank_p) {
    float s = 0.f;
#pragma unroll
    for (int g = 0; g < LQ_THREADS / 32; ++g) s += acc[g * LQ_COLS + tid];
    qa[c0 + tid] = s;
  }
}

// ------------------------------------------------------------------------------------------------ step: attention
constexpr int LS_THREADS = 128, LS_KEYS = 256, LS_GRAIN = 64;

__device__ __forceinline__ void latent_range(long long n, int splits, int s, int* k0, int* k1) {
  int per = ((int)n + splits - 1) / splits;
  per = max(LS_GRAIN, (per + LS_GRAIN - 1) / LS_GRAIN * LS_GRAIN);
  *k0 = min((int)n, s * per);
  *k1 = min((int)n, *k0 + per);
}

// Any sizes and fp32 caches, fp32 arithmetic: blocks (split, head, sequence); a warp per key for the scores, a thread per column for the sums.
template <class T>
__global__ void __launch_bounds__(LS_THREADS) latent_step_kernel(const LatentStepArgs p) {
  constexpr int VEC = 16 / sizeof(T), NC = 2048 / LS_THREADS;
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[33], stat[2];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int split = blockIdx.x % p.splits, bh = blockIdx.x / p.splits, h = bh % p.H, b = bh / p.H;
  const int pitch = p.rank_p + p.Rp;
  launch_dependents();
  wait_for_previous();
  const long long pos = pos_of(p.pos);
  float* part = p.part + ((long long)bh * p.splits + split) * part_stride(p.rank_p);
  int k0 = 0, k1 = 0;
  if (pos >= 0 && pos < p.cap) latent_range(pos + 1, p.splits, split, &k0, &k1);
  float *sq = sm, *sp = sm + pitch;
  const float* qa = p.qa + ((long long)b * p.H + h) * pitch;
  for (int i = tid; i < pitch; i += LS_THREADS) sq[i] = qa[i];
  __syncthreads();
  const T* C = (const T*)p.cache + (long long)b * p.cap * pitch;
  float m = -INFINITY, l = 0.f, acc[NC];
#pragma unroll
  for (int i = 0; i < NC; ++i) acc[i] = 0.f;
  for (int kb = k0; kb < k1; kb += LS_KEYS) {
    const int n = min(LS_KEYS, k1 - kb);
    for (int j = warp; j < n; j += LS_THREADS / 32) {
      const T* c = C + (long long)(kb + j) * pitch;
      float s = 0.f;
      for (int d = lane * VEC; d < pitch; d += 32 * VEC) {
        float f[VEC];
        load_vec(c + d, f);
#pragma unroll
        for (int i = 0; i < VEC; ++i) s += f[i] * sq[d + i];
      }
      s = warp_sum(s);
      if (lane == 0) sp[j] = s * p.scale;
    }
    __syncthreads();
    if (warp == 0) {
      float t = m;
      for (int j = lane; j < n; j += 32) t = fmaxf(t, sp[j]);
      t = warp_max(t);
      if (lane == 0) stat[0] = t;
    }
    __syncthreads();
    const float mn = stat[0], corr = expf(m - mn);
    float e = 0.f;
    for (int j = tid; j < n; j += LS_THREADS) {
      sp[j] = expf(sp[j] - mn);
      e += sp[j];
    }
    l = l * corr + block_sum(e, red);
    m = mn;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int d = tid + i * LS_THREADS;
      if (d >= p.rank_p) break;
      float a = acc[i] * corr;
      for (int j = 0; j < n; ++j) a += sp[j] * ldf(C + (long long)(kb + j) * pitch + d);
      acc[i] = a;
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < NC; ++i) {
    const int d = tid + i * LS_THREADS;
    if (d < p.rank_p) part[4 + d] = acc[i];
  }
  if (tid == 0) {
    part[0] = m;
    part[1] = l;
  }
}

// bf16 caches on the tensor cores, up to 16 heads at a time: blocks (split, group of 16 heads, sequence). Queries are fp32
// and enter as two bf16 numbers, cached rows are exact operands, softmax weights enter as two bf16 numbers again. A warp has
// the query entries of every eighth step of 32 in registers and forms its part of the scores of a tile of 64 keys; for the
// sums it has NG times 16 columns of the latent. Accumulators stay in registers, two tiles of rows alternate in shared memory.
constexpr int LM_THREADS = 256, LM_KEYS = 64, LM_PITCH = 640, LM_STEPS = (LM_PITCH / 32 + 7) / 8;

__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ld_matrix(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p))
               : "memory");
}
__device__ __forceinline__ void ld_matrix_t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p))
               : "memory");
}
__host__ __device__ constexpr int lm_row(int pitch) { return (pitch + 31) / 32 * 32 + 8; }  // shared-memory row, no bank conflicts
constexpr int LM_PROW = LM_KEYS + 8;
constexpr int LM_PARTS = 8 * 16 * LM_KEYS * 4;  // bytes of the warps' parts of the scores, in the place of the queries
__host__ __device__ constexpr int lm_queries(int pitch) { return 2 * 16 * lm_row(pitch) * 2 > LM_PARTS ? 2 * 16 * lm_row(pitch) * 2 : LM_PARTS; }
inline size_t lm_smem(int pitch) {
  return (size_t)lm_queries(pitch) + 2 * LM_KEYS * lm_row(pitch) * 2 + 2 * 16 * LM_PROW * 2 + 3 * 16 * 4;
}

template <int NG>
__global__ void __launch_bounds__(LM_THREADS) latent_step_mma_kernel(const LatentStepArgs p) {
  using bf16 = __nv_bfloat16;
  extern __shared__ __align__(16) uint8_t lm_raw[];
  const int pitch = p.rank_p + p.Rp, row = lm_row(pitch), groups = (p.H + 15) / 16;
  bf16 *qh = reinterpret_cast<bf16*>(lm_raw), *ql = qh + 16 * row, *keys = reinterpret_cast<bf16*>(lm_raw + lm_queries(pitch));
  float* ss = reinterpret_cast<float*>(lm_raw);  // [warp][head][key], once the queries are in registers
  bf16 *ph = keys + 2 * LM_KEYS * row, *pl = ph + 16 * LM_PROW;
  float *sm_m = reinterpret_cast<float*>(pl + 16 * LM_PROW), *sm_l = sm_m + 16, *sm_c = sm_l + 16;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int split = blockIdx.x % p.splits, u = blockIdx.x / p.splits, grp = u % groups, b = u / groups, h0 = grp * 16, nh = min(16, p.H - h0);
  const long long pos = pos_of(p.pos);
  int k0 = 0, k1 = 0;
  if (pos >= 0 && pos < p.cap) latent_range(pos + 1, p.splits, split, &k0, &k1);
  const bf16* C = (const bf16*)p.cache + (long long)b * p.cap * pitch;
  const int pieces = pitch / 8, wide = (row - 8) / 8;  // 16-byte pieces of a cached row, and with the zeros behind it
  auto stage = [&](int buf, int kb) {
    bf16* dst = keys + buf * LM_KEYS * row;
#pragma unroll
    for (int i = 0; i < LM_KEYS / 8; ++i) {
      const int r = warp + 8 * i;
      const bf16* src = C + (long long)(kb + r) * pitch;
#pragma unroll
      for (int j = 0; j < (LM_PITCH / 8 + 31) / 32; ++j) {
        const int c = j * 32 + lane;
        const bool on = kb + r < k1 && c < pieces;
        if (c < wide)
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst + r * row + c * 8)), "l"(on ? src + c * 8 : C),
                       "r"(on ? 16 : 0)
                       : "memory");
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // Rows of earlier positions were complete before this step's first kernel started (the embedding rows, launched without
  // overlap): they are fetched ahead of the wait. Only the position's own row comes from the kernel before this one.
  const bool ahead = k0 < k1 && min(k0 + LM_KEYS, k1) <= pos;
  if (ahead) stage(0, k0);
  launch_dependents();
  wait_for_previous();
  if (k0 < k1 && !ahead) stage(0, k0);
  const float* qa = p.qa + ((long long)b * p.H + h0) * pitch;
#pragma unroll
  for (int i = 0; i < 2; ++i) {  // a warp has two heads, a lane four neighbouring entries
    const int r = warp * 2 + i;
#pragma unroll
    for (int j = 0; j < LM_PITCH / 128; ++j) {
      const int c = (j * 32 + lane) * 4;
      if (c < row - 8) {
        const float4 x = r < nh && c < pitch ? *reinterpret_cast<const float4*>(qa + (long long)r * pitch + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        const uint32_t a = pack_bf16x2(x.x, x.y), d = pack_bf16x2(x.z, x.w);
        *reinterpret_cast<uint2*>(qh + r * row + c) = make_uint2(a, d);
        *reinterpret_cast<uint2*>(ql + r * row + c) =
            make_uint2(pack_bf16x2(x.x - __uint_as_float(a << 16), x.y - __uint_as_float(a & 0xffff0000u)),
                       pack_bf16x2(x.z - __uint_as_float(d << 16), x.w - __uint_as_float(d & 0xffff0000u)));
      }
    }
  }
  if (tid < 16) {
    sm_m[tid] = -INFINITY;
    sm_l[tid] = 0.f;
  }
  float acc[NG][8];
#pragma unroll
  for (int g = 0; g < NG; ++g)
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[g][e] = 0.f;
  __syncthreads();
  // a warp's steps beyond the row have zero queries on the first columns, which keeps the products free of branches
  uint32_t ah[LM_STEPS][2][4], al[LM_STEPS][2][4];
  int at[LM_STEPS];
#pragma unroll
  for (int i = 0; i < LM_STEPS; ++i) {
    const bool on = (warp + 8 * i) * 32 < row - 8;
    at[i] = on ? (warp + 8 * i) * 32 : 0;
    const int off = (lane & 15) * row + (lane >> 4) * 8 + at[i];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      ld_matrix(ah[i][j], qh + off + 16 * j);
      ld_matrix(al[i][j], ql + off + 16 * j);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        ah[i][j][e] = on ? ah[i][j][e] : 0u;
        al[i][j][e] = on ? al[i][j][e] : 0u;
      }
    }
  }
  for (int kb = k0, buf = 0; kb < k1; kb += LM_KEYS, buf ^= 1) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (kb + LM_KEYS < k1) stage(buf ^ 1, kb + LM_KEYS);
    const bf16* kt = keys + buf * LM_KEYS * row;
#pragma unroll
    for (int t = 0; t < LM_KEYS / 8; ++t) {
      float s[4] = {0.f, 0.f, 0.f, 0.f}, s2[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int i = 0; i < LM_STEPS; ++i) {
        uint32_t kv[4];
        ld_matrix(kv, kt + (t * 8 + (lane & 7)) * row + (lane >> 3) * 8 + at[i]);
        mma_bf16(s, ah[i][0], kv[0], kv[1]);
        mma_bf16(s2, al[i][0], kv[0], kv[1]);
        mma_bf16(s, ah[i][1], kv[2], kv[3]);
        mma_bf16(s2, al[i][1], kv[2], kv[3]);
      }
      float* o = ss + (warp * 16 + (lane >> 2)) * LM_KEYS + t * 8 + 2 * (lane & 3);
      *reinterpret_cast<float2*>(o) = make_float2(s[0] + s2[0], s[1] + s2[1]);
      *reinterpret_cast<float2*>(o + 8 * LM_KEYS) = make_float2(s[2] + s2[2], s[3] + s2[3]);
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int hh = warp * 2 + i;
      float x0 = 0.f, x1 = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) {
        const float2 v = *reinterpret_cast<const float2*>(ss + (w * 16 + hh) * LM_KEYS + 2 * lane);
        x0 += v.x;
        x1 += v.y;
      }
      x0 = kb + 2 * lane < k1 ? x0 * p.scale : -INFINITY;
      x1 = kb + 2 * lane + 1 < k1 ? x1 * p.scale : -INFINITY;
      const float mo = sm_m[hh], mn = fmaxf(mo, warp_max(fmaxf(x0, x1)));  // every tile has a key: finite
      const float e0 = expf(x0 - mn), e1 = expf(x1 - mn), l = warp_sum(e0 + e1);
      const uint32_t hi = pack_bf16x2(e0, e1);
      *reinterpret_cast<uint32_t*>(ph + hh * LM_PROW + 2 * lane) = hi;
      *reinterpret_cast<uint32_t*>(pl + hh * LM_PROW + 2 * lane) =
          pack_bf16x2(e0 - __uint_as_float(hi << 16), e1 - __uint_as_float(hi & 0xffff0000u));
      __syncwarp();
      if (lane == 0) {
        const float c = expf(mo - mn);
        sm_c[hh] = c;
        sm_l[hh] = sm_l[hh] * c + l;
        sm_m[hh] = mn;
      }
    }
    __syncthreads();
    const float c0 = sm_c[lane >> 2], c1 = sm_c[(lane >> 2) + 8];
    uint32_t wh[4][4], wl[4][4];
#pragma unroll
    for (int t = 0; t < 4; ++t) {
      ld_matrix(wh[t], ph + (lane & 15) * LM_PROW + t * 16 + (lane >> 4) * 8);
      ld_matrix(wl[t], pl + (lane & 15) * LM_PROW + t * 16 + (lane >> 4) * 8);
    }
#pragma unroll
    for (int g = 0; g < NG; ++g) {
      // groups beyond the latent repeat the first columns; they are not stored
      const int col = (warp + 8 * g) * 16 < p.rank_p ? (warp + 8 * g) * 16 : 0;
      float lo[4], hi[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        lo[e] = acc[g][e] * (e < 2 ? c0 : c1);
        hi[e] = acc[g][4 + e] * (e < 2 ? c0 : c1);
      }
#pragma unroll
      for (int t = 0; t < 4; ++t) {
        uint32_t v[4];
        ld_matrix_t(v, kt + (t * 16 + (lane & 15)) * row + col + (lane >> 4) * 8);
        mma_bf16(lo, wh[t], v[0], v[1]);
        mma_bf16(hi, wh[t], v[2], v[3]);
        mma_bf16(lo, wl[t], v[0], v[1]);
        mma_bf16(hi, wl[t], v[2], v[3]);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        acc[g][e] = lo[e];
        acc[g][4 + e] = hi[e];
      }
    }
  }
  __syncthreads();
  const int ES = part_stride(p.rank_p);
  auto part_of = [&](int hh) { return p.part + (((long long)b * p.H + h0 + hh) * p.splits + split) * ES; };
  if (tid < nh) {
    float* o = part_of(tid);
    o[0] = sm_m[tid];
    o[1] = sm_l[tid];
  }
  if (k0 >= k1) return;  // the combination does not read the values of empty splits
#pragma unroll
  for (int g = 0; g < NG; ++g) {
    const int col = (warp + 8 * g) * 16 + 2 * (lane & 3);
#pragma unroll
    for (int e = 0; e < 8; e += 2) {
      const int hh = (lane >> 2) + ((e >> 1) & 1) * 8, c = col + (e >> 2) * 8;
      if (hh < nh && c < p.rank_p) *reinterpret_cast<float2*>(part_of(hh) + 4 + c) = make_float2(acc[g][e], acc[g][e + 1]);
    }
  }
}

// ------------------------------------------------------------------------------------------------ step: values
constexpr int LV_THREADS = 512, LV_ROWS = 32;

// blocks (32 rows of a head's value expansion, head, sequence): combines the head's splits, then a warp per row
template <class T>
__global__ void __launch_bounds__(LV_THREADS) latent_value_kernel(const LatentStepArgs p, int slices) {
  constexpr int VEC = 16 / sizeof(T);
  extern __shared__ __align__(16) float sm[];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int slice = blockIdx.x % slices, bh = blockIdx.x / slices, h = bh % p.H, b = bh / p.H;
  const int ES = part_stride(p.rank_p);
  float *sa = sm, *sc = sm + p.rank_p;
  constexpr int ROWS = LV_ROWS / (LV_THREADS / 32), PRE = 2;  // rows per warp; pieces of a row fetched before the wait
  const T* up = (const T*)p.up + ((long long)h * (p.Dp + p.Ep) + p.Dp) * p.rank_p;
  uint4 pre[ROWS][PRE];
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    const int r = slice * LV_ROWS + warp + i * (LV_THREADS / 32);
#pragma unroll
    for (int j = 0; j < PRE; ++j)
      if (r < p.E && (j * 32 + lane) * VEC < p.rank_p) pre[i][j] = *reinterpret_cast<const uint4*>(up + (long long)r * p.rank_p + (j * 32 + lane) * VEC);
  }
  launch_dependents();
  wait_for_previous();
  const float* part = p.part + (long long)bh * p.splits * ES;
  int active = 1;  // splits beyond the keys hold nothing
  {
    int a, z;
    const long long n = min(pos_of(p.pos) + 1, (long long)p.cap);
    latent_range(n, p.splits, 0, &a, &z);
    active = min(p.splits, ((int)n + z - 1) / max(z, 1));
  }
  if (warp == 0) {
    const float sink = p.sink != nullptr ? p.sink[h] : -INFINITY;
    float m = sink, l = 0.f;
    for (int s = lane; s < active; s += 32) m = fmaxf(m, part[(long long)s * ES]);
    m = warp_max(m);
    for (int s = lane; s < active; s += 32) {
      const float c = expf(part[(long long)s * ES] - m);
      sc[s] = c;
      l += part[(long long)s * ES + 1] * c;
    }
    l = warp_sum(l) + (p.sink != nullptr ? expf(sink - m) : 0.f);
    float r = p.out_scale / l;
    if (p.col_g >= 0) r *= sigmoid_f(p.proj[(long long)b * p.ld + p.col_g + h]);
    __syncwarp();
    for (int s = lane; s < active; s += 32) sc[s] *= r;
  }
  __syncthreads();
  // threads of a group have the quads of a latent, the groups share the splits
  const int quads = p.rank_p / 4, groups = max(1, LV_THREADS / quads);
  float* red = sc + (p.splits + 3) / 4 * 4;
  for (int i = tid; i < quads * groups; i += LV_THREADS) {
    const int qd = i % quads, g = i / quads;
    float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 16
    for (int s = g; s < active; s += groups) {
      const float c = sc[s];
      const float4 v = *reinterpret_cast<const float4*>(part + (long long)s * ES + 4 + qd * 4);
      t.x += c * v.x; t.y += c * v.y; t.z += c * v.z; t.w += c * v.w;
    }
    *reinterpret_cast<float4*>(red + i * 4) = t;
  }
  __syncthreads();
  for (int i = tid; i < p.rank_p; i += LV_THREADS) {
    float t = 0.f;
    for (int g = 0; g < groups; ++g) t += red[g * p.rank_p + i];
    sa[i] = t;
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    const int r = slice * LV_ROWS + warp + i * (LV_THREADS / 32);
    if (r >= p.E) break;
    float s = 0.f;
    auto take = [&](const uint4& u, int d) {
      float f[VEC];
      unpack_vec<T>(u, f);
#pragma unroll
      for (int e = 0; e < VEC; ++e) s += f[e] * sa[d + e];
    };
#pragma unroll
    for (int j = 0; j < PRE; ++j)
      if ((j * 32 + lane) * VEC < p.rank_p) take(pre[i][j], (j * 32 + lane) * VEC);
    for (int d = (PRE * 32 + lane) * VEC; d < p.rank_p; d += 32 * VEC) take(*reinterpret_cast<const uint4*>(up + (long long)r * p.rank_p + d), d);
    s = warp_sum(s);
    if (lane == 0) p.out[(long long)b * p.ldo + h * p.E + r] = s;
  }
}

}  // namespace

void launch_latent_prep(const LatentPrepArgs& a, cudaStream_t s) {
  if (a.B <= 0 || a.T <= 0) return;
  const dim3 grid(a.T, a.B);
  // heads and cached rows are multiples of eight wide; the matrix itself may start anywhere
  const bool vec = a.R % 16 == 0 && a.col_q % 8 == 0 && (a.col_c < 0 || a.col_c % 8 == 0) && vec8_ok(a.proj, a.ld, a.f32) &&
                   vec8_ok(a.cache, 8, a.f32) && vec8_ok(a.rot, 4, true) && vec8_ok(a.norm_w, 4, true);
  if (a.f32) latent_prep_kernel<float><<<grid, LP_THREADS, 0, s>>>(a, vec);
  else latent_prep_kernel<__nv_bfloat16><<<grid, LP_THREADS, 0, s>>>(a, vec);
  check_launch("latent_prep");
}

// About one block per SM and group of 16 heads.
int latent_step_splits(int B, int H) {
  const int n = 148 / (B * ((H + 15) / 16));
  return n < 1 ? 1 : n > 128 ? 128 : n;
}

void launch_latent_step(const LatentStepArgs& a, cudaStream_t s) {
  if (a.B <= 0) return;
  if (a.rank_p > 2048 || a.rank_p % 8 != 0 || a.Rp % 8 != 0) throw std::runtime_error("latent_step: latents of up to 2048 entries, padded to eight");
  auto go = [&](auto tag) {
    using T = decltype(tag);
    const int slices = (a.rank_p + LQ_COLS - 1) / LQ_COLS, vs = (a.E + LV_ROWS - 1) / LV_ROWS;
    launch_chained(latent_query_kernel<T>, a.B * (slices * a.H + 1), LQ_THREADS, (size_t)(a.Dp + LQ_THREADS / 32 * LQ_COLS) * 4, s, a, slices);
    if (sizeof(T) == 2 && a.rank_p + a.Rp <= LM_PITCH) {
      const int blocks = a.B * ((a.H + 15) / 16) * a.splits, groups = (a.rank_p + 127) / 128;  // 128 columns per round of the warps
      const size_t sm = lm_smem(a.rank_p + a.Rp);
      auto run = [&](auto* kern) {
        cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm);
        launch_chained(kern, blocks, LM_THREADS, sm, s, a);
      };
      if (groups <= 1) run(latent_step_mma_kernel<1>);
      else if (groups <= 2) run(latent_step_mma_kernel<2>);
      else if (groups <= 4) run(latent_step_mma_kernel<4>);
      else run(latent_step_mma_kernel<5>);
    } else {
      launch_chained(latent_step_kernel<T>, a.B * a.H * a.splits, LS_THREADS, (size_t)(a.rank_p + a.Rp + LS_KEYS) * 4, s, a);
    }
    launch_chained(latent_value_kernel<T>, a.B * a.H * vs, LV_THREADS, (size_t)(a.rank_p + (a.splits + 3) / 4 * 4 + (a.rank_p > LV_THREADS * 4 ? a.rank_p : LV_THREADS * 4)) * 4, s, a, vs);
  };
  if (a.f32) go(float{});
  else go(__nv_bfloat16{});
  check_launch("latent_step");
}

}  // namespace tb
