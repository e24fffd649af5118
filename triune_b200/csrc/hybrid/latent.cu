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
__global__ void __launch_bounds__(LP_THREADS) latent_prep_kernel(const LatentPrepArgs p) {
  __shared__ float red[33];
  const int t = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, half = p.R / 2;
  T* pr = (T*)p.proj + ((long long)b * p.T + t) * p.ld;
  const float *cs = p.rot + (long long)t * p.R, *sn = cs + half;
  for (int i = tid; i < p.H * half; i += LP_THREADS) {
    const int h = i / half, d = i % half;
    T* q = pr + p.col_q + h * (p.Dp + p.Rp) + p.Dp;
    const float u = ldf(q + d), v = ldf(q + half + d), c = cs[d], s = sn[d];
    stf(q + d, u * c - v * s);
    stf(q + half + d, v * c + u * s);
  }
  const long long pos = pos_of(p.pos) + t;
  if (p.col_c < 0 || pos < 0 || pos >= p.cap) return;  // the host reserves before every call
  const T* z = pr + p.col_c;
  T* dst = (T*)p.cache + ((long long)b * p.cap + pos) * (p.rank_p + p.Rp);
  float ss = 0.f;
  for (int i = tid; i < p.rank; i += LP_THREADS) ss += ldf(z + i) * ldf(z + i);
  const float r = 1.f / sqrtf(block_sum(ss, red) / p.rank + p.eps);
  for (int i = tid; i < p.rank_p; i += LP_THREADS) stf(dst + i, i < p.rank ? ldf(z + i) * r * p.norm_w[i] : 0.f);
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
  const int pitch = p.rank_p + p.Rp;
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
  const int h = w / slices, c0 = (w % slices) * LQ_COLS;
  const float* q = pr + p.col_q + h * (p.Dp + p.Rp);
  float* qa = p.qa + ((long long)b * p.H + h) * pitch;
  float *sq = sm, *acc = sm + p.Dp;
  for (int i = tid; i < p.D; i += LQ_THREADS) sq[i] = q[i];
  if (c0 == 0)
    for (int i = tid; i < p.Rp; i += LQ_THREADS) qa[p.rank_p + i] = i < p.R ? turn_part(p, q + p.Dp, i, pos) : 0.f;
  __syncthreads();
  const int tx = tid % TX, gr = tid / TX, col = c0 + tx * VEC;
  float a[VEC];
#pragma unroll
  for (int i = 0; i < VEC; ++i) a[i] = 0.f;
  if (col < p.rank_p) {  // rank_p is a multiple of eight
    const T* up = (const T*)p.up + (long long)h * (p.Dp + p.Ep) * p.rank_p + col;
#pragma unroll 4
    for (int d = gr; d < p.D; d += GR) {
      float f[VEC];
      load_vec(up + (long long)d * p.rank_p, f);
#pragma unroll
      for (int i = 0; i < VEC; ++i) a[i] += f[i] * sq[d];
    }
  }
#pragma unroll
  for (int i = 0; i < VEC; ++i) acc[gr * LQ_COLS + tx * VEC + i] = a[i];
  __syncthreads();
  if (tid < LQ_COLS && c0 + tid < p.rank_p) {
    float s = 0.f;
    for (int g = 0; g < GR; ++g) s += acc[g * LQ_COLS + tid];
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

// Any sizes, fp32 arithmetic: blocks (split, head, sequence); a warp per key for the scores, a thread per column for the sums.
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

// ------------------------------------------------------------------------------------------------ step: values
constexpr int LV_THREADS = 256, LV_ROWS = 32;

// blocks (32 rows of a head's value expansion, head, sequence): combines the head's splits, then a warp per row
template <class T>
__global__ void __launch_bounds__(LV_THREADS) latent_value_kernel(const LatentStepArgs p, int slices) {
  constexpr int VEC = 16 / sizeof(T);
  extern __shared__ __align__(16) float sm[];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int slice = blockIdx.x % slices, bh = blockIdx.x / slices, h = bh % p.H, b = bh / p.H;
  const int ES = part_stride(p.rank_p);
  float *sa = sm, *sc = sm + p.rank_p;
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
  for (int i = tid * 4; i < p.rank_p; i += LV_THREADS * 4) {
    float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int s = 0; s < active; ++s) {
      const float c = sc[s];
      const float4 v = *reinterpret_cast<const float4*>(part + (long long)s * ES + 4 + i);
      t.x += c * v.x; t.y += c * v.y; t.z += c * v.z; t.w += c * v.w;
    }
    *reinterpret_cast<float4*>(sa + i) = t;
  }
  __syncthreads();
  const T* up = (const T*)p.up + ((long long)h * (p.Dp + p.Ep) + p.Dp) * p.rank_p;
  for (int r = slice * LV_ROWS + warp; r < min(p.E, (slice + 1) * LV_ROWS); r += LV_THREADS / 32) {
    const T* wr = up + (long long)r * p.rank_p;
    float s = 0.f;
    for (int d = lane * VEC; d < p.rank_p; d += 32 * VEC) {
      float f[VEC];
      load_vec(wr + d, f);
#pragma unroll
      for (int i = 0; i < VEC; ++i) s += f[i] * sa[d + i];
    }
    s = warp_sum(s);
    if (lane == 0) p.out[(long long)b * p.ldo + h * p.E + r] = s;
  }
}

}  // namespace

void launch_latent_prep(const LatentPrepArgs& a, cudaStream_t s) {
  if (a.B <= 0 || a.T <= 0) return;
  const dim3 grid(a.T, a.B);
  if (a.f32) latent_prep_kernel<float><<<grid, LP_THREADS, 0, s>>>(a);
  else latent_prep_kernel<__nv_bfloat16><<<grid, LP_THREADS, 0, s>>>(a);
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
    constexpr int VEC = 16 / sizeof(T), GR = LQ_THREADS / (LQ_COLS / VEC);
    const int slices = (a.rank_p + LQ_COLS - 1) / LQ_COLS, vs = (a.E + LV_ROWS - 1) / LV_ROWS;
    launch_chained(latent_query_kernel<T>, a.B * (slices * a.H + 1), LQ_THREADS, (size_t)(a.Dp + GR * LQ_COLS) * 4, s, a, slices);
    launch_chained(latent_step_kernel<T>, a.B * a.H * a.splits, LS_THREADS, (size_t)(a.rank_p + a.Rp + LS_KEYS) * 4, s, a);
    launch_chained(latent_value_kernel<T>, a.B * a.H * vs, LV_THREADS, (size_t)(a.rank_p + a.splits) * 4, s, a, vs);
  };
  if (a.f32) go(float{});
  else go(__nv_bfloat16{});
  check_launch("latent_step");
}

}  // namespace tb
