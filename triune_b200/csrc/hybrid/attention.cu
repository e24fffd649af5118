// Softmax attention with per-head query / key norm, partial interleaved rotation and a sink: preparation of queries,
// keys and values, and an fp32 CUDA-core attention kernel for every head size (fp32 models, and bf16 head sizes that
// the tensor-core kernel does not take).
#include "hybrid.cuh"

namespace tb {
namespace {

// block: one token of one sequence, four warps over the heads of q, k and v
template <class T>
__global__ void attn_prep_kernel(const AttnPrepArgs p) {
  extern __shared__ float sm[];  // cos [rot/2], sin [rot/2], then one head row per warp
  const int half = p.rot_dims / 2;
  float *cs = sm, *sn = sm + half;
  const int t = blockIdx.x, b = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  float* row = sm + 2 * half + warp * p.D;
  const long long pos = pos_of(p.pos) + t;
  if (pos < 0 || pos >= p.cap) return;  // outside the cache: skipped, the host reserves before every call
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float s, c;
    rotation(pos, p.freqs[i], &s, &c);
    cs[i] = c;
    sn[i] = s;
  }
  __syncthreads();
  const T* pr = (const T*)p.proj + ((long long)b * p.T + t) * p.ld;
  for (int hh = warp; hh < p.H + p.G; hh += nw) {
    const bool isq = hh < p.H;
    const int h = isq ? hh : hh - p.H;
    const T* src = pr + (isq ? p.col_q : p.col_k) + h * p.D;
    T* dst = isq ? (T*)p.q + (((long long)b * p.H + h) * p.T + t) * p.pitch_k
                 : (T*)p.kc + (((long long)b * p.G + h) * p.cap + pos) * p.pitch_k;
    const float* w = isq ? p.q_w : p.k_w;
    float ss = 0.f;
    for (int d = lane; d < p.D; d += 32) {
      const float v = ldf(src + d);
      row[d] = v;
      ss += v * v;
    }
    ss = warp_sum(ss);
    const float r = w != nullptr ? 1.f / sqrtf(ss / p.D + p.eps) : 1.f;
    __syncwarp();
    for (int d = lane; d < p.pitch_k; d += 32) {
      float v = 0.f;
      if (d < p.D) {
        v = row[d] * r * (w != nullptr ? w[d] : 1.f);
        if (d < p.rot_dims) {
          const int o = d ^ 1, i = d >> 1;
          const float other = row[o] * r * (w != nullptr ? w[o] : 1.f);
          v = (d & 1) ? v * cs[i] + other * sn[i] : v * cs[i] - other * sn[i];
        }
      }
      stf(dst + d, v);
    }
    __syncwarp();
  }
  for (int i = threadIdx.x; i < p.G * p.pitch_v; i += blockDim.x) {
    const int g = i / p.pitch_v, e = i % p.pitch_v;
    stf((T*)p.vc + (((long long)b * p.G + g) * p.cap + pos) * p.pitch_v + e, e < p.E ? ldf(pr + p.col_v + g * p.E + e) : 0.f);
  }
}

__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ld4(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16),
                     __uint_as_float(u.y & 0xffff0000u));
}
__device__ __forceinline__ void st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void st4(__nv_bfloat16* p, float4 v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 u;
  u.x = *reinterpret_cast<uint32_t*>(&a);
  u.y = *reinterpret_cast<uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = u;
}

constexpr int AP_TOK = 4, AP_WARPS = 8;

// Four tokens per block, a warp per (token, head) row, four neighbouring elements (two rotation pairs) per lane. Head
// sizes and columns are multiples of four, rot_dims is even, D <= 128 NV.
template <class T, int NV>
__global__ void __launch_bounds__(AP_WARPS * 32) attn_prep_vec_kernel(const AttnPrepArgs p) {
  extern __shared__ float2 rot[];  // [AP_TOK][rot / 2]: cos, sin
  const int half = p.rot_dims / 2, t0 = blockIdx.x * AP_TOK, b = blockIdx.y, nt = min(AP_TOK, p.T - t0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long pos0 = pos_of(p.pos) + t0;
  for (int i = threadIdx.x; i < nt * half; i += blockDim.x) {
    float s, c;
    rotation(pos0 + i / half, p.freqs[i % half], &s, &c);
    rot[i] = make_float2(c, s);
  }
  __syncthreads();
  const int rows = p.H + 2 * p.G;
  for (int it = warp; it < nt * rows; it += AP_WARPS) {
    const int ti = it / rows, hh = it % rows, t = t0 + ti;
    const long long pos = pos0 + ti;
    if (pos < 0 || pos >= p.cap) continue;
    const T* pr = (const T*)p.proj + ((long long)b * p.T + t) * p.ld;
    if (hh >= p.H + p.G) {
      const int g = hh - p.H - p.G;
      T* dst = (T*)p.vc + (((long long)b * p.G + g) * p.cap + pos) * p.pitch_v;
      for (int e = lane * 4; e < p.pitch_v; e += 128)
        st4(dst + e, e < p.E ? ld4(pr + p.col_v + g * p.E + e) : make_float4(0.f, 0.f, 0.f, 0.f));
      continue;
    }
    const bool isq = hh < p.H;
    const int h = isq ? hh : hh - p.H;
    const T* src = pr + (isq ? p.col_q : p.col_k) + h * p.D;
    T* dst = isq ? (T*)p.q + (((long long)b * p.H + h) * p.T + t) * p.pitch_k
                 : (T*)p.kc + (((long long)b * p.G + h) * p.cap + pos) * p.pitch_k;
    const float* w = isq ? p.q_w : p.k_w;
    float4 v[NV];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int d = (i * 32 + lane) * 4;
      v[i] = d < p.D ? ld4(src + d) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    const float r = w != nullptr ? 1.f / sqrtf(warp_sum(ss) / p.D + p.eps) : 1.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int d = (i * 32 + lane) * 4;
      if (d >= p.pitch_k) continue;
      float4 x = v[i];
      if (w != nullptr && d < p.D) {
        const float4 g = ld4(w + d);
        x = make_float4(x.x * r * g.x, x.y * r * g.y, x.z * r * g.z, x.w * r * g.w);
      }
      if (d < p.rot_dims) {
        const float2 a = rot[ti * half + d / 2];
        const float u = x.x * a.x - x.y * a.y;
        x.y = x.y * a.x + x.x * a.y;
        x.x = u;
      }
      if (d + 2 < p.rot_dims) {
        const float2 a = rot[ti * half + d / 2 + 1];
        const float u = x.z * a.x - x.w * a.y;
        x.w = x.w * a.x + x.z * a.y;
        x.z = u;
      }
      st4(dst + d, x);
    }
  }
}

constexpr int AS_Q = 8, AS_K = 32;

// block: AS_Q consecutive queries of one head, a warp each; keys and values in tiles of 32; value sizes up to 32 NE
template <class T, int NE>
__global__ void attn_simple_kernel(const AttnArgs p) {
  extern __shared__ float sm[];
  const int D = p.D + p.R, dp = D + 1;
  float *sk = sm, *sv = sk + AS_K * dp, *sq = sv + AS_K * p.E;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, b = blockIdx.z, t = blockIdx.x * AS_Q + warp, g = h / (p.H / p.G);
  const long long p0 = pos_of(p.pos);
  const bool live = t < p.T;
  const long long qpos = p0 + t;
  const long long kend = min(p0 + min((blockIdx.x + 1) * AS_Q, p.T), (long long)p.rows);  // keys any query of the block sees
  auto at = [&](const AttnOperand& o, long long row, int head) { return (const T*)o.p + b * o.sb + row * o.sr + head * o.sh; };
  float* q = sq + warp * D;
  if (live) {
    const T* Q = at(p.q, t, h);
    for (int d = lane; d < p.D; d += 32) q[d] = ldf(Q + d);
    if (p.R > 0) {
      const T* Q2 = at(p.q2, t, h);
      for (int d = lane; d < p.R; d += 32) q[p.D + d] = ldf(Q2 + d);
    }
  }
  float m = p.sink != nullptr ? p.sink[h] : -INFINITY, l = p.sink != nullptr ? 1.f : 0.f;
  float acc[NE];
#pragma unroll
  for (int i = 0; i < NE; ++i) acc[i] = 0.f;
  for (long long k0 = 0; k0 < kend; k0 += AS_K) {
    const int n = (int)min((long long)AS_K, kend - k0);
    __syncthreads();
    for (int i = threadIdx.x; i < n * p.D; i += blockDim.x) sk[(i / p.D) * dp + i % p.D] = ldf(at(p.k, k0 + i / p.D, g) + i % p.D);
    for (int i = threadIdx.x; i < n * p.R; i += blockDim.x) sk[(i / p.R) * dp + p.D + i % p.R] = ldf(at(p.k2, k0 + i / p.R, 0) + i % p.R);
    for (int i = threadIdx.x; i < n * p.E; i += blockDim.x) sv[i] = ldf(at(p.v, k0 + i / p.E, g) + i % p.E);
    __syncthreads();
    if (!live || k0 > qpos) continue;
    float s = -INFINITY;
    if (lane < n && k0 + lane <= qpos) {
      float a = 0.f;
      for (int d = 0; d < D; ++d) a += q[d] * sk[lane * dp + d];
      s = a * p.scale;
    }
    const float mn = fmaxf(m, warp_max(s));
    const float corr = expf(m - mn), e = expf(s - mn);
    l = l * corr + warp_sum(e);
    m = mn;
#pragma unroll
    for (int i = 0; i < NE; ++i) acc[i] *= corr;
    for (int j = 0; j < n; ++j) {
      const float w = __shfl_sync(0xffffffffu, e, j);
#pragma unroll
      for (int i = 0; i < NE; ++i)
        if (lane + 32 * i < p.E) acc[i] += w * sv[j * p.E + lane + 32 * i];
    }
  }
  if (live) {
    T* o = (T*)p.out + ((long long)b * p.T + t) * p.ldo + h * p.E;
    float r = p.out_scale / l;
    if (p.gate != nullptr) r *= sigmoid_f(ldf((const T*)p.gate + ((long long)b * p.T + t) * p.ldg + h));
#pragma unroll
    for (int i = 0; i < NE; ++i)
      if (lane + 32 * i < p.E) stf(o + lane + 32 * i, acc[i] * r);
  }
}

}  // namespace

void launch_attn_prep(const AttnPrepArgs& a, cudaStream_t s) {
  if (a.B <= 0 || a.T <= 0) return;
  const auto quad = [](const void* p, bool f32) { return (reinterpret_cast<uintptr_t>(p) & (f32 ? 15 : 7)) == 0; };
  if (a.D % 4 == 0 && a.E % 4 == 0 && a.D <= 512 && a.ld % 4 == 0 && a.col_q % 4 == 0 && a.col_k % 4 == 0 && a.col_v % 4 == 0 &&
      quad(a.proj, a.f32) && quad(a.q, a.f32) && quad(a.kc, a.f32) && quad(a.vc, a.f32) &&
      (a.q_w == nullptr || (quad(a.q_w, true) && quad(a.k_w, true)))) {
    const size_t sv = (size_t)AP_TOK * (a.rot_dims / 2) * 8;
    dim3 grid((a.T + AP_TOK - 1) / AP_TOK, a.B);
    auto go = [&](auto* kern) { kern<<<grid, AP_WARPS * 32, sv, s>>>(a); };
    if (a.f32) {
      if (a.D <= 128) go(attn_prep_vec_kernel<float, 1>);
      else go(attn_prep_vec_kernel<float, 4>);
    } else {
      if (a.D <= 128) go(attn_prep_vec_kernel<__nv_bfloat16, 1>);
      else go(attn_prep_vec_kernel<__nv_bfloat16, 4>);
    }
    check_launch("attn_prep");
    return;
  }
  const size_t sm = (size_t)(a.rot_dims / 2 * 2 + 4 * a.D) * 4;
  dim3 grid(a.T, a.B);
  if (a.f32) attn_prep_kernel<float><<<grid, 128, sm, s>>>(a);
  else attn_prep_kernel<__nv_bfloat16><<<grid, 128, sm, s>>>(a);
  check_launch("attn_prep");
}

void launch_attn_simple(const AttnArgs& a, cudaStream_t s) {
  if (a.B <= 0 || a.T <= 0) return;
  if (a.E > 512) throw std::runtime_error("attention: value dimensions up to 512");
  const size_t sm = (size_t)(AS_K * (a.D + a.R + 1) + AS_K * a.E + AS_Q * (a.D + a.R)) * 4;
  if (sm > 200 * 1024) throw std::runtime_error("attention: head dimension too large");
  dim3 grid((a.T + AS_Q - 1) / AS_Q, a.H, a.B);
  auto go = [&](auto* kern) {
    if (sm > 47 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm);
    kern<<<grid, AS_Q * 32, sm, s>>>(a);
  };
  if (a.E <= 256) {
    if (a.f32) go(attn_simple_kernel<float, 8>);
    else go(attn_simple_kernel<__nv_bfloat16, 8>);
  } else {
    if (a.f32) go(attn_simple_kernel<float, 16>);
    else go(attn_simple_kernel<__nv_bfloat16, 16>);
  }
  check_launch("attn_simple");
}

}  // namespace tb
