// Row kernels: embedding rows, layer / RMS norm of the fp32 residual stream, gated activations, gated norms.
#include <type_traits>

#include "hybrid.cuh"

namespace tb {
namespace {

template <class T>
__global__ void embed_rows_kernel(const T* __restrict__ table, const long long* __restrict__ ids, float* __restrict__ out,
                                  int W, int V) {
  const long long row = blockIdx.x;
  const long long id = ids[row];
  const bool ok = id >= 0 && id < V;
  for (int i = threadIdx.x; i < W; i += blockDim.x) out[row * W + i] = ok ? ldf(table + id * W + i) : 0.f;
}

template <class T>
__global__ void norm_rows_kernel(const float* __restrict__ x, const float* __restrict__ w, T* __restrict__ y, int W,
                                 float eps, int kind) {
  extern __shared__ float sx[];
  __shared__ float red[33];
  const float* xr = x + (long long)blockIdx.x * W;
  T* yr = y + (long long)blockIdx.x * W;
  float mean = 0.f;
  if ((W & 3) == 0) {
    float s = 0.f;
    for (int i = threadIdx.x * 4; i < W; i += blockDim.x * 4) {
      const float4 v = *reinterpret_cast<const float4*>(xr + i);
      *reinterpret_cast<float4*>(sx + i) = v;
      s += (v.x + v.y) + (v.z + v.w);
    }
    if (kind == HN_LAYER) mean = block_sum(s, red) / W;
    float q = 0.f;
    for (int i = threadIdx.x * 4; i < W; i += blockDim.x * 4) {  // each thread re-reads only what it wrote
      const float4 v = *reinterpret_cast<const float4*>(sx + i);
      const float a = v.x - mean, b = v.y - mean, c = v.z - mean, d = v.w - mean;
      q += (a * a + b * b) + (c * c + d * d);
    }
    const float r = 1.f / sqrtf(block_sum(q, red) / W + eps);
    for (int i = threadIdx.x * 4; i < W; i += blockDim.x * 4) {
      const float4 v = *reinterpret_cast<const float4*>(sx + i);
      const float4 g = *reinterpret_cast<const float4*>(w + i);
      const float o0 = (v.x - mean) * r * g.x, o1 = (v.y - mean) * r * g.y, o2 = (v.z - mean) * r * g.z,
                  o3 = (v.w - mean) * r * g.w;
      if constexpr (sizeof(T) == 4) {
        *reinterpret_cast<float4*>(yr + i) = make_float4(o0, o1, o2, o3);
      } else {
        __nv_bfloat162 p0 = __floats2bfloat162_rn(o0, o1), p1 = __floats2bfloat162_rn(o2, o3);
        uint2 u;
        u.x = *reinterpret_cast<uint32_t*>(&p0);
        u.y = *reinterpret_cast<uint32_t*>(&p1);
        *reinterpret_cast<uint2*>(yr + i) = u;
      }
    }
  } else {
    float s = 0.f;
    for (int i = threadIdx.x; i < W; i += blockDim.x) {
      sx[i] = xr[i];
      s += sx[i];
    }
    if (kind == HN_LAYER) mean = block_sum(s, red) / W;
    float q = 0.f;
    for (int i = threadIdx.x; i < W; i += blockDim.x) q += (sx[i] - mean) * (sx[i] - mean);
    const float r = 1.f / sqrtf(block_sum(q, red) / W + eps);
    for (int i = threadIdx.x; i < W; i += blockDim.x) stf(yr + i, (sx[i] - mean) * r * w[i]);
  }
}

// A warp per row, the row in registers: NV float4 per lane, W <= 128 NV, W a multiple of 4.
template <class T, int NV>
__global__ void __launch_bounds__(128) norm_warp_kernel(const float* __restrict__ x, const float* __restrict__ w,
                                                        T* __restrict__ y, int rows, int W, float eps, int kind) {
  const int row = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= rows) return;
  const float* xr = x + (long long)row * W;
  T* yr = y + (long long)row * W;
  float4 v[NV];
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * 32 + lane) * 4;
    v[i] = c < W ? *reinterpret_cast<const float4*>(xr + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    s += (v[i].x + v[i].y) + (v[i].z + v[i].w);
  }
  const float mean = kind == HN_LAYER ? warp_sum(s) / W : 0.f;
  float q = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    if ((i * 32 + lane) * 4 < W) {
      const float a = v[i].x - mean, b = v[i].y - mean, c = v[i].z - mean, d = v[i].w - mean;
      q += (a * a + b * b) + (c * c + d * d);
    }
  }
  const float r = 1.f / sqrtf(warp_sum(q) / W + eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * 32 + lane) * 4;
    if (c < W) {
      const float4 g = *reinterpret_cast<const float4*>(w + c);
      const float o0 = (v[i].x - mean) * r * g.x, o1 = (v[i].y - mean) * r * g.y, o2 = (v[i].z - mean) * r * g.z,
                  o3 = (v[i].w - mean) * r * g.w;
      if constexpr (sizeof(T) == 4) {
        *reinterpret_cast<float4*>(yr + c) = make_float4(o0, o1, o2, o3);
      } else {
        __nv_bfloat162 p0 = __floats2bfloat162_rn(o0, o1), p1 = __floats2bfloat162_rn(o2, o3);
        uint2 u;
        u.x = *reinterpret_cast<uint32_t*>(&p0);
        u.y = *reinterpret_cast<uint32_t*>(&p1);
        *reinterpret_cast<uint2*>(yr + c) = u;
      }
    }
  }
}

// L lanes per row (a warp, or a block of 128), the row's sum in registers: NV float4 per lane.
template <class Y, class T, int L, int NV>
__global__ void __launch_bounds__(128) add_norm_vec_kernel(const AddNormArgs p) {
  __shared__ float red[33];
  const long long row = (long long)blockIdx.x * (128 / L) + threadIdx.x / L;
  if (row >= p.rows) return;  // whole warps (L = 32), never part of a block (L = 128)
  const int l = threadIdx.x % L;
  float* xr = p.x + row * p.W;
  const Y* yr = (const Y*)p.y + row * p.ldy;
  auto sum = [&](float v) { return L == 32 ? warp_sum(v) : block_sum(v, red); };
  float4 v[NV], x[NV];
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * L + l) * 4;
    v[i] = x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < p.W) {
      x[i] = *reinterpret_cast<const float4*>(xr + c);
      if constexpr (sizeof(Y) == 4) {
        v[i] = *reinterpret_cast<const float4*>(yr + c);
      } else {
        const uint2 u = *reinterpret_cast<const uint2*>(yr + c);
        v[i] = make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16),
                           __uint_as_float(u.y & 0xffff0000u));
      }
      if (p.bias != nullptr) {
        const float4 b = *reinterpret_cast<const float4*>(p.bias + c);
        v[i] = make_float4(v[i].x + b.x, v[i].y + b.y, v[i].z + b.z, v[i].w + b.w);
      }
      s += (v[i].x + v[i].y) + (v[i].z + v[i].w);
    }
  }
  // v: norm of itself, times w; entries past W stay out of the sums
  auto normed = [&](int kind, float total, const float* w, float eps) {
    const float mean = kind == HN_LAYER ? sum(total) / p.W : 0.f;
    float q = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if ((i * L + l) * 4 < p.W) {
        v[i] = make_float4(v[i].x - mean, v[i].y - mean, v[i].z - mean, v[i].w - mean);
        q += (v[i].x * v[i].x + v[i].y * v[i].y) + (v[i].z * v[i].z + v[i].w * v[i].w);
      }
    const float r = 1.f / sqrtf(sum(q) / p.W + eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * L + l) * 4;
      if (c < p.W) {
        const float4 g = *reinterpret_cast<const float4*>(w + c);
        v[i] = make_float4(v[i].x * r * g.x, v[i].y * r * g.y, v[i].z * r * g.z, v[i].w * r * g.w);
      }
    }
  };
  normed(p.post_kind, s, p.post_w, p.post_eps);
  s = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * L + l) * 4;
    if (c < p.W) {
      v[i] = make_float4(x[i].x + v[i].x, x[i].y + v[i].y, x[i].z + v[i].z, x[i].w + v[i].w);
      *reinterpret_cast<float4*>(xr + c) = v[i];
      s += (v[i].x + v[i].y) + (v[i].z + v[i].w);
    }
  }
  if (p.out == nullptr) return;
  if (p.pre_w != nullptr) normed(p.pre_kind, s, p.pre_w, p.pre_eps);
  T* orow = (T*)p.out + row * p.W;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * L + l) * 4;
    if (c < p.W) {
      if constexpr (sizeof(T) == 4) {
        *reinterpret_cast<float4*>(orow + c) = v[i];
      } else {
        __nv_bfloat162 p0 = __floats2bfloat162_rn(v[i].x, v[i].y), p1 = __floats2bfloat162_rn(v[i].z, v[i].w);
        uint2 u;
        u.x = *reinterpret_cast<uint32_t*>(&p0);
        u.y = *reinterpret_cast<uint32_t*>(&p1);
        *reinterpret_cast<uint2*>(orow + c) = u;
      }
    }
  }
}

// any width: a block per row, the row in shared memory (every thread re-reads only what it wrote)
template <class Y, class T>
__global__ void __launch_bounds__(256) add_norm_kernel(const AddNormArgs p) {
  extern __shared__ float sx[];
  __shared__ float red[33];
  const long long row = blockIdx.x;
  float* xr = p.x + row * p.W;
  const Y* yr = (const Y*)p.y + row * p.ldy;
  auto stats = [&](int kind, float total, float eps, float* mean) {
    *mean = kind == HN_LAYER ? block_sum(total, red) / p.W : 0.f;
    float q = 0.f;
    for (int i = threadIdx.x; i < p.W; i += blockDim.x) q += (sx[i] - *mean) * (sx[i] - *mean);
    return 1.f / sqrtf(block_sum(q, red) / p.W + eps);
  };
  float s = 0.f, mean;
  for (int i = threadIdx.x; i < p.W; i += blockDim.x) {
    sx[i] = ldf(yr + i) + (p.bias != nullptr ? p.bias[i] : 0.f);
    s += sx[i];
  }
  float r = stats(p.post_kind, s, p.post_eps, &mean);
  s = 0.f;
  for (int i = threadIdx.x; i < p.W; i += blockDim.x) {
    sx[i] = xr[i] + (sx[i] - mean) * r * p.post_w[i];
    xr[i] = sx[i];
    s += sx[i];
  }
  if (p.out == nullptr) return;
  T* orow = (T*)p.out + row * p.W;
  if (p.pre_w == nullptr) {
    for (int i = threadIdx.x; i < p.W; i += blockDim.x) stf(orow + i, sx[i]);
    return;
  }
  r = stats(p.pre_kind, s, p.pre_eps, &mean);
  for (int i = threadIdx.x; i < p.W; i += blockDim.x) stf(orow + i, (sx[i] - mean) * r * p.pre_w[i]);
}

template <class T>
__global__ void glu_rows_kernel(const T* __restrict__ gu, long long ld, T* __restrict__ out, long long ldo, int F,
                                long long n, const GluArgs glu) {
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    const long long row = i / F, c = i % F;
    float g = ldf(gu + row * ld + c), u = ldf(gu + row * ld + F + c);
    if (glu.bias != nullptr) {
      g += glu.bias[c];
      u += glu.bias[F + c];
    }
    stf(out + row * ldo + c, glu_f(g, u, glu.act, glu.limit, glu.alpha));
  }
}

template <class T>
__global__ void side_rows_kernel(const T* __restrict__ gate, long long ldg, const T* __restrict__ table, long long ldt,
                                 const long long* __restrict__ ids, int V, int col0, T* __restrict__ out, int dim, long long n, int act) {
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    const long long row = i / dim, c = i % dim, id = ids[row];
    const float e = id >= 0 && id < V ? ldf(table + id * ldt + col0 + c) : 0.f;
    stf(out + i, act_f(ldf(gate + row * ldg + c), act) * e);
  }
}

// dim, columns and pitches multiples of eight
template <class T>
__global__ void side_rows_vec_kernel(const T* __restrict__ gate, long long ldg, const T* __restrict__ table, long long ldt,
                                     const long long* __restrict__ ids, int V, int col0, T* __restrict__ out, int pieces, int n, int act) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const long long row = i / pieces, id = ids[row];
  const int c = (i % pieces) * 8;
  float g[8], e[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
  ld8v(gate + row * ldg + c, g);
  if (id >= 0 && id < V) ld8v(table + id * ldt + col0 + c, e);
#pragma unroll
  for (int j = 0; j < 8; ++j) g[j] = act_f(g[j], act) * e[j];
  st8v(out + (long long)i * 8, g);
}

__global__ void rotation_rows_kernel(const double* __restrict__ freqs, int n, float amplitude, float* __restrict__ out, long long total,
                                     const Pos pos) {
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= total) return;
  const long long t = i / n, c = i % n;
  float s, co;
  rotation(pos_of(pos) + t, freqs[c], &s, &co);
  out[t * 2 * n + c] = co * amplitude;
  out[t * 2 * n + n + c] = s * amplitude;
}

// Gated norm of parts that are a multiple of eight wide: L lanes per part (L = 8, 16, 32 lanes of a warp, or L = 128, a
// block), NV vectors of eight per lane in registers.
template <class T, int L, int NV>
__global__ void __launch_bounds__(128) gated_norm_vec_kernel(const T* __restrict__ y, long long ldy, const T* __restrict__ gate,
                                                             long long ldg, const float* __restrict__ w, int w_period,
                                                             T* __restrict__ out, long long ldo, long long parts_total,
                                                             int groups, int part, float eps, int order, float scale) {
  __shared__ float red[33];
  const long long id = (long long)blockIdx.x * (128 / L) + threadIdx.x / L;
  const bool on = id < parts_total;
  const int l = threadIdx.x % L;
  const long long row = id / groups;
  const int c0 = (int)(id % groups) * part;
  const T *yr = y + row * ldy + c0, *gr = gate + row * ldg + c0;
  const float* wr = w == nullptr ? nullptr : w + c0 % w_period;
  float v[NV][8], q = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * L + l) * 8;
    if (on && c < part) {
      float z[8];
      ld8v(yr + c, v[i]);
      ld8v(gr + c, z);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const float s = silu_for<T>(z[j]);
        if (order == GO_GATE_THEN_NORM) {
          v[i][j] *= s;
          q += v[i][j] * v[i][j];
        } else {
          q += v[i][j] * v[i][j];
          v[i][j] *= s;
        }
      }
    }
  }
  if constexpr (L == 128) {
    q = block_sum(q, red);
  } else {
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1) q += __shfl_xor_sync(0xffffffffu, q, o);
  }
  const float r = scale / sqrtf(q / part + eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * L + l) * 8;
    if (on && c < part) {
      float g[8] = {1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f};
      if (wr != nullptr) ld8v(wr + c, g);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[i][j] *= r * g[j];
      st8v(out + row * ldo + c0 + c, v[i]);
    }
  }
}

// any part width: one warp per (row, part)
template <class T>
__global__ void gated_norm_kernel(const T* __restrict__ y, long long ldy, const T* __restrict__ gate, long long ldg,
                                  const float* __restrict__ w, int w_period, T* __restrict__ out, long long ldo,
                                  long long parts_total, int groups, int part, float eps, int order, float scale) {
  const long long id = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (id >= parts_total) return;
  const int lane = threadIdx.x & 31;
  const long long row = id / groups;
  const int c0 = (int)(id % groups) * part;
  const T *yr = y + row * ldy + c0, *gr = gate + row * ldg + c0;
  const float* wr = w == nullptr ? nullptr : w + c0 % w_period;
  T* orow = out + row * ldo + c0;
  float q = 0.f;
  for (int i = lane; i < part; i += 32) {
    float v = ldf(yr + i);
    if (order == GO_GATE_THEN_NORM) v *= silu_f(ldf(gr + i));
    q += v * v;
  }
  const float r = scale / sqrtf(warp_sum(q) / part + eps);
  for (int i = lane; i < part; i += 32) {
    const float v = ldf(yr + i) * silu_f(ldf(gr + i));
    stf(orow + i, v * r * (wr != nullptr ? wr[i] : 1.f));
  }
}

}  // namespace

void launch_embed_rows(const void* table, bool f32, const long long* ids, float* out, int rows, int W, int V,
                       cudaStream_t s) {
  if (rows <= 0) return;
  const int th = W >= 256 ? 256 : 64;
  if (f32) embed_rows_kernel<<<rows, th, 0, s>>>((const float*)table, ids, out, W, V);
  else embed_rows_kernel<<<rows, th, 0, s>>>((const __nv_bfloat16*)table, ids, out, W, V);
  check_launch("embed_rows");
}

void launch_norm_rows(const float* x, const float* w, void* y, bool f32, int rows, int W, float eps, int kind,
                      cudaStream_t s) {
  if (rows <= 0) return;
  const size_t sm = (size_t)W * 4;
  if (W % 4 == 0 && W <= 4096) {
    auto warp = [&](auto* out, auto tag) {
      using T = std::remove_pointer_t<decltype(out)>;
      norm_warp_kernel<T, decltype(tag)::value><<<(rows + 3) / 4, 128, 0, s>>>(x, w, out, rows, W, eps, kind);
    };
    auto pick = [&](auto* out) {
      if (W <= 512) warp(out, std::integral_constant<int, 4>());
      else if (W <= 1024) warp(out, std::integral_constant<int, 8>());
      else if (W <= 2048) warp(out, std::integral_constant<int, 16>());
      else if (W <= 3072) warp(out, std::integral_constant<int, 24>());
      else warp(out, std::integral_constant<int, 32>());
    };
    if (f32) pick((float*)y);
    else pick((__nv_bfloat16*)y);
    check_launch("norm_rows");
    return;
  }
  if (sm > 160 * 1024) throw std::runtime_error("norm_rows: rows of at most 40960 elements");
  const int th = W >= 2048 ? 256 : 128;
  auto run = [&](auto* kern, auto* out) {
    if (sm > 47 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm);
    kern<<<rows, th, sm, s>>>(x, w, out, W, eps, kind);
  };
  if (f32) run(norm_rows_kernel<float>, (float*)y);
  else run(norm_rows_kernel<__nv_bfloat16>, (__nv_bfloat16*)y);
  check_launch("norm_rows");
}

void launch_add_norm(const AddNormArgs& a, cudaStream_t s) {
  if (a.rows <= 0) return;
  auto go = [&](auto* y, auto* out) {
    using Y = std::remove_pointer_t<decltype(y)>;
    using T = std::remove_pointer_t<decltype(out)>;
    auto vec = [&](auto lanes, auto nv) {
      constexpr int L = decltype(lanes)::value;
      add_norm_vec_kernel<Y, T, L, decltype(nv)::value><<<(a.rows + 128 / L - 1) / (128 / L), 128, 0, s>>>(a);
    };
    using std::integral_constant;
    const auto quad = [](const void* p, int bytes) { return (reinterpret_cast<uintptr_t>(p) & (4 * bytes - 1)) == 0; };
    if (a.W % 4 == 0 && a.ldy % 4 == 0 && a.W <= 8192 && quad(a.x, 4) && quad(a.y, sizeof(Y)) && quad(a.bias, 4) && quad(a.post_w, 4) &&
        quad(a.pre_w, 4) && quad(a.out, sizeof(T))) {
      if (a.W <= 512) vec(integral_constant<int, 32>(), integral_constant<int, 4>());
      else if (a.W <= 1024) vec(integral_constant<int, 32>(), integral_constant<int, 8>());
      else if (a.W <= 2048) vec(integral_constant<int, 128>(), integral_constant<int, 4>());
      else if (a.W <= 4096) vec(integral_constant<int, 128>(), integral_constant<int, 8>());
      else vec(integral_constant<int, 128>(), integral_constant<int, 16>());
      return;
    }
    const size_t sm = (size_t)a.W * 4;
    if (sm > 160 * 1024) throw std::runtime_error("add_norm: rows of at most 40960 elements");
    auto kern = add_norm_kernel<Y, T>;
    if (sm > 47 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm);
    kern<<<a.rows, 256, sm, s>>>(a);
  };
  if (a.y_f32) {
    if (a.out_f32) go((float*)nullptr, (float*)nullptr);
    else go((float*)nullptr, (__nv_bfloat16*)nullptr);
  } else {
    if (a.out_f32) go((__nv_bfloat16*)nullptr, (float*)nullptr);
    else go((__nv_bfloat16*)nullptr, (__nv_bfloat16*)nullptr);
  }
  check_launch("add_norm");
}

void launch_side_rows(const void* gate, long long ldg, const void* table, long long ldt, const long long* ids, int V, int col0,
                      void* out, bool f32, int rows, int dim, int act, cudaStream_t s) {
  const long long n = (long long)rows * dim;
  if (n <= 0) return;
  if (dim % 8 == 0 && col0 % 8 == 0 && n / 8 < (1ll << 31) && vec8_ok(gate, ldg, f32) && vec8_ok(table, ldt, f32) && vec8_ok(out, dim, f32)) {
    const int pieces = (int)(n / 8);
    auto go = [&](auto* o) {
      using T = std::remove_pointer_t<decltype(o)>;
      side_rows_vec_kernel<T><<<(pieces + 255) / 256, 256, 0, s>>>((const T*)gate, ldg, (const T*)table, ldt, ids, V, col0, o, dim / 8, pieces, act);
    };
    if (f32) go((float*)out);
    else go((__nv_bfloat16*)out);
    check_launch("side_rows");
    return;
  }
  const int blocks = (int)((n + 255) / 256 < 148 * 16 ? (n + 255) / 256 : 148 * 16);
  if (f32) side_rows_kernel<<<blocks, 256, 0, s>>>((const float*)gate, ldg, (const float*)table, ldt, ids, V, col0, (float*)out, dim, n, act);
  else
    side_rows_kernel<<<blocks, 256, 0, s>>>((const __nv_bfloat16*)gate, ldg, (const __nv_bfloat16*)table, ldt, ids, V, col0, (__nv_bfloat16*)out,
                                            dim, n, act);
  check_launch("side_rows");
}

void launch_rotation_rows(const double* freqs, int n, float amplitude, float* out, int T, Pos pos, cudaStream_t s) {
  const long long total = (long long)T * n;
  if (total <= 0) return;
  rotation_rows_kernel<<<(unsigned)((total + 255) / 256), 256, 0, s>>>(freqs, n, amplitude, out, total, pos);
  check_launch("rotation_rows");
}

void launch_glu_rows(const void* gu, long long ld, void* out, long long ldo, bool f32, int rows, int F, const GluArgs& glu,
                     cudaStream_t s) {
  const long long n = (long long)rows * F;
  if (n <= 0) return;
  const int blocks = (int)((n + 255) / 256 < 148 * 16 ? (n + 255) / 256 : 148 * 16);
  if (f32) glu_rows_kernel<<<blocks, 256, 0, s>>>((const float*)gu, ld, (float*)out, ldo, F, n, glu);
  else glu_rows_kernel<<<blocks, 256, 0, s>>>((const __nv_bfloat16*)gu, ld, (__nv_bfloat16*)out, ldo, F, n, glu);
  check_launch("glu_rows");
}

void launch_gated_norm(const void* y, long long ldy, const void* gate, long long ldg, const float* w, int w_period,
                       void* out, long long ldo, bool f32, int rows, int inner, int groups, float eps, int order,
                       float scale, cudaStream_t s) {
  if (rows <= 0) return;
  const long long parts = (long long)rows * groups;
  const int part = inner / groups;
  if (part % 8 == 0 && part <= 8192 && vec8_ok(y, ldy, f32) && vec8_ok(gate, ldg, f32) && vec8_ok(out, ldo, f32) &&
      vec8_ok(w, 4, true) && (w == nullptr || w_period % 8 == 0)) {
    auto vec = [&](auto* yy, auto lanes, auto nv) {
      using T = std::remove_const_t<std::remove_pointer_t<decltype(yy)>>;
      constexpr int L = decltype(lanes)::value, NV = decltype(nv)::value;
      const unsigned b = (unsigned)((parts + 128 / L - 1) / (128 / L));
      gated_norm_vec_kernel<T, L, NV><<<b, 128, 0, s>>>((const T*)y, ldy, (const T*)gate, ldg, w, w_period, (T*)out, ldo, parts,
                                                        groups, part, eps, order, scale);
    };
    using std::integral_constant;
    auto pick = [&](auto* yy) {
      if (part <= 64) vec(yy, integral_constant<int, 8>(), integral_constant<int, 1>());
      else if (part <= 128) vec(yy, integral_constant<int, 16>(), integral_constant<int, 1>());
      else if (part <= 256) vec(yy, integral_constant<int, 32>(), integral_constant<int, 1>());
      else if (part <= 512) vec(yy, integral_constant<int, 32>(), integral_constant<int, 2>());
      else if (part <= 1024) vec(yy, integral_constant<int, 128>(), integral_constant<int, 1>());
      else if (part <= 2048) vec(yy, integral_constant<int, 128>(), integral_constant<int, 2>());
      else if (part <= 4096) vec(yy, integral_constant<int, 128>(), integral_constant<int, 4>());
      else vec(yy, integral_constant<int, 128>(), integral_constant<int, 8>());
    };
    if (f32) pick((const float*)y);
    else pick((const __nv_bfloat16*)y);
    check_launch("gated_norm");
    return;
  }
  const int blocks = (int)((parts + 3) / 4);
  if (f32)
    gated_norm_kernel<<<blocks, 128, 0, s>>>((const float*)y, ldy, (const float*)gate, ldg, w, w_period, (float*)out, ldo,
                                             parts, groups, inner / groups, eps, order, scale);
  else
    gated_norm_kernel<<<blocks, 128, 0, s>>>((const __nv_bfloat16*)y, ldy, (const __nv_bfloat16*)gate, ldg, w, w_period,
                                             (__nv_bfloat16*)out, ldo, parts, groups, inner / groups, eps, order, scale);
  check_launch("gated_norm");
}

}  // namespace tb
