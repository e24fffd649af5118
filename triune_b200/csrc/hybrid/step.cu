// Decoding: one token per sequence. A layer is a handful of launches that each read their weights or state once:
// a matrix-vector product whose prologue forms its input (norm of the residual, gated norm of a mixer's output) and
// whose epilogue adds into the residual or applies the gated activation, and one launch for the mixer itself.
#include "../common/ptx.cuh"
#include "hybrid.cuh"
#include "step_common.cuh"

namespace tb {
namespace {

constexpr int GV_WARPS = 8;

// Sum over the `nt` threads that work on one input row: a warp or the whole block. One barrier per sum: the warps' partial
// sums are read by everyone, from alternating halves of `red`.
__device__ __forceinline__ float row_sum(float v, int nt, float* red, int& phase) {
  v = warp_sum(v);
  if (nt == 32) return v;
  float* r = red + (phase & 1) * GV_WARPS;
  ++phase;
  if ((threadIdx.x & 31) == 0) r[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < GV_WARPS; ++i) t += r[i];
  return t;
}
template <bool EXACT>
__device__ __forceinline__ float silu_step(float x) {
  if constexpr (EXACT) return silu_f(x);
  else return __fdividef(x, 1.f + __expf(-x));
}

// One segment of input row b by nt threads (tid among them), vectors of four where the layout allows.
template <bool EXACT, int V>
__device__ void segment_row(const GemvSegment& g, int b, float* dst, float* red, int& phase, int tid, int nt) {
  const float *x = g.x + (long long)b * g.ld, *gt = g.gate + (long long)b * g.ldg;
  const int part = g.n / g.groups, step = nt * V;
  auto each = [&](const float* p, int i, float (&f)[V]) {
    if constexpr (V == 4) {
      const float4 t = *reinterpret_cast<const float4*>(p + i);
      f[0] = t.x; f[1] = t.y; f[2] = t.z; f[3] = t.w;
    } else {
      f[0] = p[i];
    }
  };
  auto put = [&](int i, const float (&f)[V]) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(dst + i) = make_float4(f[0], f[1], f[2], f[3]);
    else dst[i] = f[0];
  };
  // norm of the row in dst (its sum is s when that is needed), times weight and scale, in place
  auto norm_row = [&](int kind, float s, const float* wt, float eps, float scale, auto&& use) {
    const float mean = kind == HN_LAYER ? row_sum(s, nt, red, phase) / g.n : 0.f;
    float q = 0.f;
    for (int i = tid * V; i < g.n; i += step) {
      float f[V];
      each(dst, i, f);  // written by this thread
#pragma unroll
      for (int e = 0; e < V; ++e) q += (f[e] - mean) * (f[e] - mean);
    }
    const float r = scale / sqrtf(row_sum(q, nt, red, phase) / g.n + eps);
#pragma unroll 2
    for (int i = tid * V; i < g.n; i += step) {
      float f[V], w[V];
      each(dst, i, f);
      each(wt, i, w);
#pragma unroll
      for (int e = 0; e < V; ++e) f[e] = (f[e] - mean) * r * w[e];
      use(i, f);
      put(i, f);
    }
  };
  const auto nothing = [](int, float (&)[V]) {};
  if (g.kind == 0) {
#pragma unroll 2
    for (int i = tid * V; i < g.n; i += step) {
      float f[V];
      each(x, i, f);
#pragma unroll
      for (int e = 0; e < V; ++e) f[e] *= g.scale;
      put(i, f);
    }
  } else if (g.kind == 1) {
    float s = 0.f;
#pragma unroll 2
    for (int i = tid * V; i < g.n; i += step) {
      float f[V];
      each(x, i, f);
#pragma unroll
      for (int e = 0; e < V; ++e) s += f[e];
      put(i, f);
    }
    norm_row(g.norm_kind, s, g.w, g.eps, g.scale, nothing);
  } else if (g.kind == 3) {
    const float* y = g.y + (long long)b * g.ldy;
    float s = 0.f, total = 0.f;
#pragma unroll 2
    for (int i = tid * V; i < g.n; i += step) {
      float f[V], a[V];
      each(y, i, f);
      if (g.y_bias != nullptr) {
        each(g.y_bias, i, a);
#pragma unroll
        for (int e = 0; e < V; ++e) f[e] += a[e];
      }
#pragma unroll
      for (int e = 0; e < V; ++e) s += f[e];
      put(i, f);
    }
    // every block forms the sum for itself; the first one leaves it for the kernels behind
    float* keep = blockIdx.x == 0 && g.x_out != nullptr ? g.x_out + (long long)b * g.n : nullptr;
    norm_row(g.post_kind, s, g.post_w, g.post_eps, 1.f, [&](int i, float (&f)[V]) {
      float a[V];
      each(x, i, a);
#pragma unroll
      for (int e = 0; e < V; ++e) {
        f[e] += a[e];
        total += f[e];
        if (keep != nullptr) keep[i + e] = f[e];
      }
    });
    if (g.w != nullptr) norm_row(g.norm_kind, total, g.w, g.eps, g.scale, nothing);
  } else {
    // wide parts: all threads of the row on one part at a time; narrow parts: a warp per part
    const bool wide = part > 512 || nt == 32;
    const int lane = threadIdx.x & 31, t0 = wide ? tid : lane, ts = (wide ? nt : 32) * V;
    for (int p = wide ? 0 : tid >> 5; p < g.groups; p += wide ? 1 : nt >> 5) {
      float q = 0.f;
#pragma unroll 2
      for (int i = t0 * V; i < part; i += ts) {
        const int c = p * part + i;
        float f[V], z[V], w[V];
        each(x, c, f);
        each(gt, c, z);
        if (g.w != nullptr) {
          each(g.w, g.w_period == g.n ? c : i, w);  // one weight per channel, or one part's weights for every part
        } else {
#pragma unroll
          for (int e = 0; e < V; ++e) w[e] = 1.f;
        }
#pragma unroll
        for (int e = 0; e < V; ++e) {
          const float a = silu_step<EXACT>(z[e]), in = g.norm_kind == GO_GATE_THEN_NORM ? f[e] * a : f[e];
          q += in * in;
          f[e] *= a * w[e];
        }
        put(c, f);
      }
      const float r = g.scale / sqrtf((wide ? row_sum(q, nt, red, phase) : warp_sum(q)) / part + g.eps);
      for (int i = t0 * V; i < part; i += ts) {
        float f[V];
        each(dst, p * part + i, f);
#pragma unroll
        for (int e = 0; e < V; ++e) f[e] *= r;
        put(p * part + i, f);
      }
    }
  }
}

template <bool EXACT>
__device__ __forceinline__ void gemv_segment(const GemvSegment& g, int b, float* dst, float* red, int& phase, int tid, int nt) {
  const bool quad = ((g.n | (int)g.ld | (g.n / g.groups) | g.w_period) & 3) == 0 && (g.kind != 2 || (g.ldg & 3) == 0) && (g.kind != 3 || (g.ldy & 3) == 0) &&
                    ((reinterpret_cast<uintptr_t>(g.x) | reinterpret_cast<uintptr_t>(g.w) | reinterpret_cast<uintptr_t>(g.gate) |
                      reinterpret_cast<uintptr_t>(g.y) | reinterpret_cast<uintptr_t>(g.y_bias) | reinterpret_cast<uintptr_t>(g.post_w) |
                      reinterpret_cast<uintptr_t>(dst)) & 15) == 0;
  if (quad) segment_row<EXACT, 4>(g, b, dst, red, phase, tid, nt);
  else segment_row<EXACT, 1>(g, b, dst, red, phase, tid, nt);
}

// A warp works on two rows at a time (for the gated epilogue: a gate row and its up row).
template <class T, int NB>
__global__ void __launch_bounds__(GV_WARPS * 32, 2) gemv_kernel(const GemvArgs p) {
  extern __shared__ __align__(16) float sx[];  // [NB][KP]
  __shared__ float red[2 * GV_WARPS];
  constexpr int VEC = 16 / sizeof(T), STEP = 32 * VEC, PRE = 4;
  const int KP = (p.K + 3) & ~3;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bool glu = p.epilogue == 2;
  const int pairs = glu ? p.N : (p.N + 1) / 2;
  const bool vec = p.K % VEC == 0 && p.ldw % VEC == 0 && (reinterpret_cast<uintptr_t>(p.W) & 15) == 0;
  auto rows = [&](int pr, const T*& w0, const T*& w1) {
    const int r0 = glu ? pr : 2 * pr, r1 = glu ? pr + p.N : 2 * pr + 1;
    w0 = (const T*)p.W + (long long)r0 * p.ldw;
    w1 = glu || r1 < p.N ? (const T*)p.W + (long long)r1 * p.ldw : w0;
  };
  // The first weights of a pair of rows are fetched ahead: before the previous kernel has finished (weights do not
  // depend on it) and before the prologue, then behind the sums of the pair before.
  uint4 pre0[PRE], pre1[PRE];
  auto fetch = [&](int pr) {
    if (!vec || pr >= pairs) return;
    const T *w0, *w1;
    rows(pr, w0, w1);
#pragma unroll
    for (int i = 0; i < PRE; ++i) {
      const int k = lane * VEC + i * STEP;
      if (k < p.K) {
        pre0[i] = *reinterpret_cast<const uint4*>(w0 + k);
        pre1[i] = *reinterpret_cast<const uint4*>(w1 + k);
      }
    }
  };
  int pr = blockIdx.x * GV_WARPS + warp;
  fetch(pr);
  launch_dependents();
  wait_for_previous();
  // one row: the whole block forms it; several rows: a warp each
  const int nt = p.B == 1 ? GV_WARPS * 32 : 32;
  int phase = 0;
  for (int b = p.B == 1 ? 0 : warp; b < p.B; b += GV_WARPS) {
    int off = 0;
    for (int i = 0; i < p.nseg; ++i) {
      gemv_segment<sizeof(T) == 4>(p.seg[i], b, sx + b * KP + off, red, phase, p.B == 1 ? (int)threadIdx.x : lane, nt);
      off += p.seg[i].n;
    }
  }
  __syncthreads();
  while (pr < pairs) {
    const T *w0, *w1;
    rows(pr, w0, w1);
    float a0[NB], a1[NB];
#pragma unroll
    for (int b = 0; b < NB; ++b) a0[b] = a1[b] = 0.f;
    auto dot = [&](const float (&f0)[VEC], const float (&f1)[VEC], int k) {
#pragma unroll
      for (int b = 0; b < NB; ++b) {
        if (b < p.B) {
#pragma unroll
          for (int i = 0; i < VEC; i += 4) {
            const float4 x = *reinterpret_cast<const float4*>(sx + b * KP + k + i);
            a0[b] += f0[i] * x.x + f0[i + 1] * x.y + f0[i + 2] * x.z + f0[i + 3] * x.w;
            a1[b] += f1[i] * x.x + f1[i + 1] * x.y + f1[i + 2] * x.z + f1[i + 3] * x.w;
          }
        }
      }
    };
    if (vec) {
#pragma unroll
      for (int i = 0; i < PRE; ++i) {
        const int k = lane * VEC + i * STEP;
        if (k < p.K) {
          float f0[VEC], f1[VEC];
          unpack_vec<T>(pre0[i], f0);
          unpack_vec<T>(pre1[i], f1);
          dot(f0, f1, k);
        }
      }
#pragma unroll 4
      for (int k = lane * VEC + PRE * STEP; k < p.K; k += STEP) {
        float f0[VEC], f1[VEC];
        load_vec(w0 + k, f0);
        load_vec(w1 + k, f1);
        dot(f0, f1, k);
      }
    } else {
      for (int k = lane; k < p.K; k += 32) {
        const float f0 = ldf(w0 + k), f1 = ldf(w1 + k);
#pragma unroll
        for (int b = 0; b < NB; ++b)
          if (b < p.B) {
            a0[b] += f0 * sx[b * KP + k];
            a1[b] += f1 * sx[b * KP + k];
          }
      }
    }
    const int next = pr + gridDim.x * GV_WARPS;
    fetch(next);
    const int r0 = glu ? pr : 2 * pr, r1 = 2 * pr + 1;
    const bool two = r1 < p.N;
#pragma unroll
    for (int b = 0; b < NB; ++b) {
      if (b >= p.B) break;
      const float s0 = warp_sum(a0[b]), s1 = warp_sum(a1[b]);
      if (lane == 0) {
        float* y = p.y + (long long)b * p.ldy;
        const float* bias = p.glu.bias;
        const float b0 = bias != nullptr ? bias[r0] : 0.f, b1 = bias != nullptr && (glu || two) ? bias[glu ? r0 + p.N : r1] : 0.f;
        if (glu) {
          y[r0] = glu_f(s0 + b0, s1 + b1, p.glu.act, p.glu.limit, p.glu.alpha);
        } else if (p.epilogue == 1) {
          y[r0] += s0 + b0;
          if (two) y[r1] += s1 + b1;
        } else if (p.epilogue == 3) {
          const long long id = p.ids[b];
          const bool ok = id >= 0 && id < p.V;
          const T* e = (const T*)p.table + (ok ? id * p.ldt + p.col0 : 0);
          y[r0] = ok ? act_f(s0, p.glu.act) * ldf(e + r0) : 0.f;
          if (two) y[r1] = ok ? act_f(s1, p.glu.act) * ldf(e + r1) : 0.f;
        } else {
          y[r0] = s0 + b0;
          if (two) y[r1] = s1 + b1;
        }
      }
    }
    pr = next;
  }
}

// ------------------------------------------------------------------------------------------------ recurrent step
constexpr int ST_COLS = 16, ST_THREADS = 128;

__device__ float conv_step(const StepRecurrent& p, int b, int c, long long pos, bool write) {
  const float cur = p.proj[(long long)b * p.ld + p.col_u + c];
  float* ring = p.ring + (long long)b * p.taps * p.C + c;
  float acc = p.conv_b != nullptr ? p.conv_b[c] : 0.f;
  const float* w = p.conv_w + (long long)c * p.taps;
  for (int j = 0; j < p.taps - 1; ++j) {
    const long long q = pos - (p.taps - 1) + j;
    if (q >= 0) acc += w[j] * ring[(q % p.taps) * p.C];
  }
  acc += w[p.taps - 1] * cur;
  // the slot of this position last held position pos - taps, which no tap reads any more
  if (write) ring[(pos % p.taps) * p.C] = cur;
  return silu_f(acc);
}

// Channel d of a head's query or key as retention has it: turned with the channel half of the rotated dimensions away.
__device__ __forceinline__ float turned(const StepRecurrent& p, const float* head, int d, long long pos) {
  const float v = head[d];
  if (d >= p.rot_dims) return v;
  const int half = p.rot_dims / 2, i = d < half ? d : d - half;
  float s, c;
  rotation(pos, p.freqs[i], &s, &c);
  s *= p.amplitude;
  c *= p.amplitude;
  return d < half ? v * c - head[d + half] * s : v * c + head[d - half] * s;
}

__device__ void recurrent_step(const StepRecurrent& p, int block, long long pos, float* sm) {
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, sub = lane & 7;
  const int slices = (p.Dv + ST_COLS - 1) / ST_COLS;
  const int slice = block % slices, bh = block / slices, h = bh % p.H, b = bh / p.H;
  const int rep = p.H / p.KG, kh = h / rep;
  const int DP = (p.Dk + 31) & ~31;
  float *sk = sm, *sq = sk + DP, *sv = sq + DP, *red = sv + ST_COLS;
  const bool owner = slice == 0 && h % rep == 0;
  const bool plain = p.kind == RK_RETENTION;
  const float* pr = p.proj + (long long)b * p.ld;
  const float ks = plain ? 1.f / sqrtf((float)p.Dk) : 1.f;
  float kk = 0.f, qq = 0.f, kq = 0.f;
  for (int d = tid; d < DP; d += ST_THREADS) {
    float kv = 0.f, qv = 0.f;
    if (d < p.Dk) {
      kv = plain ? turned(p, pr + p.col_k + kh * p.Dk, d, pos) * ks : conv_step(p, b, p.off_k + kh * p.Dk + d, pos, owner);
      qv = plain ? turned(p, pr + p.col_q + kh * p.Dk, d, pos) : conv_step(p, b, p.off_q + kh * p.Dk + d, pos, owner);
    }
    sk[d] = kv;
    sq[d] = qv;
    kk += kv * kv;
    qq += qv * qv;
    kq += kv * qv;
  }
  if (tid < ST_COLS) {
    const int c = slice * ST_COLS + tid;
    sv[tid] = c >= p.Dv ? 0.f : plain ? pr[p.col_v + h * p.Dv + c] : conv_step(p, b, p.off_v + h * p.Dv + c, pos, true);
  }
  kq = block_sum(kq, red);
  float rk = 1.f, rq = 1.f;
  if (p.kind == RK_DELTA) {
    rk = 1.f / sqrtf(block_sum(kk, red) + p.unit_eps);
    rq = 1.f / (sqrtf(block_sum(qq, red) + p.unit_eps) * sqrtf((float)p.Dk));
  }
  const float dt = plain ? 1.f : softplus_f(pr[p.col_a + h] + p.dt_bias[h]);
  const float g = plain ? (float)p.decay[h] : expf(-expf(p.A_log[h]) * dt);
  const int cl = warp * 4 + (lane >> 3), col = slice * ST_COLS + cl;
  const bool live = col < p.Dv;
  float* st = p.state + (long long)bh * p.Dk * p.Dv;
  float ak = 0.f, aq = 0.f;
  const float v = sv[cl];
  float S[32];
  if (live) {
#pragma unroll
    for (int r = 0; r < 32; ++r) {
      const int d = r * 8 + sub;
      if (d < p.Dk) {
        S[r] = st[(long long)d * p.Dv + col];
        ak += sk[d] * S[r];
        aq += sq[d] * S[r];
      }
    }
  }
#pragma unroll
  for (int o = 4; o > 0; o >>= 1) {
    ak += __shfl_xor_sync(0xffffffffu, ak, o);
    aq += __shfl_xor_sync(0xffffffffu, aq, o);
  }
  const float u = p.kind == RK_DELTA ? sigmoid_f(pr[p.col_b + h]) * (v - g * rk * ak) : dt * v;
  if (live) {
#pragma unroll
    for (int r = 0; r < 32; ++r) {
      const int d = r * 8 + sub;
      if (d < p.Dk) st[(long long)d * p.Dv + col] = g * S[r] + sk[d] * rk * u;
    }
    if (sub == 0)
      p.out[(long long)b * p.ldo + h * p.Dv + col] =
          g * rq * aq + kq * rk * rq * u + (p.kind == RK_MAMBA2 ? p.D[h] * v : 0.f);
  }
}

// ------------------------------------------------------------------------------------------------ attention step
constexpr int AT_KEYS = 256;  // keys whose scores are in shared memory at a time

// Head norm and rotation of one projected head row by a warp; dst fp32 [D].
__device__ void head_row(const float* src, const float* w, float eps, int D, int rot, const float* cs, const float* sn,
                         float* dst, int padded) {
  const int lane = threadIdx.x & 31;
  float ss = 0.f;
  for (int d = lane; d < D; d += 32) ss += src[d] * src[d];
  ss = warp_sum(ss);
  const float r = w != nullptr ? 1.f / sqrtf(ss / D + eps) : 1.f;
  for (int d = lane; d < D; d += 32) {
    float v = src[d] * r * (w != nullptr ? w[d] : 1.f);
    if (d < rot) {
      const int o = d ^ 1, i = d >> 1;
      const float x = src[o] * r * (w != nullptr ? w[o] : 1.f);
      v = (d & 1) ? v * cs[i] + x * sn[i] : v * cs[i] - x * sn[i];
    }
    dst[d] = v;
  }
  for (int d = D + lane; d < padded; d += 32) dst[d] = 0.f;
}

// Keys of split `s` of `splits` over n keys: whole multiples of 32, at least 64 keys per split.
__device__ __forceinline__ void split_range(int n, int splits, int s, int* k0, int* k1) {
  int per = (n + splits - 1) / splits;
  per = max(64, (per + 31) & ~31);
  *k0 = min(n, s * per);
  *k1 = min(n, *k0 + per);
}

template <class T, int RM>
__device__ void attention_step(const StepAttention& p, int block, long long pos, float* sm) {
  constexpr int VEC = 16 / sizeof(T);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int rep = p.H / p.G, chunks = (rep + RM - 1) / RM;
  const int split = block % p.splits, bgc = block / p.splits, hc = bgc % chunks, bg = bgc / chunks, g = bg % p.G, b = bg / p.G;
  const int h0 = g * rep + hc * RM, nh = min(RM, rep - hc * RM);
  const int DP = (p.D + 7) & ~7, half = p.rot_dims / 2;
  const int ES = part_stride(p.E);
  float *sq = sm, *sp = sq + RM * DP, *sred = sp + RM * AT_KEYS, *cs = sred + ST_THREADS * 8, *sn = cs + half, *sk = sn + half,
        *ml = sk + DP, *sacc = ml + 2 * RM;
  int* flag = reinterpret_cast<int*>(sacc);
  if (pos < 0 || pos >= p.cap) return;  // the host reserves the cache before every step
  int k0, k1;
  split_range((int)pos + 1, p.splits, split, &k0, &k1);
  T *K = (T*)p.kc + (long long)bg * p.cap * p.pitch_k, *V = (T*)p.vc + (long long)bg * p.cap * p.pitch_v;
  float* part = p.part + (((long long)b * p.H + h0) * p.splits + split) * ES;
  const long long hstride = (long long)p.splits * ES;
  const float* pr = p.proj + (long long)b * p.ld;

  if (k0 < k1) {
    for (int i = tid; i < half; i += ST_THREADS) rotation(pos, p.freqs[i], sn + i, cs + i);
    __syncthreads();
    for (int r = warp; r < nh; r += 4) head_row(pr + p.col_q + (h0 + r) * p.D, p.q_w, p.eps, p.D, p.rot_dims, cs, sn, sq + r * DP, DP);
    const bool has_new = (int)pos < k1;
    if (has_new) {
      // several head chunks of a group write the same values: the readers below only need their own block's copy
      if (warp == 3) head_row(pr + p.col_k + g * p.D, p.k_w, p.eps, p.D, p.rot_dims, cs, sn, sk, DP);
      for (int i = tid; i < p.pitch_v; i += ST_THREADS) stf(V + pos * p.pitch_v + i, i < p.E ? pr[p.col_v + g * p.E + i] : 0.f);
      __syncthreads();
      for (int i = tid; i < p.pitch_k; i += ST_THREADS) stf(K + pos * p.pitch_k + i, i < p.D ? sk[i] : 0.f);
    }
    if (tid < RM) {
      ml[2 * tid] = -INFINITY;
      ml[2 * tid + 1] = 0.f;
    }
    __syncthreads();
    // value accumulation: a thread owns eight neighbouring value dimensions of a subset of the keys
    const int PC = (p.E + 7) / 8, KS = ST_THREADS / PC;  // value dimensions up to 256: PC <= 32
    float acc[RM][8];
    const int pc = tid % PC, ks = tid / PC;
    const bool vlive = ks < KS;
#pragma unroll
    for (int r = 0; r < RM; ++r)
#pragma unroll
      for (int i = 0; i < 8; ++i) acc[r][i] = 0.f;
    for (int kb = k0; kb < k1; kb += AT_KEYS) {
      const int n = min(AT_KEYS, k1 - kb);
      // scores: four lanes per key, two keys at a time
      for (int j = warp * 8 + (lane >> 2); j < ((n + 31) & ~31); j += 64) {
        float s[2][RM];
#pragma unroll
        for (int r = 0; r < RM; ++r) s[0][r] = s[1][r] = 0.f;
        // keys past the tile repeat its last one; their scores are not kept
        const T *ka = K + (long long)(kb + min(j, n - 1)) * p.pitch_k, *kc = K + (long long)(kb + min(j + 32, n - 1)) * p.pitch_k;
#pragma unroll 4
        for (int d = (lane & 3) * VEC; d < DP; d += 4 * VEC) {
          float fa[VEC], fc[VEC];
          load_vec(ka + d, fa);  // rows are padded with zeros to a multiple of 16 bytes
          load_vec(kc + d, fc);
#pragma unroll
          for (int r = 0; r < RM; ++r)
            if (r < nh) {
#pragma unroll
              for (int i = 0; i < VEC; i += 4) {
                const float4 x = *reinterpret_cast<const float4*>(sq + r * DP + d + i);
                s[0][r] += fa[i] * x.x + fa[i + 1] * x.y + fa[i + 2] * x.z + fa[i + 3] * x.w;
                s[1][r] += fc[i] * x.x + fc[i + 1] * x.y + fc[i + 2] * x.z + fc[i + 3] * x.w;
              }
            }
        }
#pragma unroll
        for (int g2 = 0; g2 < 2; ++g2)
#pragma unroll
          for (int r = 0; r < RM; ++r) {
            float t = s[g2][r];
            t += __shfl_xor_sync(0xffffffffu, t, 1);
            t += __shfl_xor_sync(0xffffffffu, t, 2);
            if ((lane & 3) == 0 && j + 32 * g2 < n && r < nh) sp[r * AT_KEYS + j + 32 * g2] = t * p.scale;
          }
      }
      __syncthreads();
      // softmax of the tile: a warp per head; the running maximum's correction goes through sk
      for (int r = warp; r < nh; r += 4) {
        float m = -INFINITY;
        for (int j = lane; j < n; j += 32) m = fmaxf(m, sp[r * AT_KEYS + j]);
        m = fmaxf(warp_max(m), ml[2 * r]);
        float l = 0.f;
        for (int j = lane; j < n; j += 32) {
          const float e = expf(sp[r * AT_KEYS + j] - m);
          sp[r * AT_KEYS + j] = e;
          l += e;
        }
        l = warp_sum(l);
        if (lane == 0) {
          const float corr = expf(ml[2 * r] - m);
          ml[2 * r + 1] = ml[2 * r + 1] * corr + l;
          ml[2 * r] = m;
          sacc[1 + r] = corr;
        }
      }
      __syncthreads();
      if (vlive) {
#pragma unroll
        for (int r = 0; r < RM; ++r)
          if (r < nh) {
#pragma unroll
            for (int i = 0; i < 8; ++i) acc[r][i] *= sacc[1 + r];
          }
#pragma unroll 4
        for (int j = ks; j < n; j += KS) {
          float v[8];
          ld8v(V + (long long)(kb + j) * p.pitch_v + 8 * pc, v);  // value rows are padded to a multiple of eight
#pragma unroll
          for (int r = 0; r < RM; ++r)
            if (r < nh) {
              const float w = sp[r * AT_KEYS + j];
#pragma unroll
              for (int i = 0; i < 8; ++i) acc[r][i] += w * v[i];
            }
        }
      }
      __syncthreads();
    }
    // sum over the key subsets, one head at a time
#pragma unroll
    for (int r = 0; r < RM; ++r) {
      if (r < nh) {
        if (vlive) {
#pragma unroll
          for (int i = 0; i < 8; ++i) sred[tid * 8 + i] = acc[r][i];
        }
        __syncthreads();
        for (int e = tid; e < p.E; e += ST_THREADS) {
          float t = 0.f;
          for (int q = 0; q < KS; ++q) t += sred[(q * PC + (e >> 3)) * 8 + (e & 7)];
          part[r * hstride + 4 + e] = t;
        }
        if (tid == 0) {
          part[r * hstride] = ml[2 * r];
          part[r * hstride + 1] = ml[2 * r + 1];
        }
        __syncthreads();
      }
    }
  } else {
    if (tid < nh) {
      part[tid * hstride] = -INFINITY;
      part[tid * hstride + 1] = 0.f;
    }
  }
  __threadfence();
  __syncthreads();
  if (tid == 0) *flag = atomicAdd(p.counters + bgc, 1) == p.splits - 1 ? 1 : 0;
  __syncthreads();
  if (*flag == 0) return;
  __threadfence();
  if (tid == 0) p.counters[bgc] = 0;
  const float* base = p.part + ((long long)b * p.H + h0) * p.splits * ES;
  // weights of the splits of every head (a warp per head), then the weighted sum of their partial values
  for (int r = warp; r < nh; r += 4) {
    const float* ph = base + r * hstride;
    const float sink = p.sink != nullptr ? p.sink[h0 + r] : -INFINITY;
    float m = sink;
    for (int s = lane; s < p.splits; s += 32) m = fmaxf(m, __ldcg(ph + s * ES));
    m = warp_max(m);
    float l = 0.f;
    for (int s = lane; s < p.splits; s += 32) {
      const float c = expf(__ldcg(ph + s * ES) - m);
      sp[r * AT_KEYS + s] = c;  // at most 64 splits
      l += __ldcg(ph + s * ES + 1) * c;
    }
    l = warp_sum(l) + (p.sink != nullptr ? expf(sink - m) : 0.f);
    __syncwarp();
    for (int s = lane; s < p.splits; s += 32) sp[r * AT_KEYS + s] *= p.out_scale / l;
  }
  __syncthreads();
  int active = p.splits;  // splits beyond the keys hold nothing
  {
    int a, z;
    split_range((int)pos + 1, p.splits, 0, &a, &z);
    active = min(active, ((int)pos + z) / max(z, 1));
  }
  const int quads = (p.E + 3) / 4;  // partial rows are padded to whole quads
  for (int i = tid; i < nh * quads; i += ST_THREADS) {
    const int r = i / quads, e = (i % quads) * 4;
    const float* ph = base + r * hstride + 4 + e;
    float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 16
    for (int s = 0; s < active; ++s) {
      const float c = sp[r * AT_KEYS + s];
      const float4 v = __ldcg(reinterpret_cast<const float4*>(ph + s * ES));
      t.x += c * v.x; t.y += c * v.y; t.z += c * v.z; t.w += c * v.w;
    }
    float* o = p.out + (long long)b * p.ldo + (h0 + r) * p.E + e;
    o[0] = t.x;
    if (e + 1 < p.E) o[1] = t.y;
    if (e + 2 < p.E) o[2] = t.z;
    if (e + 3 < p.E) o[3] = t.w;
  }
}

template <class T, int RM>
__global__ void __launch_bounds__(ST_THREADS) mixer_step_kernel(const StepArgs p, int att_blocks) {
  extern __shared__ __align__(16) float sm[];
  launch_dependents();
  wait_for_previous();
  const long long pos = pos_of(p.pos);
  if ((int)blockIdx.x < att_blocks) attention_step<T, RM>(p.att, blockIdx.x, pos, sm);
  else recurrent_step(p.rec, blockIdx.x - att_blocks, pos, sm);
}

}  // namespace

int step_part_stride(int E) { return part_stride(E); }
int step_head_chunk(int rep) { return rep <= 1 ? 1 : rep <= 2 ? 2 : rep <= 4 ? 4 : 8; }

void launch_mixer_step(const StepArgs& a, cudaStream_t s) {
  if (a.B <= 0) return;
  int att = 0, rec = 0, rm = 1;
  size_t sm = 0;
  if (a.has_att) {
    const StepAttention& p = a.att;
    if (p.E > 256 || p.D > 512) throw std::runtime_error("mixer_step: head dimensions up to 512 / 256");
    rm = step_head_chunk(p.H / p.G);
    att = a.B * p.G * ((p.H / p.G + rm - 1) / rm) * p.splits;
    const int dp = (p.D + 7) & ~7;
    sm = (size_t)(rm * dp + rm * AT_KEYS + ST_THREADS * 8 + p.rot_dims + 4 + dp + 2 * rm + rm + 4) * 4;
  }
  if (a.has_rec) {
    const StepRecurrent& p = a.rec;
    if (p.Dk > 256) throw std::runtime_error("mixer_step: key dimensions up to 256");
    rec = a.B * p.H * ((p.Dv + ST_COLS - 1) / ST_COLS);
    const size_t need = (size_t)(2 * ((p.Dk + 31) & ~31) + ST_COLS + 40) * 4;
    sm = need > sm ? need : sm;
  }
  if (att + rec == 0) return;
  const bool f32 = a.has_att && a.att.cache_f32;
  auto go = [&](auto* kern) { launch_chained(kern, att + rec, ST_THREADS, sm, s, a, att); };
  if (f32) {
    if (rm == 1) go(mixer_step_kernel<float, 1>);
    else if (rm == 2) go(mixer_step_kernel<float, 2>);
    else if (rm == 4) go(mixer_step_kernel<float, 4>);
    else go(mixer_step_kernel<float, 8>);
  } else {
    if (rm == 1) go(mixer_step_kernel<__nv_bfloat16, 1>);
    else if (rm == 2) go(mixer_step_kernel<__nv_bfloat16, 2>);
    else if (rm == 4) go(mixer_step_kernel<__nv_bfloat16, 4>);
    else go(mixer_step_kernel<__nv_bfloat16, 8>);
  }
  check_launch("mixer_step");
}

void launch_gemv(const GemvArgs& a, cudaStream_t s) {
  if (a.B <= 0 || a.N <= 0) return;
  if (a.B > 8) throw std::runtime_error("gemv: at most 8 rows");
  const size_t sm = (size_t)a.B * ((a.K + 3) & ~3) * 4;
  if (sm > 200 * 1024) throw std::runtime_error("gemv: the input rows do not fit into shared memory");
  const int pairs = a.epilogue == 2 ? a.N : (a.N + 1) / 2;
  int blocks = (pairs + GV_WARPS - 1) / GV_WARPS;
  const int per_sm = sm > 100 * 1024 ? 1 : 2;
  if (blocks > 148 * per_sm) blocks = 148 * per_sm;
  auto go = [&](auto* kern) {
    if (sm > 47 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm);
    launch_chained(kern, blocks, GV_WARPS * 32, sm, s, a);
  };
  if (a.f32) {
    if (a.B == 1) go(gemv_kernel<float, 1>);
    else if (a.B == 2) go(gemv_kernel<float, 2>);
    else if (a.B <= 4) go(gemv_kernel<float, 4>);
    else go(gemv_kernel<float, 8>);
  } else {
    if (a.B == 1) go(gemv_kernel<__nv_bfloat16, 1>);
    else if (a.B == 2) go(gemv_kernel<__nv_bfloat16, 2>);
    else if (a.B <= 4) go(gemv_kernel<__nv_bfloat16, 4>);
    else go(gemv_kernel<__nv_bfloat16, 8>);
  }
  check_launch("gemv");
}

}  // namespace tb
