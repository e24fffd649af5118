// Short causal convolution over time per channel, followed by silu, with its last inputs carried as a ring.
#include "hybrid.cuh"

namespace tb {
namespace {

constexpr int CONV_SEG = 32;  // tokens per thread

// grid: (ceil(C / 128), ceil(T / CONV_SEG), B); a thread walks one channel over a segment with its taps in registers
template <class T, int TAPS>
__global__ void conv_kernel(const T* __restrict__ u, long long ldu, const float* __restrict__ w,
                            const float* __restrict__ bias, const float* __restrict__ ring, T* __restrict__ out,
                            long long ldo, int Tn, int C, int taps_rt, Pos pos) {
  const int taps = TAPS > 0 ? TAPS : taps_rt;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= C) return;
  const int b = blockIdx.z, t0 = blockIdx.y * CONV_SEG, t1 = min(t0 + CONV_SEG, Tn);
  const long long p0 = pos_of(pos);
  const T* ub = u + (long long)b * Tn * ldu + c;
  T* ob = out + (long long)b * Tn * ldo + c;
  const float* rb = ring + (long long)b * taps * C + c;
  const float bb = bias != nullptr ? bias[c] : 0.f;
  auto input = [&](int t) -> float {  // input of token t of this call; earlier positions come from the ring
    if (t >= 0) return ldf(ub + (long long)t * ldu);
    const long long p = p0 + t;
    return p >= 0 ? rb[(long long)(p % taps) * C] : 0.f;
  };
  if constexpr (TAPS > 0) {
    float wr[TAPS], xr[TAPS];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) wr[j] = w[(long long)c * TAPS + j];
#pragma unroll
    for (int j = 1; j < TAPS; ++j) xr[j] = input(t0 - TAPS + j);
#pragma unroll 4
    for (int t = t0; t < t1; ++t) {
#pragma unroll
      for (int j = 1; j < TAPS; ++j) xr[j - 1] = xr[j];
      xr[TAPS - 1] = ldf(ub + (long long)t * ldu);
      float acc = bb;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) acc += wr[j] * xr[j];
      stf(ob + (long long)t * ldo, silu_f(acc));
    }
  } else {
    for (int t = t0; t < t1; ++t) {
      float acc = bb;
      for (int j = 0; j < taps; ++j) acc += w[(long long)c * taps + j] * input(t - taps + 1 + j);
      stf(ob + (long long)t * ldo, silu_f(acc));
    }
  }
}

// Four taps, eight channels per thread: grid (ceil(C / 8 / 64), ceil(T / CONV_SEG), B), all rows 16-byte aligned.
template <class T, int TAPS>
__global__ void __launch_bounds__(64) conv_vec_kernel(const T* __restrict__ u, long long ldu, const float* __restrict__ w,
                                                      const float* __restrict__ bias, const float* __restrict__ ring,
                                                      T* __restrict__ out, long long ldo, int Tn, int C, Pos pos) {
  const int c = (blockIdx.x * 64 + threadIdx.x) * 8;
  if (c >= C) return;
  const int b = blockIdx.z, t0 = blockIdx.y * CONV_SEG, t1 = min(t0 + CONV_SEG, Tn);
  const long long p0 = pos_of(pos);
  const T* ub = u + (long long)b * Tn * ldu + c;
  T* ob = out + (long long)b * Tn * ldo + c;
  float wr[TAPS][8], bb[8], x[TAPS][8];
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    bb[i] = bias != nullptr ? bias[c + i] : 0.f;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) wr[j][i] = w[(long long)(c + i) * TAPS + j];
  }
#pragma unroll
  for (int j = 1; j < TAPS; ++j) {
    const int t = t0 - TAPS + j;
    const long long p = p0 + t;
    if (t >= 0) ld8v(ub + (long long)t * ldu, x[j]);
    else if (p >= 0) ld8v(ring + ((long long)b * TAPS + p % TAPS) * C + c, x[j]);
    else
#pragma unroll
      for (int i = 0; i < 8; ++i) x[j][i] = 0.f;
  }
#pragma unroll 4
  for (int t = t0; t < t1; ++t) {
#pragma unroll
    for (int j = 1; j < TAPS; ++j)
#pragma unroll
      for (int i = 0; i < 8; ++i) x[j - 1][i] = x[j][i];
    ld8v(ub + (long long)t * ldu, x[TAPS - 1]);
    float o[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      float acc = bb[i];
#pragma unroll
      for (int j = 0; j < TAPS; ++j) acc += wr[j][i] * x[j][i];
      o[i] = silu_for<T>(acc);
    }
    st8v(ob + (long long)t * ldo, o);
  }
}

template <class T>
__global__ void conv_ring_kernel(const T* __restrict__ u, long long ldu, const float* __restrict__ ring_in,
                                 float* __restrict__ ring_out, int Tn, int C, int taps, Pos pos) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= C) return;
  const int slot = blockIdx.y, b = blockIdx.z;
  const long long p0 = pos_of(pos), last = p0 + Tn - 1;
  const long long p = last - (((last - slot) % taps) + taps) % taps;  // newest position kept in this slot
  const long long at = ((long long)b * taps + slot) * C + c;
  ring_out[at] = p >= p0 ? ldf(u + ((long long)b * Tn + (p - p0)) * ldu + c) : ring_in[at];
}

template <class T>
void conv_typed(const T* u, long long ldu, const float* w, const float* bias, const float* ring_in, float* ring_out,
                T* out, long long ldo, int B, int Tn, int C, int taps, Pos pos, cudaStream_t s) {
  dim3 grid((C + 127) / 128, (Tn + CONV_SEG - 1) / CONV_SEG, B);
  const bool f32 = sizeof(T) == 4;
  if (taps == 4 && C % 8 == 0 && vec8_ok(u, ldu, f32) && vec8_ok(out, ldo, f32) && vec8_ok(ring_in, 4, true))
    conv_vec_kernel<T, 4><<<dim3((C / 8 + 63) / 64, (Tn + CONV_SEG - 1) / CONV_SEG, B), 64, 0, s>>>(u, ldu, w, bias, ring_in, out, ldo,
                                                                                                    Tn, C, pos);
  else if (taps == 4) conv_kernel<T, 4><<<grid, 128, 0, s>>>(u, ldu, w, bias, ring_in, out, ldo, Tn, C, taps, pos);
  else if (taps == 3) conv_kernel<T, 3><<<grid, 128, 0, s>>>(u, ldu, w, bias, ring_in, out, ldo, Tn, C, taps, pos);
  else if (taps == 2) conv_kernel<T, 2><<<grid, 128, 0, s>>>(u, ldu, w, bias, ring_in, out, ldo, Tn, C, taps, pos);
  else conv_kernel<T, 0><<<grid, 128, 0, s>>>(u, ldu, w, bias, ring_in, out, ldo, Tn, C, taps, pos);
  conv_ring_kernel<<<dim3((C + 127) / 128, taps, B), 128, 0, s>>>(u, ldu, ring_in, ring_out, Tn, C, taps, pos);
}

}  // namespace

void launch_causal_conv(const void* u, long long ldu, const float* w, const float* bias, const float* ring_in,
                        float* ring_out, void* out, long long ldo, bool f32, int B, int T, int C, int taps, Pos pos,
                        cudaStream_t s) {
  if (B <= 0 || T <= 0) return;
  if (ring_in == ring_out) throw std::runtime_error("causal_conv: the new ring must not alias the old one");
  if (f32) conv_typed((const float*)u, ldu, w, bias, ring_in, ring_out, (float*)out, ldo, B, T, C, taps, pos, s);
  else
    conv_typed((const __nv_bfloat16*)u, ldu, w, bias, ring_in, ring_out, (__nv_bfloat16*)out, ldo, B, T, C, taps, pos, s);
  check_launch("causal_conv");
}

}  // namespace tb
