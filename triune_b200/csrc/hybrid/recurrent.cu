// Token recurrence of the matrix-state mixers (Mamba-2, gated delta rule and retention), exact in fp32, any number of tokens.
//
// The columns of a head's Dk x Dv state are independent given the head's keys, queries and scalars, so a head is cut
// into slices of 16 columns and every slice is a block of four warps. A warp owns four columns; eight lanes share a
// column and each keeps Dk / 8 of its rows in registers. Both contractions of a token act on the state BEFORE it:
//   S_new = g S + k u^T   =>   S_new^T q = g S^T q + (k . q) u
// so a token costs one pass over the registers and one 8-lane reduction. Tokens are staged 16 at a time: a warp loads
// a token's key and query, makes them unit vectors or turns them where the rule asks for it, and leaves fp32 rows, k . q and the
// scalars (g, beta or dt) in shared memory.
#include "hybrid.cuh"

namespace tb {
namespace {

constexpr int RB_TOK = 16, RB_COLS = 16, RB_WARPS = 4;

template <class T, int R>  // R rows per lane: 8 R >= Dk
__global__ void __launch_bounds__(RB_WARPS * 32) recurrent_kernel(const RecurrentArgs p) {
  constexpr int DK = 8 * R;
  __shared__ float sk[RB_TOK][DK + 8], sq[RB_TOK][DK + 8], sv[RB_TOK][RB_COLS];
  __shared__ float sg[RB_TOK], sb[RB_TOK], skq[RB_TOK];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, sub = lane & 7;
  const int slices = (p.Dv + RB_COLS - 1) / RB_COLS;
  const int slice = blockIdx.x % slices, bh = blockIdx.x / slices, h = bh % p.H, b = bh / p.H;
  const int col = slice * RB_COLS + warp * 4 + (lane >> 3);
  const int kh = h / (p.H / p.KG);
  const bool live = col < p.Dv;
  float* st = p.state + (long long)bh * p.Dk * p.Dv;
  // lane `sub` of a column owns rows sub*4 + 32*j + {0..3}: its shared-memory reads are 16-byte and conflict-free
  float S[R];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int d = (r >> 2) * 32 + sub * 4 + (r & 3);
    S[r] = live && d < p.Dk ? st[(long long)d * p.Dv + col] : 0.f;
  }
  const T *Q = (const T*)p.q + (long long)b * p.rows * p.ldq + kh * p.Dk, *K = (const T*)p.k + (long long)b * p.rows * p.ldk + kh * p.Dk;
  const T* V = (const T*)p.v + (long long)b * p.rows * p.ldv + h * p.Dv;
  const bool turn = p.kind == RK_RETENTION;
  const T* A = turn ? nullptr : (const T*)p.a + (long long)b * p.rows * p.lda + h;
  const T* Bt = p.kind == RK_DELTA ? (const T*)p.b + (long long)b * p.rows * p.ldb + h : nullptr;
  T* O = (T*)p.out + (long long)b * p.rows * p.ldo + h * p.Dv;
  const float ea = turn ? 0.f : expf(p.A_log[h]), bias = turn ? 0.f : p.dt_bias[h], Dh = p.kind == RK_MAMBA2 ? p.D[h] : 0.f;
  const float fixed = turn ? (float)p.decay[h] : 0.f, ks = turn ? 1.f / sqrtf((float)p.Dk) : 1.f;
  const int half = p.rot_dims / 2;
  const float qs = p.kind == RK_DELTA ? 1.f / sqrtf((float)p.Dk) : 1.f;

  for (int t0 = 0; t0 < p.T; t0 += RB_TOK) {
    const int n = min(RB_TOK, p.T - t0);
    __syncthreads();
    for (int i = warp; i < n; i += RB_WARPS) {
      const long long t = t0 + i;
      float kk = 0.f, qq = 0.f, kq = 0.f;
      for (int d = lane; d < DK; d += 32) {
        float kv = d < p.Dk ? ldf(K + t * p.ldk + d) : 0.f, qv = d < p.Dk ? ldf(Q + t * p.ldq + d) : 0.f;
        if (turn && d < p.rot_dims) {
          const int i = d < half ? d : d - half, o = d < half ? d + half : d - half;
          const float c = p.rot[t * p.rot_dims + i], s = d < half ? -p.rot[t * p.rot_dims + half + i] : p.rot[t * p.rot_dims + half + i];
          kv = kv * c + ldf(K + t * p.ldk + o) * s;
          qv = qv * c + ldf(Q + t * p.ldq + o) * s;
        }
        kv *= ks;
        sk[i][d] = kv;
        sq[i][d] = qv;
        kk += kv * kv;
        qq += qv * qv;
        kq += kv * qv;
      }
      kq = warp_sum(kq);
      if (p.kind == RK_DELTA) {
        const float rk = 1.f / sqrtf(warp_sum(kk) + p.unit_eps), rq = qs / sqrtf(warp_sum(qq) + p.unit_eps);
        for (int d = lane; d < DK; d += 32) {
          sk[i][d] *= rk;
          sq[i][d] *= rq;
        }
        kq *= rk * rq;
      }
      if (lane < RB_COLS) sv[i][lane] = slice * RB_COLS + lane < p.Dv ? ldf(V + t * p.ldv + slice * RB_COLS + lane) : 0.f;
      if (lane == 0) {
        const float dt = turn ? 1.f : softplus_f(ldf(A + t * p.lda) + bias);
        sg[i] = turn ? fixed : expf(-ea * dt);
        sb[i] = p.kind == RK_DELTA ? sigmoid_f(ldf(Bt + t * p.ldb)) : dt;
        skq[i] = kq;
      }
    }
    __syncthreads();
    for (int i = 0; i < n; ++i) {
      const float g = sg[i], bt = sb[i], v = sv[i][warp * 4 + (lane >> 3)];
      float ak = 0.f, aq = 0.f;
      float kr[R];
#pragma unroll
      for (int j = 0; j < R / 4; ++j) {
        const float4 k4 = *reinterpret_cast<const float4*>(&sk[i][j * 32 + sub * 4]);
        const float4 q4 = *reinterpret_cast<const float4*>(&sq[i][j * 32 + sub * 4]);
        kr[4 * j] = k4.x; kr[4 * j + 1] = k4.y; kr[4 * j + 2] = k4.z; kr[4 * j + 3] = k4.w;
        ak += k4.x * S[4 * j] + k4.y * S[4 * j + 1] + k4.z * S[4 * j + 2] + k4.w * S[4 * j + 3];
        aq += q4.x * S[4 * j] + q4.y * S[4 * j + 1] + q4.z * S[4 * j + 2] + q4.w * S[4 * j + 3];
      }
#pragma unroll
      for (int o = 4; o > 0; o >>= 1) {
        aq += __shfl_xor_sync(0xffffffffu, aq, o);
        ak += __shfl_xor_sync(0xffffffffu, ak, o);
      }
      const float u = p.kind == RK_DELTA ? bt * (v - g * ak) : bt * v;
#pragma unroll
      for (int r = 0; r < R; ++r) S[r] = g * S[r] + kr[r] * u;
      if (sub == 0 && live) stf(O + (t0 + i) * p.ldo + col, g * aq + skq[i] * u + Dh * v);
    }
  }
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int d = (r >> 2) * 32 + sub * 4 + (r & 3);
    if (live && d < p.Dk) st[(long long)d * p.Dv + col] = S[r];
  }
}

template <class T>
void run(const RecurrentArgs& a, cudaStream_t s) {
  const int blocks = a.B * a.H * ((a.Dv + RB_COLS - 1) / RB_COLS);
  if (a.Dk <= 32) recurrent_kernel<T, 4><<<blocks, RB_WARPS * 32, 0, s>>>(a);
  else if (a.Dk <= 64) recurrent_kernel<T, 8><<<blocks, RB_WARPS * 32, 0, s>>>(a);
  else if (a.Dk <= 128) recurrent_kernel<T, 16><<<blocks, RB_WARPS * 32, 0, s>>>(a);
  else if (a.Dk <= 256) recurrent_kernel<T, 32><<<blocks, RB_WARPS * 32, 0, s>>>(a);
  else throw std::runtime_error("recurrent: key dimensions up to 256");
}

}  // namespace

void launch_recurrent(const RecurrentArgs& a, cudaStream_t s) {
  if (a.B <= 0 || a.T <= 0) return;
  if (a.H % a.KG != 0) throw std::runtime_error("recurrent: heads must be a multiple of the key groups");
  if (a.f32) run<float>(a, s);
  else run<__nv_bfloat16>(a, s);
  check_launch("recurrent");
}

}  // namespace tb
