// Kernels of the heterogeneous-layer family: models whose layers mix softmax attention (per-head query / key norm,
// partial rotation, a sink in the softmax), multi-head latent attention, gated delta rule, Mamba-2 and retention mixers,
// with a 32-bit residual stream.
//
// Every kernel exists for bf16 and for fp32 compute tensors (`f32` flag of the launchers). Sequence rows are laid out
// [B * T, ld]; `pos` is the position of the first of the T tokens, given by value or, when `pos_ptr` is not null, in
// device memory (graph-replayed decoding). Norms, positions, scores, softmax, decays and recurrent states are fp32 in
// both. These translation units are compiled without fast-math: angles reach thousands of radians and the decay
// chain is an exponential of an exponential.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <stdexcept>
#include <string>

namespace tb {

enum HybridNorm : int { HN_LAYER = 0, HN_RMS = 1 };
enum HybridAct : int { HA_RELU = 0, HA_SILU = 1, HA_GELU_TANH = 2, HA_IDENTITY = 3, HA_CLAMPED = 4 };
enum GateOrder : int { GO_GATE_THEN_NORM = 0, GO_NORM_THEN_GATE = 1 };
enum RecurrentKind : int { RK_MAMBA2 = 0, RK_DELTA = 1, RK_RETENTION = 2 };

struct Pos {
  long long host;
  const long long* dev;
};

// ---- rows ------------------------------------------------------------------------------------------------------
// out[row] = table[ids[row]] as fp32; ids outside [0, V) give zero rows.
void launch_embed_rows(const void* table, bool f32, const long long* ids, float* out, int rows, int W, int V,
                       cudaStream_t s);
// y = norm(x) * w over fp32 rows.
void launch_norm_rows(const float* x, const float* w, void* y, bool f32, int rows, int W, float eps, int kind,
                      cudaStream_t s);
// x += post(y + bias), then out = pre(x): the residual sum of a sublayer with a norm behind it, and the next sublayer's
// input, in one pass. bias, out and pre_w may be null: no bias, no output, the sum itself as output.
struct AddNormArgs {
  float* x;
  const void* y;
  long long ldy;
  bool y_f32, out_f32;
  const float *bias, *post_w, *pre_w;
  void* out;
  int rows, W, post_kind, pre_kind;
  float post_eps, pre_eps;
};
void launch_add_norm(const AddNormArgs& a, cudaStream_t s);
// How a gated activation combines gate g and up u (both after their biases): act(g) * u, or for HA_CLAMPED
// g sigmoid(alpha g) (u + 1) with g at most `limit` and u within +- `limit`.
struct GluArgs {
  int act;
  float limit, alpha;
  const float* bias;  // [2 F]: of the gate, then of the up projection; or null
};
// gate at column 0 and up at column F of gu
void launch_glu_rows(const void* gu, long long ld, void* out, long long ldo, bool f32, int rows, int F, const GluArgs& glu,
                     cudaStream_t s);
// out = act(gate) * table[ids[row], col0 ...]
void launch_side_rows(const void* gate, long long ldg, const void* table, long long ldt, const long long* ids, int V, int col0,
                      void* out, bool f32, int rows, int dim, int act, cudaStream_t s);
// [T, 2 n]: cosines, then sines of the turns pos + t times freqs[n], times amplitude
void launch_rotation_rows(const double* freqs, int n, float amplitude, float* out, int T, Pos pos, cudaStream_t s);
// Gated norm of a mixer's output y [rows, inner] with gate rows: parts of inner / groups elements are divided by their
// own root mean square. w has inner entries (w_period = inner), one part's entries repeated (w_period = part), or is null.
void launch_gated_norm(const void* y, long long ldy, const void* gate, long long ldg, const float* w, int w_period,
                       void* out, long long ldo, bool f32, int rows, int inner, int groups, float eps, int order,
                       float scale, cudaStream_t s);

// ---- causal convolution ----------------------------------------------------------------------------------------
// u [B*T, ldu] (C channels), w [C, taps] fp32, bias [C] or null, silu. The state is a ring [B, taps, C] (fp32): slot
// p % taps holds the input of position p. ring_out receives the ring after the last token; it must not alias ring_in.
void launch_causal_conv(const void* u, long long ldu, const float* w, const float* bias, const float* ring_in,
                        float* ring_out, void* out, long long ldo, bool f32, int B, int T, int C, int taps, Pos pos,
                        cudaStream_t s);

// ---- recurrences -----------------------------------------------------------------------------------------------
//   delta:   k, q unit vectors (q also times Dk^-1/2), g = exp(-exp(A_log) softplus(a + dt_bias)), beta = sigmoid(b)
//            u = beta (v - g S^T k)
//   mamba2:  dt = softplus(a + dt_bias), g = exp(-exp(A_log) dt), u = dt v
//   retention: q and k turned by the rows of `rot` (dimension i with i + rot_dims / 2), k times Dk^-1/2, g = decay[h], u = v
//   S <- g S + k u^T,  out = S^T q (+ D v)      (S: Dk x Dv fp32 per head)
struct RecurrentArgs {
  const void *q, *k, *v;             // [B*T, ld*]: head groups of Dk (q, k: KG groups), heads of Dv (v)
  long long ldq, ldk, ldv;
  const void *a, *b;                 // [B*T, ld]: one column per head (b: delta only)
  long long lda, ldb;
  const float *A_log, *dt_bias, *D;  // [H] (D: mamba2 only)
  float* state;                      // [B, H, Dk, Dv], updated in place
  void* out;                         // [B*T, ldo], heads of Dv
  long long ldo;
  int B, T, H, KG, Dk, Dv;
  long long rows;                    // rows between the sequences of a batch (T unless this is a part of longer ones)
  int kind;
  float unit_eps;                    // under the root of the unit norm (delta)
  bool f32;
  const float* rot;                  // retention: [T, rot_dims] cosines and sines of the tokens
  int rot_dims;
  const double* decay;               // retention: [H]
};
void launch_recurrent(const RecurrentArgs& a, cudaStream_t s);
// Chunk-parallel form for prompts (bf16, Dk <= 128); scratch of chunk_scan_scratch(a) bytes, 16-byte aligned.
bool chunk_scan_supported(const RecurrentArgs& a);
long long chunk_scan_scratch(const RecurrentArgs& a);
void launch_chunk_scan(const RecurrentArgs& a, void* scratch, cudaStream_t s);
// Mamba-2 prompts on tcgen05 (aligned bf16, key sizes 65 to 128); `status` (or null) receives a KernelStatus.
bool ssd_tc_supported(const RecurrentArgs& a);
long long ssd_tc_scratch(const RecurrentArgs& a);
void launch_ssd_tc(const RecurrentArgs& a, void* scratch, int* status, cudaStream_t s);
// Retention prompts on tcgen05 (aligned bf16, key sizes up to 128), every chunk of 128 tokens on its own.
bool retention_tc_supported(const RecurrentArgs& a);
long long retention_tc_scratch(const RecurrentArgs& a);
void launch_retention_tc(const RecurrentArgs& a, void* scratch, int* status, cudaStream_t s);
// [nseg, B, H, Dk, Dv] contributions of segments (then [nseg, B, H] decays) -> states before the segments, from a.state
void launch_ssd_scan(const RecurrentArgs& a, float* seg_state, int nseg, cudaStream_t s);

// ---- softmax attention -----------------------------------------------------------------------------------------
// Query / key head norm + rotation; appends k and v to the cache [B, G, cap, pitch*] at positions pos .. pos+T-1 and
// writes q [B, H, T, pitch_k].
struct AttnPrepArgs {
  const void* proj;  // [B*T, ld]: q at col_q (H*D), k at col_k (G*D), v at col_v (G*E)
  long long ld;
  int col_q, col_k, col_v;
  const float *q_w, *k_w;  // [D] or null (no norm)
  float eps;
  int rot_dims;
  const double* freqs;  // [rot_dims / 2], radians per position
  void *q, *kc, *vc;
  int B, T, H, G, D, E, cap, pitch_k, pitch_v;
  Pos pos;
  bool f32;
};
void launch_attn_prep(const AttnPrepArgs& a, cudaStream_t s);

// Element (batch, row, head, d) of an operand is at batch * sb + row * sr + head * sh + d. A key row may have a second part
// (R > 0) that all heads of a sequence share; queries then have it behind their first part, at q2.
struct AttnOperand {
  const void* p;
  long long sr, sh, sb;
};
struct AttnArgs {
  AttnOperand q, k, v, q2, k2;
  const float* sink;        // [H] or null
  const void* gate;         // [B*T, ldg], one column per head: outputs are multiplied by its sigmoid; or null
  long long ldg;
  void* out;                // [B*T, ldo], heads of E
  long long ldo;
  int B, T, H, G, D, E, R, rows;  // rows: key rows per sequence that may be read
  float scale, out_scale;
  Pos pos;
  bool f32;
};
void launch_attn_simple(const AttnArgs& a, cudaStream_t s);
// tcgen05 kernel: bf16, heads up to 128 (plus a second part up to 64), positive scale. `status` (or null) receives a KernelStatus if a wait expires.
bool attn_tc_supported(const AttnArgs& a);
void launch_attn_tc(const AttnArgs& a, int* status, cudaStream_t s);

// ---- latent attention --------------------------------------------------------------------------------------------
// Prompts: turns the second part of every query head in place and, where the layer has latents of its own (col_c >= 0),
// appends their normed form and the turned key part to the cache [B, cap, rank_p + Rp].
struct LatentPrepArgs {
  void* proj;  // [B*T, ld]
  long long ld;
  int col_q, H, Dp, Rp;  // heads of [Dp | Rp]
  int col_c;
  const float* norm_w;   // [rank]
  float eps;
  void* cache;
  int cap, rank, rank_p, R;
  const float* rot;      // [T, R]: cosines, sines
  int B, T;
  Pos pos;
  bool f32;
};
void launch_latent_prep(const LatentPrepArgs& a, cudaStream_t s);

// One token per sequence in the latent space, three launches: (1) qa = [W_uk^T q | turned q part] per head, and the append
// of the new row; (2) attention of qa over the cached rows in split ranges; (3) combination of the splits, value expansion,
// gate.
struct LatentStepArgs {
  const float* proj;  // [B, ld]
  long long ld;
  int col_q, col_g, col_c;  // col_g, col_c: -1 where there is none
  int H, D, Dp, R, Rp, E, Ep, rank, rank_p;
  const float* norm_w;
  float eps;
  void* cache;        // [B, cap, rank_p + Rp]
  const void* up;     // [H, Dp + Ep, rank_p]
  bool f32;           // cache and up
  int cap;
  const double* freqs;  // [R / 2]
  float amplitude;
  const float* sink;
  float* qa;          // [B, H, rank_p + Rp]
  float* part;        // [B, H, splits, step_part_stride(rank_p)]
  int splits;
  float* out;         // [B, ldo], heads of E
  long long ldo;
  float scale, out_scale;
  int B;
  Pos pos;
};
int latent_step_splits(int B, int H);
void launch_latent_step(const LatentStepArgs& a, cudaStream_t s);

// ---- decoding (one token per sequence, B <= 8) ------------------------------------------------------------------
// y[b, n] (+)= sum_k W[n, k] in[b, k] with the input formed in the kernel's prologue from one or two segments:
// plain fp32 rows, norm(x) * w, the gated norm of a mixer output, or norm(x + post(y + bias)) (which also leaves the sum in
// x_out for the kernels behind it). Everything but W is fp32.
struct GemvSegment {
  const float* x;     // [B, ld]
  long long ld;
  int n;              // entries of this segment
  int kind;           // 0 plain, 1 norm over the n entries, 2 gated norm, 3 norm of a sum
  int norm_kind;      // kinds 1, 3: HN_*; kind 2: GO_*
  const float* w;     // norm weight; null: kind 2 has none, kind 3 is the sum itself
  int w_period;
  const float* gate;  // kind 2: [B, ldg]
  long long ldg;
  int groups;
  float eps, scale;
  const float *y, *y_bias, *post_w;  // kind 3: [B, ldy], [n] or null, [n]
  long long ldy;
  int post_kind;
  float post_eps;
  float* x_out;       // kind 3: [B, n] or null
};
struct GemvArgs {
  GemvSegment seg[2];
  int nseg;
  const void* W;  // [N, ldw] bf16 or fp32
  long long ldw;
  bool f32;
  float* y;       // [B, ldy]
  long long ldy;
  int B, N, K;    // K = sum of the segments' entries
  int epilogue;   // 0 store, 1 add, 2 gated activation of rows n and n + N (W has 2 N rows), 3 act(row n) * table entry
  GluArgs glu;    // act of 2 and 3; bias of 0, 1 ([N]) and 2 ([2 N])
  const void* table;     // epilogue 3: [V, ldt] in W's type, row ids[b], column col0 + n
  long long ldt;
  const long long* ids;  // [B]
  int V, col0;
};
void launch_gemv(const GemvArgs& a, cudaStream_t s);

// One step of a mixer: any of a recurrence (short convolution, unit norms and scalars, state update) and an attention
// (head norm, rotation, cache append, split-key softmax and its combination), as blocks of one launch.
struct StepRecurrent {
  const float* proj;  // [B, ld]: conv channels at col_u, a at col_a, b at col_b
  long long ld;
  int col_u, col_a, col_b;
  int off_q, off_k, off_v;         // inside the conv channels
  const float *conv_w, *conv_b;    // [C, taps], [C] or null
  float* ring;                     // [B, taps, C], slot pos % taps is written
  int C, taps;
  const float *A_log, *dt_bias, *D;
  float* state;
  float* out;                      // [B, ldo]
  long long ldo;
  int H, KG, Dk, Dv, kind;
  float unit_eps;
  int col_q, col_k, col_v;         // retention: columns of proj (no convolution)
  const double *decay, *freqs;     // retention: [H], [rot_dims / 2]
  int rot_dims;
  float amplitude;
};
struct StepAttention {
  const float* proj;
  long long ld;
  int col_q, col_k, col_v;
  const float *q_w, *k_w;
  float eps;
  int rot_dims;
  const double* freqs;
  const float* sink;
  void *kc, *vc;
  bool cache_f32;
  int cap, pitch_k, pitch_v;
  float* part;      // [B, H, splits, step_part_stride(E)]
  int* counters;    // [B * G * head chunks], zero between calls
  int splits;
  float* out;       // [B, ldo]
  long long ldo;
  int H, G, D, E;
  float scale, out_scale;
};
struct StepArgs {
  StepRecurrent rec;
  StepAttention att;
  bool has_rec, has_att;
  int B;
  Pos pos;
};
int step_part_stride(int E);
int step_head_chunk(int heads_per_group);  // query heads one attention block serves
void launch_mixer_step(const StepArgs& a, cudaStream_t s);

// ---- device helpers --------------------------------------------------------------------------------------------
#ifdef __CUDACC__
__device__ __forceinline__ float ldf(const float* p) { return *p; }
__device__ __forceinline__ float ldf(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void stf(float* p, float v) { *p = v; }
__device__ __forceinline__ void stf(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ long long pos_of(const Pos& p) { return p.dev != nullptr ? *p.dev : p.host; }
__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
// silu feeding a value that is stored as T: bf16 results take the fast exponential and divide
template <class T>
__device__ __forceinline__ float silu_for(float x) {
  if constexpr (sizeof(T) == 4) return silu_f(x);
  else return __fdividef(x, 1.f + __expf(-x));
}
// eight consecutive values, 16-byte (bf16) or 2 x 16-byte (fp32) accesses
__device__ __forceinline__ void ld8v(const float* p, float (&f)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void ld8v(const __nv_bfloat16* p, float (&f)[8]) {
  const uint4 u = *reinterpret_cast<const uint4*>(p);
  const uint32_t a[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    f[2 * i] = __uint_as_float(a[i] << 16);
    f[2 * i + 1] = __uint_as_float(a[i] & 0xffff0000u);
  }
}
__device__ __forceinline__ void st8v(float* p, const float (&f)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(f[4], f[5], f[6], f[7]);
}
__device__ __forceinline__ void st8v(__nv_bfloat16* p, const float (&f)[8]) {
  uint4 u;
  uint32_t* a = &u.x;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    __nv_bfloat162 t = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
    a[i] = *reinterpret_cast<uint32_t*>(&t);
  }
  *reinterpret_cast<uint4*>(p) = u;
}
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float act_f(float x, int act) {
  if (act == HA_RELU) return fmaxf(x, 0.f);
  if (act == HA_SILU) return silu_f(x);
  if (act == HA_GELU_TANH) return 0.5f * x * (1.f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x)));
  return x;
}
__device__ __forceinline__ float glu_f(float g, float u, int act, float limit, float alpha) {
  if (act != HA_CLAMPED) return act_f(g, act) * u;
  g = fminf(g, limit);
  return g / (1.f + expf(-alpha * g)) * (fminf(fmaxf(u, -limit), limit) + 1.f);
}
// sine and cosine of pos * f radians; the turn count is removed in double so that far positions lose nothing
__device__ __forceinline__ void rotation(long long pos, double f, float* s, float* c) {
  const double a = (double)pos * f;
  sincosf((float)(a - 6.283185307179586 * rint(a * 0.15915494309189535)), s, c);
}
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}
// Sum over a block of up to 32 warps; every thread receives it. `red` holds 33 floats.
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = (blockDim.x + 31) >> 5;
  __syncthreads();
  if (l == 0) red[w] = v;
  __syncthreads();
  if (w == 0) {
    float t = l < nw ? red[l] : 0.f;
    t = warp_sum(t);
    if (l == 0) red[32] = t;
  }
  __syncthreads();
  return red[32];
}
#endif

// rows that 8-wide vector accesses may touch: base and pitch on 16-byte boundaries
inline bool vec8_ok(const void* p, long long ld, bool f32) {
  return (reinterpret_cast<uintptr_t>(p) & 15) == 0 && ld % (f32 ? 4 : 8) == 0;
}
inline void check_launch(const char* what) {
  cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string(what) + " launch failed: " + cudaGetErrorString(e));
}

}  // namespace tb
