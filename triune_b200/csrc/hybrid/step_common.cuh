// What the kernels of a decoding step share: 16-byte weight loads, chained launches, the layout of split attention results.
#pragma once
#include "hybrid.cuh"

namespace tb {
namespace {

template <class T>
__device__ __forceinline__ void unpack_vec(const uint4& u, float (&f)[16 / sizeof(T)]) {
  if constexpr (sizeof(T) == 4) {
    f[0] = __uint_as_float(u.x); f[1] = __uint_as_float(u.y); f[2] = __uint_as_float(u.z); f[3] = __uint_as_float(u.w);
  } else {
    const uint32_t a[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      f[2 * i] = __uint_as_float(a[i] << 16);
      f[2 * i + 1] = __uint_as_float(a[i] & 0xffff0000u);
    }
  }
}

template <class T>
__device__ __forceinline__ void load_vec(const T* p, float (&f)[16 / sizeof(T)]) {
  unpack_vec<T>(*reinterpret_cast<const uint4*>(p), f);
}

// Programmatic dependent launch: the step's kernels follow one another closely, so each lets its successor start at once
// and itself waits for its predecessor's results before it touches anything but weights.
__device__ __forceinline__ void launch_dependents() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void wait_for_previous() { asm volatile("griddepcontrol.wait;" ::: "memory"); }

template <class Args, class... Rest>
void launch_chained(void (*kern)(Args, Rest...), int blocks, int threads, size_t smem, cudaStream_t s, const Args& a, Rest... rest) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(blocks);
  cfg.blockDim = dim3(threads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = s;
  cudaLaunchAttribute at[1];
  at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  at[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = at;
  cfg.numAttrs = 1;
  cudaLaunchKernelEx(&cfg, kern, a, rest...);
}

// Floats of one partial result: maximum, sum, two of padding, the values padded to whole quads.
__host__ __device__ constexpr int part_stride(int E) { return ((E + 3) & ~3) + 4; }

}  // namespace
}  // namespace tb
