// Types shared by the kernels that run on a ragged serving batch (see serve_layers.cu for the batch description).
#pragma once
#include "common.cuh"

namespace apb {

constexpr int kServePage = 16;   // tokens per KV page

struct ServeEntries {
  const int* start;   // first row of the entry
  const int* len;     // rows of the entry (0: nothing to do)
  const int* slot;    // state slot of its sequence
  const int* pos0;    // position of its first row
};

template <typename T>
__device__ __forceinline__ float to_f32(T v);
template <>
__device__ __forceinline__ float to_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ float to_f32<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f32(float v);
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

// ---- norms in equal groups of a row, blocks of 256 threads.  A group's squares are summed by `group_parts` warps, each of which
// leaves a partial sum; with more than 8 groups a warp takes every eighth.
__device__ __forceinline__ int group_parts(int groups) { return groups > 4 ? 1 : groups > 2 ? 2 : groups > 1 ? 4 : 8; }

// sums [max(8, groups)]: partial sums of the squares of value(c), the first of group g at g * group_parts.
template <typename F>
__device__ __forceinline__ void group_sums(int groups, int size, float* sums, F value) {
  const int parts = group_parts(groups), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int i = warp; i < groups * parts; i += 8) {
    const int c0 = i / parts * size;
    float s = 0.f;
    for (int c = (i % parts) * 32 + lane; c < size; c += parts * 32) {
      const float v = value(c0 + c);
      s += v * v;
    }
    s = warp_sum(s);
    if (lane == 0) sums[i] = s;
  }
}
__device__ __forceinline__ float group_rms_inverse(const float* sums, int group, int parts, int size, float eps) {
  float s = 0.f;
  for (int i = 0; i < parts; ++i) s += sums[group * parts + i];
  return 1.f / sqrtf(s / size + eps);
}

}  // namespace apb

// Runs `...` with T bound to the activation type named by `dtype` (0 = bf16, 1 = fp32).
#define APB_SERVE_DTYPE(dtype, ...)     \
  do {                                  \
    if ((dtype) == 0) {                 \
      using T = __nv_bfloat16;          \
      __VA_ARGS__;                      \
    } else if ((dtype) == 1) {          \
      using T = float;                  \
      __VA_ARGS__;                      \
    }                                   \
    return kBadArgument;                \
  } while (0)
