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
