// Declarations shared by the retention kernels (retention.cu, retention_mma.cu).
#pragma once
#include "serve_common.cuh"

namespace apb {

struct RetentionParams {
  ServeEntries e;
  const void* p;          // projection buffer [rows, ld]
  long long ld;
  int q_col, k_col, v_col, g_col;
  const float* cos_t;     // [positions, rot_dims / 2]
  const float* sin_t;
  int rot_dims;
  const float* log2_decay;  // [H] log2 of the decay (-inf for 0)
  float k_scale;
  float* state;           // [slots, H, D, E]
  float* o;               // [rows, H, E] fp32, un-normalised (chunk kernels)
  void* out;              // [rows, ldo] (activation type), already offset to its first column
  long long ldo;
  float out_scale, eps;
  int H, D, E;
};

__device__ __forceinline__ float decay_pow(float log2_decay, int n) { return n == 0 ? 1.f : exp2f(log2_decay * n); }

// Element d of a rotated head whose raw values start at `src`.
template <typename T>
__device__ __forceinline__ float rotated(const T* src, int d, int rot, const float* c, const float* s) {
  const int half = rot >> 1;
  const float a = to_f32(src[d]);
  if (d >= rot) return a;
  if (d < half) return a * c[d] - to_f32(src[d + half]) * s[d];
  return a * c[d - half] + to_f32(src[d - half]) * s[d - half];
}

}  // namespace apb
