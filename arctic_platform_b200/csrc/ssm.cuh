// Declarations shared by the state-space mixer's kernels (ssm.cu, ssm_mma.cu).
#pragma once
#include "serve_common.cuh"

namespace apb {

// Selective state space with one decay per head and token (Mamba-2):
//     dt = softplus(raw dt + bias_h),  a = exp(-exp(A_log_h) dt)
//     S_t = a S_{t-1} + dt B_t x_t^T          S [N, E] per head, fp32, carried from step to step in a state slot
//     y_t = S_t^T C_t + D_h x_t
// x (H heads of E), B and C (G groups of N; head h reads group h / (H / G)) are the silu of a causal depth-wise convolution
// over the projected columns [x | B | C]; its last taps - 1 inputs are carried as well (double buffered, see serve_layers.cu).
struct SsmParams {
  ServeEntries e;
  const void* p;            // projection buffer [rows, ld] (activation type)
  long long ld;
  int xbc_col, dt_col;
  const void* conv_w;       // [taps, channels] and [channels] (activation type); channels = H E + 2 G N
  const void* conv_b;
  int taps;
  float* hist;              // [slots, 2, taps - 1, channels] fp32, or null (taps = 1)
  const int* parity;
  const void* dt_bias;      // [H] each (activation type)
  const void* a_log;
  const void* d_skip;
  void* xbc;                // [rows, ldx] convolved columns (activation type), rows of entries longer than one token
  long long ldx;
  float2* steps;            // [rows, H] (dt, log2 a), rows of entries longer than one token
  float* state;             // [slots, H, N, E]
  float* y;                 // [rows, H * E] fp32
  int H, E, G, N;
};

__device__ __forceinline__ float softplus_f(float v) { return v > 20.f ? v : log1pf(expf(v)); }
// silu of an activation: to fp32 accuracy for fp32 engines, well inside a bf16 rounding step for bf16 ones
template <typename T>
__device__ __forceinline__ float silu_act(float v) {
  if constexpr (sizeof(T) == 2) return __fdividef(v, 1.f + __expf(-v));
  return v / (1.f + expf(-v));
}

template <typename T>
__device__ __forceinline__ float2 ssm_step_of(const SsmParams& p, long long row, int h) {
  const float raw = to_f32(static_cast<const T*>(p.p)[row * p.ld + p.dt_col + h]) + to_f32(static_cast<const T*>(p.dt_bias)[h]);
  const float dt = softplus_f(raw);
  return make_float2(dt, -expf(to_f32(static_cast<const T*>(p.a_log)[h])) * dt * 1.4426950408889634f);
}

}  // namespace apb
