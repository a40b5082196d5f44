// Declarations shared by the paged softmax attention kernels (serve_softmax.cu, serve_softmax_tc.cu).
#pragma once
#include "serve_common.cuh"

namespace apb {

// Score shaping and output stage of a softmax attention.
//   score = scale q.k, then cap * tanh(score / cap) when cap > 0; key j of query i is visible when j <= i, with chunk > 0
//   floor(i / chunk) = floor(j / chunk) (positions of the sequence) and with window > 0 i - j < window.
// sink: a score per head that has no key and no value and counts once in the denominator (null: none).
// maps = 2 (differential attention): a head has two query and two key vectors of D columns side by side and one value
// head; with a1, a2 the two softmax outputs, o = a1 - lambda a2, out = o / rms(o) * post_scale.
// gate: out is multiplied by sigmoid of gate[row, head] (gate_cols 1) or gate[row, head * E + c] (gate_cols E), in the
// activation type.  maps = 1 only, as is the sink.
struct SoftmaxSpec {
  float scale, cap;
  int chunk;
  int maps;
  const float* lambda;     // device scalar (maps = 2)
  float post_scale, eps;
  int window;
  const float* sink;       // [heads] or null
  const void* gate;        // or null
  long long ldg;
  int gate_cols;
};

// First position that the query at `pos` sees.
__device__ __forceinline__ int visible_begin(int pos, const SoftmaxSpec& sp) {
  const int c = sp.chunk > 0 ? pos - pos % sp.chunk : 0;
  return sp.window > 0 ? max(c, pos - sp.window + 1) : c;
}

template <typename T>
__device__ __forceinline__ float output_gate(const SoftmaxSpec& sp, long long row, int head, int c) {
  if (!sp.gate) return 1.f;
  const T* g = static_cast<const T*>(sp.gate) + row * sp.ldg + static_cast<long long>(head) * sp.gate_cols;
  return 1.f / (1.f + expf(-to_f32(g[sp.gate_cols == 1 ? 0 : c])));
}

// Reciprocal of the denominator of a sum of weights relative to 2^ref, with the head's sink; times 2^ref over the common
// reference.  In units of log 2.
__device__ __forceinline__ float inverse_sum(const SoftmaxSpec& sp, int head, float ref, float sum) {
  if (!sp.sink) return 1.f / sum;
  const float s = sp.sink[head] * 1.4426950408889634f, top = fmaxf(ref, s), f = exp2f(ref - top);
  return f / (sum * f + exp2f(s - top));
}

// |scores| <= cap: with cap up to kMaxFixedCap a fixed reference keeps exp(score - ref) and its sums inside the fp32 range
// (exponents between -2 cap + 44 >= -84 and 44), so no running maximum is needed.
constexpr float kMaxFixedCap = 64.f;
__host__ __device__ inline bool fixed_reference(float cap) { return cap > 0.f && cap <= kMaxFixedCap; }
__host__ __device__ inline float score_reference(float cap) { return cap > 44.f ? cap - 44.f : 0.f; }

// tanh to fp32 accuracy.  Near zero (|z| <= kSmallTanh) its odd series to z^9, whose next term is below 4e-7; elsewhere
// through the exponential.
constexpr float kSmallTanh = 0.4f;
__device__ __forceinline__ float tanh_series(float z) {
  const float t = z * z;
  float s = fmaf(t, 62.f / 2835.f, -17.f / 315.f);
  s = fmaf(t, s, 2.f / 15.f);
  s = fmaf(t, s, -1.f / 3.f);
  return fmaf(z * t, s, z);
}
__device__ __forceinline__ float tanh_exp(float z) { return 1.f - __fdividef(2.f, 1.f + __expf(2.f * z)); }
__device__ __forceinline__ float tanh_any(float z) { return fabsf(z) <= kSmallTanh ? tanh_series(z) : tanh_exp(z); }

}  // namespace apb
