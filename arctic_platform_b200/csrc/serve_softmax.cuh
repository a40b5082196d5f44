// Declarations shared by the paged softmax attention kernels (serve_softmax*.cu, serve_flash_tc.cu).
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

// ---------------------------------------------------------------------------- pieces of the tcgen05 kernels
__device__ __forceinline__ float xtc_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// Pairs of fp32 values in one 64-bit register: half the issue slots of the scalar forms.
__device__ __forceinline__ uint64_t xtc_pair(float lo, float hi) {
  uint64_t v;
  asm("mov.b64 %0, {%1, %2};" : "=l"(v) : "f"(lo), "f"(hi));
  return v;
}
__device__ __forceinline__ float2 xtc_unpair(uint64_t v) {
  float2 f;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(v));
  return f;
}
__device__ __forceinline__ uint64_t xtc_mul2(uint64_t a, uint64_t b) {
  uint64_t v;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(v) : "l"(a), "l"(b));
  return v;
}
__device__ __forceinline__ uint64_t xtc_fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t v;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(v) : "l"(a), "l"(b), "l"(c));
  return v;
}
__device__ __forceinline__ uint64_t xtc_add2(uint64_t a, uint64_t b) {
  uint64_t v;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(v) : "l"(a), "l"(b));
  return v;
}
// Waits for a tensor-memory load into r; nothing that reads r can move in front of it.
__device__ __forceinline__ void xtc_wait_load(uint32_t (&r)[32]) {
  asm volatile("tcgen05.wait::ld.sync.aligned;"
               : "+r"(r[0]), "+r"(r[1]), "+r"(r[2]), "+r"(r[3]), "+r"(r[4]), "+r"(r[5]), "+r"(r[6]), "+r"(r[7]),
               "+r"(r[8]), "+r"(r[9]), "+r"(r[10]), "+r"(r[11]), "+r"(r[12]), "+r"(r[13]), "+r"(r[14]),
               "+r"(r[15]), "+r"(r[16]), "+r"(r[17]), "+r"(r[18]), "+r"(r[19]), "+r"(r[20]), "+r"(r[21]),
               "+r"(r[22]), "+r"(r[23]), "+r"(r[24]), "+r"(r[25]), "+r"(r[26]), "+r"(r[27]), "+r"(r[28]),
               "+r"(r[29]), "+r"(r[30]), "+r"(r[31])
               :: "memory");
}

}  // namespace apb
