// Recurrent mixers with an fp32 matrix state per head, carried from step to step in a state slot (recurrent.cu, memory_mma.cu,
// delta_mma.cu, time_mix_mma.cu).
//
// With S [D, E] the state of a head, one token does
//   matrix memory   i = cap tanh((z_i + b_i) / cap), f = logsigmoid(cap tanh((z_f + b_f) / cap)),  m' = max(f + m, i)
//                   S' = exp(f + m - m') S + exp(i - m') k v^T,  n' alike with k alone
//                   o  = S'^T q / (max(|n' . q|, exp(-m')) + 1e-6),  q = D^-1/2 times its projection;  m starts at 0
//   delta rule      q, k, v: silu of a causal convolution per channel; q, k unit vectors (1e-6 under the root), q times D^-1/2
//                   S1 = g S,  u = beta (v - S1^T k),  S' = S1 + k u^T,  o = S'^T q
//                   g = exp(-exp(A) softplus(z_a + b_a)),  beta = sigmoid(z_b)
//   time mixing     o = (S + diag(u) k v^T)^T r,  S' = diag(w) S + k v^T,  w = exp(-exp(z + w0)) per key channel
// and the head's output is o / rms(o) * gain * gate, the gate a sigmoid or silu of projected columns.  q, k, v are activations; all
// else is fp32.
#pragma once
#include "serve_common.cuh"

namespace apb {

enum RecurrentRule : int { kRuleMemory = 0, kRuleDelta = 1, kRuleTimeMix = 2 };

struct RecurrentParams {    // filled by the caller (ops/serving.py mirrors the layout)
  ServeEntries e;
  const void* p;            // projected columns (activation type), rows `ld` apart; the offsets are in elements
  long long ld, q_off, k_off, v_off;
  long long a_off, b_off;   // memory: z_i, z_f; delta: z_a, z_b; one column per head
  const void* w0;           // activation type.  memory: b_i [H]; delta: A [H]; time mixing: w0 [H * D]
  const void* w1;           // memory: b_f [H]; delta: b_a [H]; time mixing: u [H * D]
  const float* z;           // time mixing: [rows, ldz] decay projections
  long long ldz;
  float cap;
  const void* conv_w;       // delta: [taps, channels], channels = 2 KH D + H E (q, k, v side by side)
  int taps;
  float* hist;              // [slots, 2, taps - 1, channels], or null (taps = 1)
  const int* parity;
  const void* xc;           // delta: [rows, ldx] convolved columns of the entries longer than one token
  long long ldx;
  float* state;             // [slots, H, D, E]
  float* aux;               // memory: [slots, H, D + 1] n, m
  int H, KH, D, E;          // KH: heads of q and k; head h reads h / (H / KH)
  float* y;                 // [rows, H * E] o of the entries longer than one token
  const void* gain;         // activation type; head h reads gain + h * gain_step
  int gain_step;
  long long g_off;          // gate columns (H * E) in p
  int silu;                 // gate: silu, else sigmoid
  void* out;                // [rows, ldo] activation type
  long long ldo;
  float eps;
};

inline bool recurrent_params_ok(int rule, const RecurrentParams& a) {
  return a.p && a.state && a.w0 && a.w1 && a.gain && a.out && a.H > 0 && a.KH > 0 && a.H % a.KH == 0 && a.D > 0 && a.E > 0 &&
         a.D <= 1024 && a.E <= 1024 &&
         (rule == kRuleMemory  ? a.aux && a.cap > 0.f
          : rule == kRuleDelta ? a.conv_w && a.taps >= 1 && (a.taps == 1 || (a.hist && a.parity))
                               : rule == kRuleTimeMix && a.z);
}

// Chunked kernels sum log2 decays and exponentiate differences of the sums.  A token's decay counts at most this much there: 2^-64
// leaves nothing of a state either, and the sums of a chunk stay small enough for fp32 differences.
constexpr float kMaxLogDecay = 64.f;

__device__ __forceinline__ float rec_softplus(float v) { return v > 20.f ? v : log1pf(expf(v)); }
__device__ __forceinline__ float rec_gate(float z, int silu) {
  const float s = 1.f / (1.f + expf(-z));
  return silu ? z * s : s;
}
// (log forget gate, log input gate) of a matrix memory
template <typename T>
__device__ __forceinline__ float2 memory_gates(const RecurrentParams& p, long long row, int h) {
  const T* pr = static_cast<const T*>(p.p) + row * p.ld;
  const float zi = to_f32(pr[p.a_off + h]) + to_f32(static_cast<const T*>(p.w0)[h]);
  const float zf = to_f32(pr[p.b_off + h]) + to_f32(static_cast<const T*>(p.w1)[h]);
  return make_float2(-rec_softplus(-p.cap * tanhf(zf / p.cap)), p.cap * tanhf(zi / p.cap));
}
// (log decay, beta) of a delta rule
template <typename T>
__device__ __forceinline__ float2 delta_gates(const RecurrentParams& p, long long row, int h) {
  const T* pr = static_cast<const T*>(p.p) + row * p.ld;
  const float za = to_f32(pr[p.a_off + h]) + to_f32(static_cast<const T*>(p.w1)[h]);
  return make_float2(-expf(to_f32(static_cast<const T*>(p.w0)[h])) * rec_softplus(za), 1.f / (1.f + expf(-to_f32(pr[p.b_off + h]))));
}

}  // namespace apb
