// Residual update between two sublayers of a decoder that may norm a sublayer's output as well as its input.
//
// With y [rows, W] the (fp32) output of the last sublayer,
//     x <- x + mult * sigmoid(gate + bias) * (y / rms(y) * (offset + post) + y2 / rms(y2) * (offset + post2))
//            (+ embed[token] * scale: the embedding output, ahead of a pass over looped layers)
//     h  = x / rms(x) * (offset + pre)       rms over `groups` equal parts of the row
// in one pass: read x and y once, write x and h once.  y may come in parts: routed experts leave rows `eo` that are weighted and
// summed here, identity experts return the sublayer's own input h_in times their weight (ExpertParts).  Without `post` y is
// added as it is, without y nothing is; y2, the output of a second mixer beside the first, and the gate may be absent; without
// `pre` the fp32 x is written instead of h; write_x = 0 leaves x alone (a look at the stream in between).  clear_y resets y and y2
// to zero after reading them, for producers that add into them.
#include "common.cuh"
#include "host_utils.cuh"
#include "serve_common.cuh"

namespace apb {

constexpr int kResThreads = 256;

struct ExpertParts {
  const void* eo;          // [slots, W] outputs of the routed experts (activation type), or null
  const int* slots;        // [rows, top] row of eo, -1: none
  const float* weights;    // [rows, top], or null: all 1
  const float* ident;      // [rows] weight of h_in, or null: none
  const void* h_in;        // [rows, W] activation type
  int top;
};

struct ResidualParams {
  float* x;
  float* y;
  const void* post;
  const void* pre;
  void* h;                 // activation type, or fp32 without `pre`
  const int* tokens;
  const void* embed;       // [vocab, W] or null
  int vocab;
  float embed_scale, offset, eps;
  int W, write_x, clear_y;
  ExpertParts ex;
  float* y2;               // second output, or null
  const void* post2;
  const void* gate;        // [rows, ld_gate] columns (activation type, or fp32 with gate_f32), or null
  long long ld_gate;
  int gate_f32;
  const void* gate_bias;   // [W] activation type
  float mult;
  int groups;              // of the norm ahead of the next sublayer
};

template <int V>
struct Run {
  float v[V];
};
template <int V, typename T>
__device__ __forceinline__ Run<V> load_run(const T* p) {
  Run<V> r;
  if constexpr (V == 4 && sizeof(T) == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    r.v[0] = f.x, r.v[1] = f.y, r.v[2] = f.z, r.v[3] = f.w;
  } else if constexpr (V == 4) {
    const uint2 w = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w.y));
    r.v[0] = a.x, r.v[1] = a.y, r.v[2] = b.x, r.v[3] = b.y;
  } else {
    r.v[0] = to_f32(*p);
  }
  return r;
}
template <int V, typename T>
__device__ __forceinline__ void store_run(T* p, const Run<V>& r) {
  if constexpr (V == 4 && sizeof(T) == 4)
    *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
  else if constexpr (V == 4)
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(r.v[0], r.v[1]), pack_bf16x2(r.v[2], r.v[3]));
  else
    *p = from_f32<T>(r.v[0]);
}
template <int V>
__device__ __forceinline__ void axpy(Run<V>& a, float f, const Run<V>& b) {
#pragma unroll
  for (int i = 0; i < V; ++i) a.v[i] += f * b.v[i];
}
template <int V>
__device__ __forceinline__ float sumsq(const Run<V>& a) {
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < V; ++i) s += a.v[i] * a.v[i];
  return s;
}

// Sums over the block of one or two values per thread.
template <bool TWO>
__device__ __forceinline__ float2 block_sum_residual(float a, float b, float (*red)[kResThreads / 32]) {
  a = warp_sum(a);
  if (TWO) b = warp_sum(b);
  if ((threadIdx.x & 31) == 0) {
    red[0][threadIdx.x >> 5] = a;
    if (TWO) red[1][threadIdx.x >> 5] = b;
  }
  __syncthreads();
  a = b = 0.f;
#pragma unroll
  for (int i = 0; i < kResThreads / 32; ++i) {
    a += red[0][i];
    if (TWO) b += red[1][i];
  }
  return make_float2(a, b);
}

template <typename T, int V>
__device__ __forceinline__ Run<V> gate_run(const ResidualParams& p, int row, int c) {
  const long long o = static_cast<long long>(row) * p.ld_gate + c;
  Run<V> z = p.gate_f32 ? load_run<V>(static_cast<const float*>(p.gate) + o) : load_run<V>(static_cast<const T*>(p.gate) + o);
  const Run<V> b = load_run<V>(static_cast<const T*>(p.gate_bias) + c);
#pragma unroll
  for (int i = 0; i < V; ++i) {
    const float x = -(z.v[i] + b.v[i]);
    z.v[i] = sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(x)) : 1.f / (1.f + expf(x));
  }
  return z;
}

// One block per row; every thread keeps its own columns in shared memory between the passes.  SIDES: there is a y2; GATED: a gate or
// a multiplier; GROUPED: several groups.
template <typename T, int V, bool SIDES, bool GATED, bool GROUPED>
__global__ void __launch_bounds__(kResThreads)
residual_step_kernel(const ResidualParams p) {
  pdl_entry();
  extern __shared__ __align__(16) float buf[];     // [W], with y2 [2 W], then [max(8, groups)] partial sums of the groups
  __shared__ float red[2][kResThreads / 32], red2[2][kResThreads / 32];
  const int row = blockIdx.x, W = p.W;
  float* x = p.x + static_cast<long long>(row) * W;
  float* y = p.y ? p.y + static_cast<long long>(row) * W : nullptr;
  float* y2 = SIDES ? p.y2 + static_cast<long long>(row) * W : nullptr;
  float* buf2 = buf + W;
  const bool has_y = y || p.ex.eo;
  float2 ry = make_float2(1.f, 1.f);
  if (has_y) {
    float ss = 0.f, ss2 = 0.f;
    const int* slots = p.ex.slots + static_cast<long long>(row) * p.ex.top;
    const float* wts = p.ex.weights ? p.ex.weights + static_cast<long long>(row) * p.ex.top : nullptr;
    const float ident = p.ex.eo && p.ex.ident ? p.ex.ident[row] : 0.f;
#pragma unroll 2
    for (int c = threadIdx.x * V; c < W; c += kResThreads * V) {
      Run<V> v = {};
      if (y) {
        v = load_run<V>(y + c);
        if (p.clear_y) store_run<V>(y + c, Run<V>{});
      }
      if constexpr (SIDES) {
        const Run<V> v2 = load_run<V>(y2 + c);
        if (p.clear_y) store_run<V>(y2 + c, Run<V>{});
        store_run<V>(buf2 + c, v2);
        ss2 += sumsq<V>(v2);
      }
      if (p.ex.eo) {
        for (int k = 0; k < p.ex.top; ++k) {
          const int s = slots[k];
          if (s >= 0) axpy<V>(v, wts ? wts[k] : 1.f, load_run<V>(static_cast<const T*>(p.ex.eo) + static_cast<long long>(s) * W + c));
        }
        if (ident != 0.f) axpy<V>(v, ident, load_run<V>(static_cast<const T*>(p.ex.h_in) + static_cast<long long>(row) * W + c));
      }
      store_run<V>(buf + c, v);
      ss += sumsq<V>(v);
    }
    if (p.post) {
      const float2 s = block_sum_residual<SIDES>(ss, ss2, red);
      ry = make_float2(1.f / sqrtf(s.x / W + p.eps), SIDES ? 1.f / sqrtf(s.y / W + p.eps) : 0.f);
    }
  }
  const T* e = nullptr;
  if (p.embed) {
    const int tok = min(max(p.tokens[row], 0), p.vocab - 1);
    e = static_cast<const T*>(p.embed) + static_cast<long long>(tok) * W;
  }
  float ss = 0.f;
#pragma unroll 2
  for (int c = threadIdx.x * V; c < W; c += kResThreads * V) {
    Run<V> v = load_run<V>(x + c);
    if (has_y) {
      Run<V> u = load_run<V>(buf + c);
      if (p.post) {
        const Run<V> g = load_run<V>(static_cast<const T*>(p.post) + c);
#pragma unroll
        for (int i = 0; i < V; ++i) u.v[i] *= ry.x * (p.offset + g.v[i]);
      }
      if constexpr (SIDES) {
        const Run<V> u2 = load_run<V>(buf2 + c), g = load_run<V>(static_cast<const T*>(p.post2) + c);
#pragma unroll
        for (int i = 0; i < V; ++i) u.v[i] += u2.v[i] * ry.y * (p.offset + g.v[i]);
      }
      if (GATED && p.gate) {
        const Run<V> g = gate_run<T, V>(p, row, c);
#pragma unroll
        for (int i = 0; i < V; ++i) u.v[i] *= g.v[i];
      }
      axpy<V>(v, GATED ? p.mult : 1.f, u);
    }
    if (e) axpy<V>(v, p.embed_scale, load_run<V>(e + c));
    if (p.write_x && (has_y || e)) store_run<V>(x + c, v);
    if (p.pre) {
      store_run<V>(buf + c, v);
      if (!GROUPED) ss += sumsq<V>(v);
    } else {
      store_run<V>(static_cast<float*>(p.h) + static_cast<long long>(row) * W + c, v);
    }
  }
  if (!p.pre) return;
  T* h = static_cast<T*>(p.h) + static_cast<long long>(row) * W;
  if constexpr (!GROUPED) {
    const float r = 1.f / sqrtf(block_sum_residual<false>(ss, 0.f, red2).x / W + p.eps);
#pragma unroll 2
    for (int c = threadIdx.x * V; c < W; c += kResThreads * V) {
      Run<V> v = load_run<V>(buf + c);
      const Run<V> g = load_run<V>(static_cast<const T*>(p.pre) + c);
#pragma unroll
      for (int i = 0; i < V; ++i) v.v[i] *= r * (p.offset + g.v[i]);
      store_run<V>(h + c, v);
    }
    return;
  }
  float* sums = buf + (SIDES ? 2 * W : W);
  const int size = W / p.groups, parts = group_parts(p.groups);
  __syncthreads();
  group_sums(p.groups, size, sums, [&](int c) { return buf[c]; });
  __syncthreads();
  for (int c = threadIdx.x * V; c < W; c += kResThreads * V) {
    Run<V> v = load_run<V>(buf + c);
    const Run<V> g = load_run<V>(static_cast<const T*>(p.pre) + c);
    float r = 0.f;
#pragma unroll
    for (int i = 0; i < V; ++i) {
      if (i == 0 || (c + i) % size == 0) r = group_rms_inverse(sums, (c + i) / size, parts, size, p.eps);
      v.v[i] *= r * (p.offset + g.v[i]);
    }
    store_run<V>(h + c, v);
  }
}

}  // namespace apb

extern "C" {
using namespace apb;

// gate [rows, ld_gate] (fp32 with gate_f32) and gate_bias [W], or null; y2 and post2 only beside y and post.
int apb_residual_step(float* x, float* y, const void* post, const void* pre, void* h, const int* tokens, const void* embed,
                      int vocab, float embed_scale, const void* eo, const int* slots, const float* weights,
                      const float* ident, const void* h_in, int top, int rows, int W, float offset, float eps, int write_x,
                      int clear_y, float* y2, const void* post2, const void* gate, long long ld_gate, int gate_f32,
                      const void* gate_bias, float mult, int groups, int dtype, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (!x || !h || W <= 0 || W > 49152 || (embed && (!tokens || vocab <= 0)) || (eo && (!slots || top < 1 || (ident && !h_in))) ||
      (y2 && (!y || !post || !post2 || W > 24576)) || (gate && (!gate_bias || ld_gate < W)) || groups < 1 || W % groups)
    return kBadArgument;
  const ResidualParams p{x, y, post, pre, h, tokens, embed, vocab, embed_scale, offset, eps, W, write_x, clear_y,
                         ExpertParts{eo, slots, weights, ident, h_in, top}, y2, post2, gate, ld_gate, gate_f32, gate_bias, mult, groups};
  const int smem = ((y2 ? 2 * W : W) + (groups > 8 ? groups : 8)) * static_cast<int>(sizeof(float));
  auto run = [&](auto fn) -> int {
    if (smem > 46 * 1024) {                  // the default limit counts the static arrays too
      const cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
      if (e != cudaSuccess) return static_cast<int>(e);
    }
    return static_cast<int>(launch_kernel(fn, dim3(rows), dim3(kResThreads), smem, s, p));
  };
  const bool vec = (W & 3) == 0 && (!gate || (!(ld_gate & 3) && !(reinterpret_cast<uintptr_t>(gate) & 15)));
  const bool grouped = groups > 1 && pre;
#define APB_RESIDUAL(V)                                                                                          \
  do {                                                                                                           \
    if (y2) return grouped ? run(residual_step_kernel<T, V, true, true, true>) : run(residual_step_kernel<T, V, true, true, false>);    \
    if (scaled) return grouped ? run(residual_step_kernel<T, V, false, true, true>) : run(residual_step_kernel<T, V, false, true, false>); \
    return grouped ? run(residual_step_kernel<T, V, false, false, true>) : run(residual_step_kernel<T, V, false, false, false>);       \
  } while (0)
  const bool scaled = gate || mult != 1.f;
  APB_SERVE_DTYPE(dtype, if (vec) APB_RESIDUAL(4); APB_RESIDUAL(1));
#undef APB_RESIDUAL
}
}
