// Residual update between two sublayers of a decoder that norms a sublayer's output as well as its input.
//
// With y [rows, W] the (fp32) output of the last sublayer,
//     x <- x + y / rms(y) * (offset + post)  (+ embed[token] * scale: the embedding output, ahead of a pass over looped layers)
//     h  = x / rms(x) * (offset + pre)
// in one pass: read x and y once, write x and h once.  y may come in parts: routed experts leave rows `eo` that are weighted and
// summed here, identity experts return the sublayer's own input h_in times their weight (ExpertParts).  Without `post` y is
// added as it is, without y nothing is; without `pre` the fp32 x is written instead of h; write_x = 0 leaves x alone (a look at
// the stream in between).  clear_y resets y to zero after reading it, for producers that add into it.
#include "common.cuh"
#include "host_utils.cuh"
#include "serve_common.cuh"

namespace apb {

constexpr int kResThreads = 256;

struct ExpertParts {
  const void* eo;          // [slots, W] outputs of the routed experts (activation type), or null
  const int* slots;        // [rows, top] row of eo, -1: none
  const float* weights;    // [rows, top]
  const float* ident;      // [rows] weight of h_in
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

__device__ __forceinline__ float block_sum_residual(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  v = 0.f;
#pragma unroll
  for (int i = 0; i < kResThreads / 32; ++i) v += red[i];
  return v;
}

// One block per row; every thread keeps its own columns in shared memory between the passes.
template <typename T, int V>
__global__ void __launch_bounds__(kResThreads)
residual_step_kernel(const ResidualParams p) {
  pdl_entry();
  extern __shared__ __align__(16) float buf[];     // [W]
  __shared__ float red[2][kResThreads / 32];
  const int row = blockIdx.x, W = p.W;
  float* x = p.x + static_cast<long long>(row) * W;
  float* y = p.y ? p.y + static_cast<long long>(row) * W : nullptr;
  const bool has_y = y || p.ex.eo;
  float ry = 1.f;
  if (has_y) {
    float ss = 0.f;
    const int* slots = p.ex.slots + static_cast<long long>(row) * p.ex.top;
    const float* wts = p.ex.weights + static_cast<long long>(row) * p.ex.top;
    const float ident = p.ex.eo ? p.ex.ident[row] : 0.f;
#pragma unroll 2
    for (int c = threadIdx.x * V; c < W; c += kResThreads * V) {
      Run<V> v = {};
      if (y) {
        v = load_run<V>(y + c);
        if (p.clear_y) store_run<V>(y + c, Run<V>{});
      }
      if (p.ex.eo) {
        for (int k = 0; k < p.ex.top; ++k) {
          const int s = slots[k];
          if (s >= 0) axpy<V>(v, wts[k], load_run<V>(static_cast<const T*>(p.ex.eo) + static_cast<long long>(s) * W + c));
        }
        if (ident != 0.f) axpy<V>(v, ident, load_run<V>(static_cast<const T*>(p.ex.h_in) + static_cast<long long>(row) * W + c));
      }
      store_run<V>(buf + c, v);
      ss += sumsq<V>(v);
    }
    if (p.post) ry = 1.f / sqrtf(block_sum_residual(ss, red[0]) / W + p.eps);
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
        for (int i = 0; i < V; ++i) u.v[i] *= ry * (p.offset + g.v[i]);
      }
      axpy<V>(v, 1.f, u);
    }
    if (e) axpy<V>(v, p.embed_scale, load_run<V>(e + c));
    if (p.write_x && (has_y || e)) store_run<V>(x + c, v);
    if (p.pre) {
      store_run<V>(buf + c, v);
      ss += sumsq<V>(v);
    } else {
      store_run<V>(static_cast<float*>(p.h) + static_cast<long long>(row) * W + c, v);
    }
  }
  if (!p.pre) return;
  const float r = 1.f / sqrtf(block_sum_residual(ss, red[1]) / W + p.eps);
  T* h = static_cast<T*>(p.h) + static_cast<long long>(row) * W;
#pragma unroll 2
  for (int c = threadIdx.x * V; c < W; c += kResThreads * V) {
    Run<V> v = load_run<V>(buf + c);
    const Run<V> g = load_run<V>(static_cast<const T*>(p.pre) + c);
#pragma unroll
    for (int i = 0; i < V; ++i) v.v[i] *= r * (p.offset + g.v[i]);
    store_run<V>(h + c, v);
  }
}

}  // namespace apb

extern "C" {
using namespace apb;

int apb_residual_step(float* x, float* y, const void* post, const void* pre, void* h, const int* tokens, const void* embed,
                      int vocab, float embed_scale, const void* eo, const int* slots, const float* weights,
                      const float* ident, const void* h_in, int top, int rows, int W, float offset, float eps, int write_x,
                      int clear_y, int dtype, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (!x || !h || W <= 0 || W > 49152 || (embed && (!tokens || vocab <= 0)) ||
      (eo && (!slots || !weights || !ident || !h_in || top < 1)))
    return kBadArgument;
  const ResidualParams p{x, y, post, pre, h, tokens, embed, vocab, embed_scale, offset, eps, W, write_x, clear_y,
                         ExpertParts{eo, slots, weights, ident, h_in, top}};
  const int smem = W * static_cast<int>(sizeof(float));
  auto run = [&](auto fn) -> int {
    if (smem > 46 * 1024) {                  // the default limit counts the static arrays too
      const cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
      if (e != cudaSuccess) return static_cast<int>(e);
    }
    return static_cast<int>(launch_kernel(fn, dim3(rows), dim3(kResThreads), smem, s, p));
  };
  APB_SERVE_DTYPE(dtype, if ((W & 3) == 0) return run(residual_step_kernel<T, 4>); return run(residual_step_kernel<T, 1>));
}
}
