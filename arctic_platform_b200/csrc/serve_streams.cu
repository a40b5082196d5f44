// Parallel residual streams (hyper-connections) with the norm of the next sublayer.
//
// A row has S fp32 streams x [rows, S, W].  Between two sublayers, with y the output of the first one,
//     x_t <- sum_s mix[s, t] x_s + out[t] y          (all streams at once, from the old ones)
//     u   =  sum_t in[t] x_t                          (the input of the next sublayer)
//     h   =  u / rms(u) * w
// which is one pass over the streams: read x and y once, write x and h once.  Without y the streams are left alone (first
// sublayer); without w the raw sum u is written in fp32 instead of h; write_x = 0 leaves the streams alone although y is
// mixed in (the end of the model, or a look at the sum of the streams in between).
// `clear_y` resets y to zero after reading it, for producers that add into it.
#include "common.cuh"
#include "host_utils.cuh"
#include "serve_common.cuh"

namespace apb {

constexpr int kStreamThreads = 256;
constexpr int kMaxStreams = 16;

struct StreamParams {
  float* x;            // [rows, S, W]
  float* y;            // [rows, W] or null
  const void* mix;     // [S, S] (from, to), out [S], in [S] (null: ones), norm weight [W] or null: activation type
  const void* out;
  const void* in;
  const void* w;
  void* h;             // [rows, W] activation type, or fp32 without w
  int W, S, write_x, clear_y;
  float eps;
};

__device__ __forceinline__ float block_sum_streams(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  v = 0.f;
#pragma unroll
  for (int i = 0; i < kStreamThreads / 32; ++i) v += red[i];
  return v;
}

template <typename T>
__device__ __forceinline__ float4 load4(const T* p) {
  if constexpr (sizeof(T) == 2) {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
    return make_float4(a.x, a.y, b.x, b.y);
  } else {
    return *reinterpret_cast<const float4*>(p);
  }
}
template <typename T>
__device__ __forceinline__ void store4(T* p, float4 v) {
  if constexpr (sizeof(T) == 2)
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
  else
    *reinterpret_cast<float4*>(p) = v;
}
__device__ __forceinline__ void axpy4(float4& a, float f, const float4& v) {
  a.x += f * v.x;
  a.y += f * v.y;
  a.z += f * v.z;
  a.w += f * v.w;
}

// S streams known at compile time, W a multiple of 4.  One block per row; u waits in shared memory for the row's norm.
template <typename T, int S>
__global__ void __launch_bounds__(kStreamThreads)
stream_step_vec_kernel(const StreamParams p) {
  pdl_entry();
  extern __shared__ float4 u_s[];                  // [W / 4]
  __shared__ float red[kStreamThreads / 32];
  const long long row = blockIdx.x;
  float* x = p.x + row * S * p.W;
  float* y = p.y ? p.y + row * p.W : nullptr;
  float mix[S][S], out[S], in[S];
#pragma unroll
  for (int t = 0; t < S; ++t) {
    in[t] = p.in ? to_f32(static_cast<const T*>(p.in)[t]) : 1.f;
    out[t] = y ? to_f32(static_cast<const T*>(p.out)[t]) : 0.f;
#pragma unroll
    for (int s = 0; s < S; ++s) mix[s][t] = y ? to_f32(static_cast<const T*>(p.mix)[s * S + t]) : 0.f;
  }
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float ss = 0.f;
#pragma unroll 2
  for (int c = threadIdx.x * 4; c < p.W; c += kStreamThreads * 4) {
    float4 old[S], u = zero;
#pragma unroll
    for (int s = 0; s < S; ++s) old[s] = *reinterpret_cast<const float4*>(x + static_cast<long long>(s) * p.W + c);
    if (y) {
      const float4 yv = *reinterpret_cast<const float4*>(y + c);
      if (p.clear_y) *reinterpret_cast<float4*>(y + c) = zero;
#pragma unroll
      for (int t = 0; t < S; ++t) {
        float4 v = zero;
#pragma unroll
        for (int s = 0; s < S; ++s) axpy4(v, mix[s][t], old[s]);
        axpy4(v, out[t], yv);
        if (p.write_x) *reinterpret_cast<float4*>(x + static_cast<long long>(t) * p.W + c) = v;
        axpy4(u, in[t], v);
      }
    } else {
#pragma unroll
      for (int t = 0; t < S; ++t) axpy4(u, in[t], old[t]);
    }
    if (p.w) {
      u_s[c >> 2] = u;
      ss += u.x * u.x + u.y * u.y + u.z * u.z + u.w * u.w;
    } else {
      *reinterpret_cast<float4*>(static_cast<float*>(p.h) + row * p.W + c) = u;
    }
  }
  if (!p.w) return;
  const float f = 1.f / sqrtf(block_sum_streams(ss, red) / p.W + p.eps);
  T* h = static_cast<T*>(p.h) + row * p.W;
  for (int c = threadIdx.x * 4; c < p.W; c += kStreamThreads * 4) {        // the thread's own elements
    const float4 u = u_s[c >> 2], w = load4(static_cast<const T*>(p.w) + c);
    store4(h + c, make_float4(u.x * f * w.x, u.y * f * w.y, u.z * f * w.z, u.w * f * w.w));
  }
}

// Any number of streams up to kMaxStreams, any W.
template <typename T>
__global__ void __launch_bounds__(kStreamThreads)
stream_step_kernel(const StreamParams p) {
  pdl_entry();
  extern __shared__ float us[];                    // [W]
  __shared__ float red[kStreamThreads / 32];
  __shared__ float mix[kMaxStreams * kMaxStreams], out[kMaxStreams], in[kMaxStreams];
  const long long row = blockIdx.x;
  const int S = p.S;
  float* x = p.x + row * S * p.W;
  float* y = p.y ? p.y + row * p.W : nullptr;
  for (int i = threadIdx.x; i < S * S; i += kStreamThreads) mix[i] = y ? to_f32(static_cast<const T*>(p.mix)[i]) : 0.f;
  if (threadIdx.x < S) {
    in[threadIdx.x] = p.in ? to_f32(static_cast<const T*>(p.in)[threadIdx.x]) : 1.f;
    out[threadIdx.x] = y ? to_f32(static_cast<const T*>(p.out)[threadIdx.x]) : 0.f;
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = threadIdx.x; c < p.W; c += kStreamThreads) {
    float old[kMaxStreams], u = 0.f;
#pragma unroll
    for (int s = 0; s < kMaxStreams; ++s) old[s] = s < S ? x[static_cast<long long>(s) * p.W + c] : 0.f;
    const float yv = y ? y[c] : 0.f;
    if (y && p.clear_y) y[c] = 0.f;
    if (y) {
#pragma unroll 1
      for (int t = 0; t < S; ++t) {
        float v = out[t] * yv;
#pragma unroll
        for (int s = 0; s < kMaxStreams; ++s)
          if (s < S) v += mix[s * S + t] * old[s];
        if (p.write_x) x[static_cast<long long>(t) * p.W + c] = v;
        u += in[t] * v;
      }
    } else {
#pragma unroll
      for (int s = 0; s < kMaxStreams; ++s)
        if (s < S) u += in[s] * old[s];
    }
    if (p.w) {
      us[c] = u;
      ss += u * u;
    } else {
      static_cast<float*>(p.h)[row * p.W + c] = u;
    }
  }
  if (!p.w) return;
  const float f = 1.f / sqrtf(block_sum_streams(ss, red) / p.W + p.eps);
  for (int c = threadIdx.x; c < p.W; c += kStreamThreads)
    static_cast<T*>(p.h)[row * p.W + c] = from_f32<T>(us[c] * f * to_f32(static_cast<const T*>(p.w)[c]));
}

}  // namespace apb

extern "C" {
using namespace apb;

int apb_stream_step(float* x, float* y, const void* mix, const void* out, const void* in, const void* w, void* h, int rows,
                    int W, int S, int write_x, int clear_y, float eps, int dtype, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (!x || !h || W <= 0 || S < 1 || S > kMaxStreams || (y && (!mix || !out)) || W > 49152) return kBadArgument;
  const StreamParams p{x, y, mix, out, in, w, h, W, S, write_x, clear_y, eps};
  const int smem = w ? W * static_cast<int>(sizeof(float)) : 0;
  auto run = [&](auto fn) -> int {
    if (smem > 46 * 1024) {                  // the default limit counts the static arrays too
      const cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
      if (e != cudaSuccess) return static_cast<int>(e);
    }
    return static_cast<int>(launch_kernel(fn, dim3(rows), dim3(kStreamThreads), smem, s, p));
  };
  const bool vec = (W & 3) == 0;
  APB_SERVE_DTYPE(dtype, if (vec && S == 1) return run(stream_step_vec_kernel<T, 1>);
                  if (vec && S == 2) return run(stream_step_vec_kernel<T, 2>);
                  if (vec && S == 3) return run(stream_step_vec_kernel<T, 3>);
                  if (vec && S == 4) return run(stream_step_vec_kernel<T, 4>); return run(stream_step_kernel<T>));
}
}
