// State-space mixer (see ssm.cuh) on a ragged serving batch.
//
//  * ssm_decode_kernel  entries of one token: convolution, step size and state update fused; streams the state of a
//                       (sequence, head) once (read, update, write) -- bound by the bytes of the state;
//  * ssm_conv_kernel    longer entries: convolution + silu of every row, step sizes, the new convolution history;
//  * ssm_scan_kernel    longer entries, token by token in fp32 (the fp32 engine, odd sizes): one CTA per (entry, head,
//                       32-column slice of E), the slice of the state in shared memory;
//  * gate_norm kernels  every row: y silu(z), normalised in equal parts, times a weight.
//
// bf16 engines run the longer entries' recurrence on tensor cores (ssm_mma.cu).
#include "common.cuh"
#include "host_utils.cuh"
#include "ssm.cuh"

namespace apb {

// ---------------------------------------------------------------------------- one token
constexpr int kSsmDecThreads = 256;
constexpr int kSsmDecAhead = 8;    // state rows per thread that are on their way while the convolution is computed

template <typename T, int VEC>
__global__ void __launch_bounds__(kSsmDecThreads)
ssm_decode_kernel(const SsmParams p) {
  pdl_entry();
  extern __shared__ float ssm_smem[];
  const int en = blockIdx.x, h = blockIdx.y;
  if (p.e.len[en] != 1) return;
  const int N = p.N, E = p.E, rep = p.H / p.G, g = h / rep;
  float* xs = ssm_smem;            // [E]
  float* bs = xs + E;              // [N]
  float* cs = bs + N;              // [N]
  float* red = cs + N;             // [ny][E]
  const long long row = p.e.start[en];
  const int slot = p.e.slot[en], pos = p.e.pos0[en];
  const int channels = p.H * E + 2 * p.G * N, hist = p.taps - 1;
  const T* in = static_cast<const T*>(p.p) + row * p.ld + p.xbc_col;
  const float* old_h = nullptr;
  float* new_h = nullptr;
  if (hist > 0) {
    const int par = p.parity[slot] & 1;
    old_h = p.hist + (static_cast<long long>(slot) * 2 + par) * hist * channels;
    new_h = p.hist + (static_cast<long long>(slot) * 2 + (par ^ 1)) * hist * channels;
  }
  float* S = p.state + (static_cast<long long>(slot) * p.H + h) * N * E;
  const int nx = min(E / VEC, kSsmDecThreads), ny = kSsmDecThreads / nx;
  const int tx = threadIdx.x % nx, ty = threadIdx.x / nx;
  float4 ahead[kSsmDecAhead];
  if (VEC == 4) {
#pragma unroll
    for (int k = 0; k < kSsmDecAhead; ++k) {
      const int d = ty + k * ny;
      ahead[k] = make_float4(0.f, 0.f, 0.f, 0.f);            // position 0: the slot may hold anything
      if (pos > 0 && ty < ny && d < N) ahead[k] = __ldcs(reinterpret_cast<const float4*>(S + static_cast<long long>(d) * E + tx * 4));
    }
  }
  const bool group_owner = h % rep == 0;                     // writes the history of its group's B and C
  for (int i = threadIdx.x; i < E + 2 * N; i += kSsmDecThreads) {
    const int c = i < E ? h * E + i : (i < E + N ? p.H * E + g * N + i - E : p.H * E + (p.G + g) * N + i - E - N);
    const float cur = to_f32(in[c]);
    const T* w = static_cast<const T*>(p.conv_w) + c;
    float v = to_f32(static_cast<const T*>(p.conv_b)[c]) + to_f32(w[static_cast<long long>(hist) * channels]) * cur;
    for (int j = 0; j < hist; ++j) {
      const float x = pos - hist + j >= 0 ? old_h[static_cast<long long>(j) * channels + c] : 0.f;
      v += to_f32(w[static_cast<long long>(j) * channels]) * x;
      if (j > 0 && (i < E || group_owner)) new_h[static_cast<long long>(j - 1) * channels + c] = x;
    }
    if (hist > 0 && (i < E || group_owner)) new_h[static_cast<long long>(hist - 1) * channels + c] = cur;
    xs[i] = to_f32(from_f32<T>(silu_act<T>(v)));                // x, B and C are activations
  }
  const float2 st = ssm_step_of<T>(p, row, h);
  const float dt = st.x, dec = pos == 0 ? 0.f : exp2f(st.y);
  __syncthreads();
  if (ty < ny) {
    for (int cx = tx; cx < E / VEC; cx += nx) {
      float acc[VEC], v[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        acc[i] = 0.f;
        v[i] = xs[cx * VEC + i] * dt;
      }
      int d = ty;
      if (VEC == 4 && cx == tx) {
#pragma unroll
        for (int k = 0; k < kSsmDecAhead; ++k, d += ny)
          if (d < N) {
            const float bd = bs[d], cd = cs[d];
            const float4 o = ahead[k];
            const float4 n = make_float4(o.x * dec + bd * v[0], o.y * dec + bd * v[1 % VEC], o.z * dec + bd * v[2 % VEC],
                                         o.w * dec + bd * v[3 % VEC]);
            acc[0] += n.x * cd;
            acc[1 % VEC] += n.y * cd;
            acc[2 % VEC] += n.z * cd;
            acc[3 % VEC] += n.w * cd;
            __stcs(reinterpret_cast<float4*>(S + static_cast<long long>(d) * E + cx * 4), n);
          }
      }
#pragma unroll 4
      for (; d < N; d += ny) {
        float* sp = S + static_cast<long long>(d) * E + cx * VEC;
        float s[VEC];
#pragma unroll
        for (int i = 0; i < VEC; ++i) s[i] = 0.f;
        if (pos > 0) {
          if (VEC == 4) {
            const float4 t = __ldcs(reinterpret_cast<const float4*>(sp));
            s[0] = t.x;
            s[1 % VEC] = t.y;
            s[2 % VEC] = t.z;
            s[3 % VEC] = t.w;
          } else {
            s[0] = *sp;
          }
        }
        const float bd = bs[d], cd = cs[d];
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          s[i] = s[i] * dec + bd * v[i];
          acc[i] += s[i] * cd;
        }
        if (VEC == 4)
          __stcs(reinterpret_cast<float4*>(sp), make_float4(s[0], s[1 % VEC], s[2 % VEC], s[3 % VEC]));
        else
          *sp = s[0];
      }
#pragma unroll
      for (int i = 0; i < VEC; ++i) red[ty * E + cx * VEC + i] = acc[i];
    }
  }
  __syncthreads();
  const float skip = to_f32(static_cast<const T*>(p.d_skip)[h]);
  for (int i = threadIdx.x; i < E; i += kSsmDecThreads) {
    float o = skip * xs[i];
    for (int y = 0; y < ny; ++y) o += red[y * E + i];
    p.y[row * p.H * E + static_cast<long long>(h) * E + i] = o;
  }
}

// ---------------------------------------------------------------------------- convolution of longer entries
// One block = up to kSsmRows rows of one entry (tiles[2 i] = entry, tiles[2 i + 1] = first row) x 512 channels, two
// neighbouring channels per thread.  The first channel block also computes the rows' step sizes.
constexpr int kSsmRows = 16;
constexpr int kSsmConvThreads = 256;

template <typename T, int TAPS>                              // TAPS 0: any number
__global__ void __launch_bounds__(kSsmConvThreads)
ssm_conv_kernel(const SsmParams p, const int* __restrict__ tiles) {
  pdl_entry();
  const int en = tiles[2 * blockIdx.x], r0 = tiles[2 * blockIdx.x + 1];
  const int len = p.e.len[en];
  if (len <= 1 || r0 >= len) return;
  const int nr = min(kSsmRows, len - r0);
  const long long start = p.e.start[en];
  const int pos0 = p.e.pos0[en], slot = p.e.slot[en];
  if (blockIdx.y == 0 && p.steps)
    for (int i = threadIdx.x; i < nr * p.H; i += kSsmConvThreads) {
      const long long row = start + r0 + i / p.H;
      p.steps[row * p.H + i % p.H] = ssm_step_of<T>(p, row, i % p.H);
    }
  const int channels = p.H * p.E + 2 * p.G * p.N;
  const int taps = TAPS ? TAPS : p.taps, hist = taps - 1;
  const float* old_h = nullptr;
  float* new_h = nullptr;
  if (hist > 0) {
    const int par = p.parity[slot] & 1;
    old_h = p.hist + (static_cast<long long>(slot) * 2 + par) * hist * channels;
    new_h = p.hist + (static_cast<long long>(slot) * 2 + (par ^ 1)) * hist * channels;
  }
  const T* in = static_cast<const T*>(p.p) + start * p.ld + p.xbc_col;
  const T* cw = static_cast<const T*>(p.conv_w);
  const T* cb = static_cast<const T*>(p.conv_b);
  const int c = (blockIdx.y * kSsmConvThreads + threadIdx.x) * 2;
  if (c >= channels) return;
  const bool pair = c + 1 < channels;
  // input of row r of the entry (negative rows come from the history or lie before the sequence)
  auto at = [&](int r, int ch) -> float {
    if (r >= 0) return to_f32(in[r * p.ld + ch]);
    return pos0 + r >= 0 ? old_h[static_cast<long long>(hist + r) * channels + ch] : 0.f;
  };
  auto at2 = [&](int r) -> float2 {
    if constexpr (sizeof(T) == 2) {
      if (r >= 0 && !((p.ld | p.xbc_col) & 1)) return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(in + r * p.ld + c));
    }
    return make_float2(at(r, c), pair ? at(r, c + 1) : 0.f);
  };
  T* out = static_cast<T*>(p.xbc) + (start + r0) * p.ldx + c;
  auto put = [&](int i, float2 v) {
    v = make_float2(silu_act<T>(v.x), silu_act<T>(v.y));
    if constexpr (sizeof(T) == 2) {
      *reinterpret_cast<uint32_t*>(out + i * p.ldx) = pack_bf16x2(v.x, v.y);     // ldx is even, the pad column exists
    } else {
      out[i * p.ldx] = v.x;
      if (pair) out[i * p.ldx + 1] = v.y;
    }
  };
  const float2 bias = cb ? make_float2(to_f32(cb[c]), pair ? to_f32(cb[c + 1]) : 0.f) : make_float2(0.f, 0.f);
  if constexpr (TAPS > 0) {
    constexpr int kHist = TAPS - 1;
    float2 w[TAPS], x[kHist + kSsmRows];
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
      w[j] = make_float2(to_f32(cw[static_cast<long long>(j) * channels + c]), pair ? to_f32(cw[static_cast<long long>(j) * channels + c + 1]) : 0.f);
#pragma unroll
    for (int i = 0; i < kHist + kSsmRows; ++i) x[i] = make_float2(0.f, 0.f);
    bool whole = false;                        // every row of the window is one of the entry's: loads without branches
    if constexpr (sizeof(T) == 2) {
      whole = r0 >= kHist && nr == kSsmRows && !((p.ld | p.xbc_col) & 1);
      if (whole) {
        const T* src = in + (r0 - kHist) * p.ld + c;
        uint32_t raw[kHist + kSsmRows];
#pragma unroll
        for (int i = 0; i < kHist + kSsmRows; ++i, src += p.ld) raw[i] = *reinterpret_cast<const uint32_t*>(src);
#pragma unroll
        for (int i = 0; i < kHist + kSsmRows; ++i) x[i] = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw[i]));
      }
    }
    if (!whole) {
#pragma unroll
      for (int i = 0; i < kHist + kSsmRows; ++i)
        if (i < kHist + nr) x[i] = at2(r0 - kHist + i);
    }
#pragma unroll
    for (int i = 0; i < kSsmRows; ++i)
      if (i < nr) {
        float2 v = bias;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
          v.x += w[j].x * x[i + j].x;
          v.y += w[j].y * x[i + j].y;
        }
        put(i, v);
      }
  } else {
    for (int i = 0; i < nr; ++i) {
      float2 v = bias;
      for (int j = 0; j < taps; ++j) {
        const float2 x = at2(r0 + i - hist + j);
        v.x += to_f32(cw[static_cast<long long>(j) * channels + c]) * x.x;
        if (pair) v.y += to_f32(cw[static_cast<long long>(j) * channels + c + 1]) * x.y;
      }
      put(i, v);
    }
  }
  if (new_h && r0 + nr == len)
    for (int i = 0; i < hist; ++i) {
      new_h[static_cast<long long>(i) * channels + c] = at(len - hist + i, c);
      if (pair) new_h[static_cast<long long>(i) * channels + c + 1] = at(len - hist + i, c + 1);
    }
}

// ---------------------------------------------------------------------------- recurrence of longer entries, fp32
constexpr int kSsmScanThreads = 256;
constexpr int kSsmScanCols = 32;

template <typename T>
__global__ void __launch_bounds__(kSsmScanThreads)
ssm_scan_kernel(const SsmParams p) {
  pdl_entry();
  extern __shared__ float ssm_smem[];
  const int en = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * kSsmScanCols;
  const int len = p.e.len[en];
  if (len <= 1) return;
  const int N = p.N, E = p.E, g = h / (p.H / p.G);
  float* S = ssm_smem;                         // [N][32]
  float* bs = S + N * kSsmScanCols;            // [N]
  float* cs = bs + N;                          // [N]
  float* red = cs + N;                         // [8][32]
  const long long start = p.e.start[en];
  const int slot = p.e.slot[en], lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int col = e0 + lane;
  const bool ok = col < E;
  float* Sg = p.state + (static_cast<long long>(slot) * p.H + h) * N * E;
  for (int d = warp; d < N; d += 8) S[d * kSsmScanCols + lane] = p.e.pos0[en] > 0 && ok ? Sg[static_cast<long long>(d) * E + col] : 0.f;
  const float skip = to_f32(static_cast<const T*>(p.d_skip)[h]);
  for (int t = 0; t < len; ++t) {
    const T* xr = static_cast<const T*>(p.xbc) + (start + t) * p.ldx;
    for (int i = threadIdx.x; i < 2 * N; i += kSsmScanThreads)
      bs[i] = to_f32(xr[p.H * E + (i < N ? g * N + i : (p.G + g) * N + i - N)]);
    const float2 st = p.steps[(start + t) * p.H + h];
    const float dec = exp2f(st.y), x = ok ? to_f32(xr[h * E + col]) : 0.f, dx = st.x * x;
    __syncthreads();
    float acc = 0.f;
    for (int d = warp; d < N; d += 8) {
      const float s = S[d * kSsmScanCols + lane] * dec + bs[d] * dx;
      S[d * kSsmScanCols + lane] = s;
      acc += s * cs[d];
    }
    red[threadIdx.x] = acc;
    __syncthreads();
    if (warp == 0 && ok) {
      float o = skip * x;
#pragma unroll
      for (int w = 0; w < 8; ++w) o += red[w * 32 + lane];
      p.y[(start + t) * p.H * E + static_cast<long long>(h) * E + col] = o;
    }
  }
  for (int d = warp; d < N; d += 8)
    if (ok) Sg[static_cast<long long>(d) * E + col] = S[d * kSsmScanCols + lane];
}

// ---------------------------------------------------------------------------- gate and norm
// out = w * (v / rms(v) per part), v = y silu(z): the gate comes before the norm.
struct GateNormParams {
  const float* y;           // [rows, inner]
  const void* z;            // [rows, inner] columns, row stride ldz
  long long ldz;
  const void* w;            // [inner]
  void* out;                // row stride ldo
  long long ldo;
  int rows, inner, parts;
  float eps;
};

__device__ __forceinline__ float4 gated4(const float* y, const __nv_bfloat16* z) {
  using T = __nv_bfloat16;
  const float4 v = __ldcs(reinterpret_cast<const float4*>(y));
  const uint2 raw = *reinterpret_cast<const uint2*>(z);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(v.x * silu_act<T>(a.x), v.y * silu_act<T>(a.y), v.z * silu_act<T>(b.x), v.w * silu_act<T>(b.y));
}
__device__ __forceinline__ void scaled4(__nv_bfloat16* out, const float4& v, float f, const __nv_bfloat16* w) {
  const uint2 raw = *reinterpret_cast<const uint2*>(w);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  *reinterpret_cast<uint2*>(out) = make_uint2(pack_bf16x2(v.x * f * a.x, v.y * f * a.y), pack_bf16x2(v.z * f * b.x, v.w * f * b.y));
}

// bf16, parts of a multiple of 4 up to 1024 columns, 8-byte aligned: one warp per (row, part).
constexpr int kGateWarpCols = 1024;

__global__ void __launch_bounds__(256)
gate_norm_warp_kernel(const GateNormParams p) {
  pdl_entry();
  const long long gw = (blockIdx.x * 256LL + threadIdx.x) >> 5;
  if (gw >= static_cast<long long>(p.rows) * p.parts) return;
  const int lane = threadIdx.x & 31, n = p.inner / p.parts, c0 = static_cast<int>(gw % p.parts) * n;
  const long long row = gw / p.parts;
  const float* y = p.y + row * p.inner + c0;
  const __nv_bfloat16* z = static_cast<const __nv_bfloat16*>(p.z) + row * p.ldz + c0;
  const __nv_bfloat16* w = static_cast<const __nv_bfloat16*>(p.w) + c0;
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + row * p.ldo + c0;
  float4 v[kGateWarpCols / 128];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < kGateWarpCols / 128; ++k) {
    const int i = k * 128 + lane * 4;
    v[k] = i < n ? gated4(y + i, z + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    ss += v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w;
  }
  const float f = 1.f / sqrtf(warp_sum(ss) / n + p.eps);
#pragma unroll
  for (int k = 0; k < kGateWarpCols / 128; ++k) {
    const int i = k * 128 + lane * 4;
    if (i < n) scaled4(out + i, v[k], f, w + i);
  }
}

// One block per (row, part), any size.  VEC: bf16 with the alignment of the kernel above.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
gate_norm_kernel(const GateNormParams p) {
  pdl_entry();
  extern __shared__ float ssm_smem[];          // [inner / parts]
  __shared__ float red[8];
  const int n = p.inner / p.parts, c0 = blockIdx.y * n;
  const long long row = blockIdx.x;
  const float* y = p.y + row * p.inner + c0;
  const T* z = static_cast<const T*>(p.z) + row * p.ldz + c0;
  const T* w = static_cast<const T*>(p.w) + c0;
  T* out = static_cast<T*>(p.out) + row * p.ldo + c0;
  float ss = 0.f;
  if constexpr (VEC) {
#pragma unroll 4
    for (int i = threadIdx.x * 4; i < n; i += 1024) {
      const float4 v = gated4(y + i, z + i);
      *reinterpret_cast<float4*>(ssm_smem + i) = v;
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
  } else {
    for (int i = threadIdx.x; i < n; i += 256) {
      const float v = y[i] * silu_act<T>(to_f32(z[i]));
      ssm_smem[i] = v;
      ss += v * v;
    }
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) ss += red[i];
  const float f = 1.f / sqrtf(ss / n + p.eps);
  if constexpr (VEC) {
    for (int i = threadIdx.x * 4; i < n; i += 1024) scaled4(out + i, *reinterpret_cast<const float4*>(ssm_smem + i), f, w + i);
  } else {
    for (int i = threadIdx.x; i < n; i += 256) out[i] = from_f32<T>(ssm_smem[i] * f * to_f32(w[i]));
  }
}

template <typename F>
static int ssm_smem_limit(F fn, size_t bytes) {
  if (bytes > 220 * 1024) return kBadArgument;
  return bytes <= 46 * 1024 ? 0 : static_cast<int>(cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes)));
}

static int ssm_conv_run(const SsmParams& a, int channels, const int* tiles, int n_tiles, int dtype, cudaStream_t s) {
  const dim3 grid(n_tiles, (channels + 2 * kSsmConvThreads - 1) / (2 * kSsmConvThreads));
  auto run = [&](auto fn) -> int { return static_cast<int>(launch_kernel(fn, grid, dim3(kSsmConvThreads), 0, s, a, tiles)); };
#define APB_SSM_CONV(T)                                                                                     \
  return a.taps == 2 ? run(ssm_conv_kernel<T, 2>) : a.taps == 3 ? run(ssm_conv_kernel<T, 3>) : a.taps == 4  \
           ? run(ssm_conv_kernel<T, 4>) : run(ssm_conv_kernel<T, 0>)
  if (dtype == 0) APB_SSM_CONV(__nv_bfloat16);
  if (dtype == 1) APB_SSM_CONV(float);
#undef APB_SSM_CONV
  return kBadArgument;
}

}  // namespace apb

extern "C" {
using namespace apb;

// Runs the one-token entries (decode != 0), the convolution of the longer ones (n_tiles > 0; xbc and steps are written) and /
// or their recurrence in fp32 (scan != 0).  y [rows, H * E] fp32.
int apb_ssm(const void* p, long long ld, int xbc_col, int dt_col, const void* conv_w, const void* conv_b, int taps, float* hist,
            const int* parity, const void* dt_bias, const void* a_log, const void* d_skip, void* xbc, long long ldx,
            void* steps, float* state, float* y, const int* e_start, const int* e_len, const int* e_slot, const int* e_pos0,
            int n_entries, const int* tiles, int n_tiles, int H, int E, int G, int N, int decode, int scan, int dtype,
            cudaStream_t s) {
  if (n_entries <= 0) return 0;
  if (H <= 0 || E <= 0 || G <= 0 || N <= 0 || H % G || taps < 1 || (taps > 1 && (!hist || !parity)) || !p || !state || !y ||
      (n_tiles > 0 && (!tiles || !xbc || !steps || (ldx & 1))) || (scan && n_tiles <= 0))
    return kBadArgument;
  SsmParams a{ServeEntries{e_start, e_len, e_slot, e_pos0}, p, ld, xbc_col, dt_col, conv_w, conv_b, taps, hist, parity, dt_bias,
              a_log, d_skip, xbc, ldx, static_cast<float2*>(steps), state, y, H, E, G, N};
  const int channels = H * E + 2 * G * N;
  if (decode) {
    const bool v4 = (E & 3) == 0;
    const int cols = v4 ? E / 4 : E, nx = cols < kSsmDecThreads ? cols : kSsmDecThreads;
    const size_t smem = (E + 2 * N + static_cast<size_t>(kSsmDecThreads / nx) * E) * sizeof(float);
    auto run = [&](auto fn) -> int {
      const int rc = ssm_smem_limit(fn, smem);
      return rc ? rc : static_cast<int>(launch_kernel(fn, dim3(n_entries, H), dim3(kSsmDecThreads), smem, s, a));
    };
    int rc = kBadArgument;
    if (dtype == 0) rc = v4 ? run(ssm_decode_kernel<__nv_bfloat16, 4>) : run(ssm_decode_kernel<__nv_bfloat16, 1>);
    if (dtype == 1) rc = v4 ? run(ssm_decode_kernel<float, 4>) : run(ssm_decode_kernel<float, 1>);
    if (rc) return rc;
  }
  if (n_tiles > 0) {
    const int rc = ssm_conv_run(a, channels, tiles, n_tiles, dtype, s);
    if (rc) return rc;
  }
  if (scan) {
    const size_t smem = (static_cast<size_t>(N) * (kSsmScanCols + 2) + kSsmScanThreads) * sizeof(float);
    auto run = [&](auto fn) -> int {
      const int rc = ssm_smem_limit(fn, smem);
      return rc ? rc : static_cast<int>(launch_kernel(fn, dim3(n_entries, H, (E + kSsmScanCols - 1) / kSsmScanCols), dim3(kSsmScanThreads), smem, s, a));
    };
    if (dtype == 0) return run(ssm_scan_kernel<__nv_bfloat16>);
    if (dtype == 1) return run(ssm_scan_kernel<float>);
    return kBadArgument;
  }
  return 0;
}

// The convolution alone, over `channels` columns from `col` on, for the entries longer than one token: out [rows, ldx] (ldx even) =
// silu(conv); bias may be null.
int apb_short_conv(const void* p, long long ld, int col, const void* conv_w, const void* bias, int taps, float* hist, const int* parity,
                   void* out, long long ldx, int channels, const int* e_start, const int* e_len, const int* e_slot, const int* e_pos0,
                   const int* tiles, int n_tiles, int dtype, cudaStream_t s) {
  if (n_tiles <= 0) return 0;
  if (!p || !conv_w || !out || !tiles || channels <= 0 || taps < 1 || (taps > 1 && (!hist || !parity)) || (ldx & 1)) return kBadArgument;
  SsmParams a{};
  a.e = ServeEntries{e_start, e_len, e_slot, e_pos0};
  a.p = p;
  a.ld = ld;
  a.xbc_col = col;
  a.conv_w = conv_w;
  a.conv_b = bias;
  a.taps = taps;
  a.hist = hist;
  a.parity = parity;
  a.xbc = out;
  a.ldx = ldx;
  a.H = 1;
  a.E = channels;
  return ssm_conv_run(a, channels, tiles, n_tiles, dtype, s);
}

// y [rows, inner] fp32, z [rows, inner] columns (row stride ldz), w [inner]; inner a multiple of parts.
int apb_ssm_out(const float* y, const void* z, long long ldz, const void* w, void* out, long long ldo, int rows, int inner,
                int parts, float eps, int dtype, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (inner <= 0 || parts <= 0 || inner % parts) return kBadArgument;
  const GateNormParams p{y, z, ldz, w, out, ldo, rows, inner, parts, eps};
  const int n = inner / parts;
  const bool vec = dtype == 0 && !(n & 3) && !((ldz | ldo) & 3) &&
                   !((reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(out)) & 7);
  if (vec && n <= kGateWarpCols)
    return static_cast<int>(launch_kernel(gate_norm_warp_kernel, dim3(static_cast<unsigned>((static_cast<long long>(rows) * parts + 7) / 8)),
                                          dim3(256), 0, s, p));
  const size_t smem = static_cast<size_t>(n) * sizeof(float);
  auto run = [&](auto fn) -> int {
    const int rc = ssm_smem_limit(fn, smem);
    return rc ? rc : static_cast<int>(launch_kernel(fn, dim3(rows, parts), dim3(256), smem, s, p));
  };
  if (vec) return run(gate_norm_kernel<__nv_bfloat16, true>);
  if (dtype == 0) return run(gate_norm_kernel<__nv_bfloat16, false>);
  if (dtype == 1) return run(gate_norm_kernel<float, false>);
  return kBadArgument;
}
}
