// Retention: linear attention with one fixed decay per head,
//     S_t = decay_h S_{t-1} + k_t v_t^T        (S [D, E] per head, fp32, carried from step to step in a state slot)
//     o_t = S_t^T q_t
// with rotary positions on q and k (first rot_dims dimensions, rotate-half pairs) and k scaled after the rotation, and
// the output stage  y = o / rms(o) * silu(g) * out_scale.  q, k, v and the gate g are columns of the step's projection
// buffer; rotation, decay powers, products and the state are fp32.
//
//  * retention_decode_kernel  entries of one token: streams the state of a (sequence, head) once (read, update, write)
//                             and finishes with the fused norm and gate -- bound by the bytes of the state;
//  * retention_chunk_kernel   longer entries, chunk by chunk: inside a chunk of C tokens the masked products
//                             (q_i . k_j) decay^(i-j), across chunks the carried state.  One CTA per (entry, head,
//                             32-column slice of E), fp32 CUDA-core arithmetic; followed by retention_out_kernel.
//
// bf16 engines run longer entries on tensor cores (retention_mma.cu).
#include "common.cuh"
#include "host_utils.cuh"
#include "retention.cuh"

namespace apb {

// ---------------------------------------------------------------------------- one token
constexpr int kRetDecThreads = 256;

template <typename T, int VEC>
__global__ void __launch_bounds__(kRetDecThreads)
retention_decode_kernel(const RetentionParams p) {
  pdl_entry();
  extern __shared__ float ret_smem[];
  const int en = blockIdx.x, h = blockIdx.y;
  if (p.e.len[en] != 1) return;
  const int D = p.D, E = p.E;
  float* qs = ret_smem;            // [D]
  float* ks = qs + D;              // [D]
  float* vs = ks + D;              // [E]
  float* red = vs + E;             // [ny][E]
  __shared__ float wsum[kRetDecThreads / 32];
  const int row = p.e.start[en], slot = p.e.slot[en], pos = p.e.pos0[en];
  const T* pr = static_cast<const T*>(p.p) + static_cast<long long>(row) * p.ld;
  const float* c = p.cos_t + static_cast<long long>(pos) * (p.rot_dims / 2);
  const float* sn = p.sin_t + static_cast<long long>(pos) * (p.rot_dims / 2);
  for (int d = threadIdx.x; d < D; d += kRetDecThreads) {
    qs[d] = rotated(pr + p.q_col + static_cast<long long>(h) * D, d, p.rot_dims, c, sn);
    ks[d] = rotated(pr + p.k_col + static_cast<long long>(h) * D, d, p.rot_dims, c, sn) * p.k_scale;
  }
  for (int i = threadIdx.x; i < E; i += kRetDecThreads)
    vs[i] = to_f32(pr[p.v_col + static_cast<long long>(h) * E + i]);
  __syncthreads();
  const float dec = pos == 0 ? 0.f : exp2f(p.log2_decay[h]);
  float* S = p.state + (static_cast<long long>(slot) * p.H + h) * D * E;
  const int nx = min(E / VEC, kRetDecThreads), ny = kRetDecThreads / nx;
  const int tx = threadIdx.x % nx, ty = threadIdx.x / nx;
  if (ty < ny) {
    for (int cx = tx; cx < E / VEC; cx += nx) {
      float acc[VEC], v[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        acc[i] = 0.f;
        v[i] = vs[cx * VEC + i];
      }
      if (pos == 0) {                // the slot may hold anything: write only
        for (int d = ty; d < D; d += ny) {
          float s[VEC];
#pragma unroll
          for (int i = 0; i < VEC; ++i) {
            s[i] = ks[d] * v[i];
            acc[i] += s[i] * qs[d];
          }
          if (VEC == 4)
            *reinterpret_cast<float4*>(S + static_cast<long long>(d) * E + cx * VEC) = make_float4(s[0], s[1 % VEC], s[2 % VEC], s[3 % VEC]);
          else
            S[static_cast<long long>(d) * E + cx] = s[0];
        }
      } else {
#pragma unroll 8
        for (int d = ty; d < D; d += ny) {
          float* sp = S + static_cast<long long>(d) * E + cx * VEC;
          float s[VEC];
          if (VEC == 4) {
            const float4 t = __ldcs(reinterpret_cast<const float4*>(sp));
            s[0] = t.x;
            s[1 % VEC] = t.y;
            s[2 % VEC] = t.z;
            s[3 % VEC] = t.w;
          } else {
            s[0] = *sp;
          }
          const float kd = ks[d], qd = qs[d];
#pragma unroll
          for (int i = 0; i < VEC; ++i) {
            s[i] = s[i] * dec + kd * v[i];
            acc[i] += s[i] * qd;
          }
          if (VEC == 4)
            __stcs(reinterpret_cast<float4*>(sp), make_float4(s[0], s[1 % VEC], s[2 % VEC], s[3 % VEC]));
          else
            *sp = s[0];
        }
      }
#pragma unroll
      for (int i = 0; i < VEC; ++i) red[ty * E + cx * VEC + i] = acc[i];
    }
  }
  __syncthreads();
  float ss = 0.f;
  for (int i = threadIdx.x; i < E; i += kRetDecThreads) {
    float o = 0.f;
    for (int y = 0; y < ny; ++y) o += red[y * E + i];
    red[i] = o;
    ss += o * o;
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) wsum[threadIdx.x >> 5] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < kRetDecThreads / 32; ++i) ss += wsum[i];
  const float f = p.out_scale / sqrtf(ss / E + p.eps);
  T* out = static_cast<T*>(p.out) + static_cast<long long>(row) * p.ldo + static_cast<long long>(h) * E;
  for (int i = threadIdx.x; i < E; i += kRetDecThreads) {
    const float g = to_f32(pr[p.g_col + static_cast<long long>(h) * E + i]);
    out[i] = from_f32<T>(red[i] * f * (g / (1.f + expf(-g))));
  }
}

// ---------------------------------------------------------------------------- chunks, fp32 arithmetic
constexpr int kRetThreads = 256;
constexpr int kRetC = 32;      // tokens per chunk
constexpr int kRetBE = 32;     // E columns per CTA

template <typename T>
__global__ void __launch_bounds__(kRetThreads)
retention_chunk_kernel(const RetentionParams p) {
  pdl_entry();
  extern __shared__ float ret_smem[];
  const int en = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * kRetBE;
  const int len = p.e.len[en];
  if (len <= 1) return;
  const int D = p.D, E = p.E, Dp = D + 1;
  float* S = ret_smem;                       // [D][32]
  float* Q = S + D * kRetBE;                 // [C][D + 1]
  float* K = Q + kRetC * Dp;                 // [C][D + 1]
  float* V = K + kRetC * Dp;                 // [C][32]
  float* A = V + kRetC * kRetBE;             // [C][C + 1]
  const int start = p.e.start[en], slot = p.e.slot[en], pos0 = p.e.pos0[en];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const float l2 = p.log2_decay[h];
  float* Sg = p.state + (static_cast<long long>(slot) * p.H + h) * D * E;
  for (int i = threadIdx.x; i < D * kRetBE; i += kRetThreads) {
    const int d = i >> 5, c = e0 + (i & 31);
    S[i] = (pos0 > 0 && c < E) ? Sg[static_cast<long long>(d) * E + c] : 0.f;
  }
  for (int t0 = 0; t0 < len; t0 += kRetC) {
    const int n = min(kRetC, len - t0);
    __syncthreads();
    for (int i = threadIdx.x; i < kRetC * D; i += kRetThreads) {
      const int r = i / D, d = i % D;
      float qv = 0.f, kv = 0.f;
      if (r < n) {
        const T* pr = static_cast<const T*>(p.p) + static_cast<long long>(start + t0 + r) * p.ld;
        const long long tr = static_cast<long long>(pos0 + t0 + r) * (p.rot_dims / 2);
        qv = rotated(pr + p.q_col + static_cast<long long>(h) * D, d, p.rot_dims, p.cos_t + tr, p.sin_t + tr);
        kv = rotated(pr + p.k_col + static_cast<long long>(h) * D, d, p.rot_dims, p.cos_t + tr, p.sin_t + tr) * p.k_scale;
      }
      Q[r * Dp + d] = qv;
      K[r * Dp + d] = kv;
    }
    for (int i = threadIdx.x; i < kRetC * kRetBE; i += kRetThreads) {
      const int r = i >> 5, c = e0 + (i & 31);
      V[i] = (r < n && c < E) ? to_f32(static_cast<const T*>(p.p)[static_cast<long long>(start + t0 + r) * p.ld + p.v_col + static_cast<long long>(h) * E + c]) : 0.f;
    }
    __syncthreads();
    // masked, decayed products inside the chunk: lane = key, warp = every 8th query
    for (int i = warp; i < kRetC; i += 8) {
      float a = 0.f;
      if (lane <= i) {
        for (int d = 0; d < D; ++d) a += Q[i * Dp + d] * K[lane * Dp + d];
        a *= decay_pow(l2, i - lane);
      }
      A[i * (kRetC + 1) + lane] = a;
    }
    __syncthreads();
    for (int i = warp; i < n; i += 8) {
      float o = 0.f;
      for (int d = 0; d < D; ++d) o += Q[i * Dp + d] * S[d * kRetBE + lane];
      o *= decay_pow(l2, i + 1);
      for (int j = 0; j <= i; ++j) o += A[i * (kRetC + 1) + j] * V[j * kRetBE + lane];
      if (e0 + lane < E) p.o[(static_cast<long long>(start + t0 + i) * p.H + h) * E + e0 + lane] = o;
    }
    __syncthreads();
    for (int j = warp; j < n; j += 8) V[j * kRetBE + lane] *= decay_pow(l2, n - 1 - j);
    __syncthreads();
    const float dn = decay_pow(l2, n);
    for (int d = warp; d < D; d += 8) {
      float s = S[d * kRetBE + lane] * dn;
      for (int j = 0; j < n; ++j) s += K[j * Dp + d] * V[j * kRetBE + lane];
      S[d * kRetBE + lane] = s;
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < D * kRetBE; i += kRetThreads) {
    const int d = i >> 5, c = e0 + (i & 31);
    if (c < E) Sg[static_cast<long long>(d) * E + c] = S[i];
  }
}

// y = o / rms(o) * silu(g) * out_scale for the rows of entries longer than one token; one warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(256)
retention_out_kernel(const RetentionParams p, const int* __restrict__ row_entry, int rows) {
  pdl_entry();
  const int lane = threadIdx.x & 31;
  const long long gw = (blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x) >> 5;
  if (gw >= static_cast<long long>(rows) * p.H) return;
  const int row = static_cast<int>(gw / p.H), h = static_cast<int>(gw % p.H);
  if (p.e.len[row_entry ? row_entry[row] : row] <= 1) return;
  const int E = p.E;
  const float* o = p.o + gw * E;
  const T* g = static_cast<const T*>(p.p) + static_cast<long long>(row) * p.ld + p.g_col + static_cast<long long>(h) * E;
  T* out = static_cast<T*>(p.out) + static_cast<long long>(row) * p.ldo + static_cast<long long>(h) * E;
  float ss = 0.f;
  if (sizeof(T) == 2 && (E & 3) == 0 && E <= 512 && ((reinterpret_cast<uintptr_t>(g) | reinterpret_cast<uintptr_t>(out)) & 7) == 0) {
    float4 v[4];                                    // four elements per lane and 128-column step
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int i = k * 128 + lane * 4;
      v[k] = i < E ? __ldcs(reinterpret_cast<const float4*>(o + i)) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w;
    }
    const float f = p.out_scale / sqrtf(warp_sum(ss) / E + p.eps);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int i = k * 128 + lane * 4;
      if (i >= E) continue;
      const uint2 gr = *reinterpret_cast<const uint2*>(g + i);
      const float2 g0 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gr.x));
      const float2 g1 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gr.y));
      uint2 r;
      r.x = pack_bf16x2(v[k].x * f * (g0.x / (1.f + expf(-g0.x))), v[k].y * f * (g0.y / (1.f + expf(-g0.y))));
      r.y = pack_bf16x2(v[k].z * f * (g1.x / (1.f + expf(-g1.x))), v[k].w * f * (g1.y / (1.f + expf(-g1.y))));
      *reinterpret_cast<uint2*>(out + i) = r;
    }
    return;
  }
  for (int i = lane; i < E; i += 32) ss += o[i] * o[i];
  const float f = p.out_scale / sqrtf(warp_sum(ss) / E + p.eps);
  for (int i = lane; i < E; i += 32) {
    const float gv = to_f32(g[i]);
    out[i] = from_f32<T>(o[i] * f * (gv / (1.f + expf(-gv))));
  }
}

static int retention_smem_limit(const void* fn, size_t bytes) {
  return bytes <= 48 * 1024 ? 0 : static_cast<int>(cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes)));
}

}  // namespace apb

extern "C" {
using namespace apb;

// Runs the one-token entries (decode != 0) and / or the longer entries (chunk != 0; o is fp32 scratch [rows, H, E]).
int apb_retention(const void* p, long long ld, int q_col, int k_col, int v_col, int g_col, const float* cos_t,
                  const float* sin_t, int rot_dims, const float* log2_decay, float k_scale, float* state, float* o,
                  void* out, long long ldo, float out_scale, float eps, const int* row_entry, const int* e_start,
                  const int* e_len, const int* e_slot, const int* e_pos0, int n_entries, int rows, int H, int D, int E,
                  int decode, int chunk, int dtype, cudaStream_t s) {
  if (rows <= 0 || n_entries <= 0) return 0;
  if (H <= 0 || D <= 0 || E <= 0 || D > 512 || (rot_dims & 1) || rot_dims > D || rot_dims < 0) return kBadArgument;
  RetentionParams a{};
  a.e = ServeEntries{e_start, e_len, e_slot, e_pos0};
  a.p = p;
  a.ld = ld;
  a.q_col = q_col;
  a.k_col = k_col;
  a.v_col = v_col;
  a.g_col = g_col;
  a.cos_t = cos_t;
  a.sin_t = sin_t;
  a.rot_dims = rot_dims;
  a.log2_decay = log2_decay;
  a.k_scale = k_scale;
  a.state = state;
  a.o = o;
  a.out = out;
  a.ldo = ldo;
  a.out_scale = out_scale;
  a.eps = eps;
  a.H = H;
  a.D = D;
  a.E = E;
  if (decode) {
    const bool v4 = (E & 3) == 0;
    const int cols = v4 ? E / 4 : E;
    const int nx = cols < kRetDecThreads ? cols : kRetDecThreads;
    const size_t smem = (2 * D + E + static_cast<size_t>(kRetDecThreads / nx) * E) * sizeof(float);
    int rc = 0;
    if (dtype == 0) {
      auto fn = v4 ? retention_decode_kernel<__nv_bfloat16, 4> : retention_decode_kernel<__nv_bfloat16, 1>;
      rc = retention_smem_limit(reinterpret_cast<const void*>(fn), smem);
      if (!rc) rc = static_cast<int>(launch_kernel(fn, dim3(n_entries, H), dim3(kRetDecThreads), smem, s, a));
    } else if (dtype == 1) {
      auto fn = v4 ? retention_decode_kernel<float, 4> : retention_decode_kernel<float, 1>;
      rc = retention_smem_limit(reinterpret_cast<const void*>(fn), smem);
      if (!rc) rc = static_cast<int>(launch_kernel(fn, dim3(n_entries, H), dim3(kRetDecThreads), smem, s, a));
    } else {
      rc = kBadArgument;
    }
    if (rc) return rc;
  }
  if (chunk) {
    if (!o) return kBadArgument;
    const size_t smem = (static_cast<size_t>(D) * kRetBE + 2 * kRetC * (D + 1) + kRetC * kRetBE + kRetC * (kRetC + 1)) * sizeof(float);
    const dim3 grid(n_entries, H, (E + kRetBE - 1) / kRetBE);
    const int og = static_cast<int>((static_cast<long long>(rows) * H * 32 + 255) / 256);
    auto run = [&](auto chunk_fn, auto out_fn) -> int {
      int rc = retention_smem_limit(reinterpret_cast<const void*>(chunk_fn), smem);
      if (rc) return rc;
      rc = static_cast<int>(launch_kernel(chunk_fn, grid, dim3(kRetThreads), smem, s, a));
      if (rc) return rc;
      return static_cast<int>(launch_kernel(out_fn, dim3(og), dim3(256), 0, s, a, row_entry, rows));
    };
    if (dtype == 0) return run(retention_chunk_kernel<__nv_bfloat16>, retention_out_kernel<__nv_bfloat16>);
    if (dtype == 1) return run(retention_chunk_kernel<float>, retention_out_kernel<float>);
    return kBadArgument;
  }
  return 0;
}

// The output stage alone, for o written by apb_retention_mma: out [rows, ldo] = o / rms(o) * silu(g) * out_scale for the
// rows of entries longer than one token.
int apb_retention_out(const void* p, long long ld, int g_col, float* o, void* out, long long ldo, float out_scale, float eps,
                      const int* row_entry, const int* e_start, const int* e_len, const int* e_slot, const int* e_pos0,
                      int rows, int H, int E, int dtype, cudaStream_t s) {
  if (rows <= 0) return 0;
  RetentionParams a{};
  a.e = ServeEntries{e_start, e_len, e_slot, e_pos0};
  a.p = p;
  a.ld = ld;
  a.g_col = g_col;
  a.o = o;
  a.out = out;
  a.ldo = ldo;
  a.out_scale = out_scale;
  a.eps = eps;
  a.H = H;
  a.E = E;
  const int grid = static_cast<int>((static_cast<long long>(rows) * H * 32 + 255) / 256);
  APB_SERVE_DTYPE(dtype, return static_cast<int>(launch_kernel(retention_out_kernel<T>, dim3(grid), dim3(256), 0, s, a, row_entry, rows)));
}
}
