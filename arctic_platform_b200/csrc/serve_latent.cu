// Latent attention: the small steps around its products.
//
// A token keeps one latent of C columns and one rotated key part of R columns that all heads share; both lie side by side in a
// page row [pages, 1, 16, ldk] of at least C + R columns.  A head's keys and values are projections of the latent, so attention
// can run either on the expanded keys and values, or -- with the key projection moved to the query and the value projection
// behind the sum -- on the latents themselves.  Rotary positions pair neighbouring dimensions.
#include "common.cuh"
#include "host_utils.cuh"
#include "serve_common.cuh"

namespace apb {

constexpr int kLatThreads = 128;

__device__ __forceinline__ float block_sum_latent(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  v = 0.f;
#pragma unroll
  for (int i = 0; i < kLatThreads / 32; ++i) v += red[i];
  return v;
}

// p [rows, ld]: the query latent (Q columns at q_col) is normed in place; the key/value latent (C columns at c_col) is normed,
// the R columns behind it are rotated, and both go to the row's cache slot.  One block per row.
template <typename T>
__global__ void __launch_bounds__(kLatThreads)
latent_norm_cache_kernel(T* __restrict__ p, long long ld, int q_col, int c_col, const T* __restrict__ q_gain,
                         const T* __restrict__ c_gain, const int* __restrict__ row_entry, const ServeEntries e,
                         const int* __restrict__ kv_slot, const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                         T* __restrict__ cache, int ldk, int Q, int C, int R, float eps) {
  pdl_entry();
  __shared__ float red[2][kLatThreads / 32];
  const int row = blockIdx.x;
  T* pr = p + static_cast<long long>(row) * ld;
  T *q = pr + q_col, *c = pr + c_col;
  float ssq = 0.f, ssc = 0.f;
  for (int i = threadIdx.x; i < Q; i += kLatThreads) {
    const float v = to_f32(q[i]);
    ssq += v * v;
  }
  for (int i = threadIdx.x; i < C; i += kLatThreads) {
    const float v = to_f32(c[i]);
    ssc += v * v;
  }
  const float rq = 1.f / sqrtf(block_sum_latent(ssq, red[0]) / Q + eps), rc = 1.f / sqrtf(block_sum_latent(ssc, red[1]) / C + eps);
  for (int i = threadIdx.x; i < Q; i += kLatThreads) q[i] = from_f32<T>(to_f32(q[i]) * rq * to_f32(q_gain[i]));
  const int slot = kv_slot[row];
  if (slot < 0) return;
  T* dst = cache + static_cast<long long>(slot) * ldk;
  for (int i = threadIdx.x; i < C; i += kLatThreads) dst[i] = from_f32<T>(to_f32(c[i]) * rc * to_f32(c_gain[i]));
  const int en = row_entry ? row_entry[row] : row;
  const long long tr = static_cast<long long>(e.pos0[en] + row - e.start[en]) * (R >> 1);
  for (int i = threadIdx.x; i < (R >> 1); i += kLatThreads) {
    const float u = to_f32(c[C + 2 * i]), v = to_f32(c[C + 2 * i + 1]), cs = cos_t[tr + i], sn = sin_t[tr + i];
    dst[C + 2 * i] = from_f32<T>(u * cs - v * sn);
    dst[C + 2 * i + 1] = from_f32<T>(v * cs + u * sn);
  }
}

// The rotated part (R columns behind D) of every head of q [rows, H * (D + R)]: in place, or (dst) into column C of the head's
// row of dst [rows, H * (C + R)].  One thread per V pairs (V 4: 16-byte accesses, bf16).
template <typename T, int V>
__global__ void __launch_bounds__(256)
latent_rotate_kernel(T* __restrict__ q, long long ld, const int* __restrict__ row_entry, const ServeEntries e,
                     const float* __restrict__ cos_t, const float* __restrict__ sin_t, T* __restrict__ dst, int rows, int H,
                     int D, int R, int C) {
  pdl_entry();
  const int half = R >> 1, per = half / V;
  const long long idx = blockIdx.x * 256LL + threadIdx.x;
  if (idx >= static_cast<long long>(rows) * H * per) return;
  const int i = static_cast<int>(idx % per) * V, h = static_cast<int>(idx / per % H);
  const int row = static_cast<int>(idx / per / H);
  const int en = row_entry ? row_entry[row] : row;
  const int at = row - e.start[en];
  if (at < 0 || at >= e.len[en]) return;
  const long long tr = static_cast<long long>(e.pos0[en] + at) * half + i;
  T* src = q + static_cast<long long>(row) * ld + static_cast<long long>(h) * (D + R) + D + 2 * i;
  T* out = dst ? dst + (static_cast<long long>(row) * H + h) * (C + R) + C + 2 * i : src;
  if constexpr (V == 4) {
    const uint4 raw = *reinterpret_cast<const uint4*>(src);
    const float4 cs = *reinterpret_cast<const float4*>(cos_t + tr), sn = *reinterpret_cast<const float4*>(sin_t + tr);
    const uint32_t w[4] = {raw.x, raw.y, raw.z, raw.w};
    const float c[4] = {cs.x, cs.y, cs.z, cs.w}, s[4] = {sn.x, sn.y, sn.z, sn.w};
    uint32_t o[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w[j]));
      o[j] = pack_bf16x2(f.x * c[j] - f.y * s[j], f.y * c[j] + f.x * s[j]);
    }
    *reinterpret_cast<uint4*>(out) = make_uint4(o[0], o[1], o[2], o[3]);
  } else {
    const float u = to_f32(src[0]), v = to_f32(src[1]), cs = cos_t[tr], sn = sin_t[tr];
    out[0] = from_f32<T>(u * cs - v * sn);
    out[1] = from_f32<T>(v * cs + u * sn);
  }
}

// Page rows of some entries side by side: work [n][4] = entry, page of the entry, first row of the copy, tokens.
// latents [*, C], rotated [*, R].  One block per page.
template <typename V>
__global__ void __launch_bounds__(128)
latent_gather_kernel(const V* __restrict__ cache, const int* __restrict__ work, const int* __restrict__ page_table, int max_pages,
                     V* __restrict__ latents, V* __restrict__ rotated, int ldk, int C, int R) {
  pdl_entry();
  const int4 w = reinterpret_cast<const int4*>(work)[blockIdx.x];
  const V* src = cache + static_cast<long long>(page_table[static_cast<long long>(w.x) * max_pages + w.y]) * kServePage * ldk;
  for (int i = threadIdx.x; i < w.w * (C + R); i += 128) {
    const int t = i / (C + R), c = i % (C + R);
    const V v = src[t * ldk + c];
    if (c < C)
      latents[static_cast<long long>(w.z + t) * C + c] = v;
    else
      rotated[static_cast<long long>(w.z + t) * R + c - C] = v;
  }
}

}  // namespace apb

extern "C" {
using namespace apb;

int apb_latent_norm_cache(void* p, long long ld, int q_col, int c_col, const void* q_gain, const void* c_gain,
                          const int* row_entry, const int* e_start, const int* e_len, const int* e_slot, const int* e_pos0,
                          const int* kv_slot, const float* cos_t, const float* sin_t, void* cache, int ldk, int rows, int Q, int C,
                          int R, float eps, int dtype, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (Q <= 0 || C <= 0 || R < 0 || (R & 1) || ldk < C + R || !kv_slot || !cache || (R && (!cos_t || !sin_t))) return kBadArgument;
  const ServeEntries e{e_start, e_len, e_slot, e_pos0};
  APB_SERVE_DTYPE(dtype, return static_cast<int>(launch_kernel(
                             latent_norm_cache_kernel<T>, dim3(rows), dim3(kLatThreads), 0, s, static_cast<T*>(p), ld, q_col,
                             c_col, static_cast<const T*>(q_gain), static_cast<const T*>(c_gain), row_entry, e, kv_slot, cos_t,
                             sin_t, static_cast<T*>(cache), ldk, Q, C, R, eps)));
}

int apb_latent_rotate(void* q, long long ld, const int* row_entry, const int* e_start, const int* e_len, const int* e_slot,
                      const int* e_pos0, const float* cos_t, const float* sin_t, void* dst, int rows, int H, int D,
                      int R, int C, int dtype, cudaStream_t s) {
  if (rows <= 0 || R == 0) return 0;
  if (H <= 0 || D < 0 || R < 0 || (R & 1) || !cos_t || !sin_t) return kBadArgument;
  const ServeEntries e{e_start, e_len, e_slot, e_pos0};
  const bool vec = dtype == 0 && !((D | R | ld | (dst ? C : 0)) & 7) &&
                   !((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(dst) | reinterpret_cast<uintptr_t>(cos_t) |
                      reinterpret_cast<uintptr_t>(sin_t)) & 15);
  const long long n = static_cast<long long>(rows) * H * (R >> 1) / (vec ? 4 : 1);
  const dim3 grid(static_cast<unsigned>((n + 255) / 256));
#define APB_ROTATE(TT, VV)                                                                                                  \
  return static_cast<int>(launch_kernel(latent_rotate_kernel<TT, VV>, grid, dim3(256), 0, s, static_cast<TT*>(q), ld, row_entry, \
                                        e, cos_t, sin_t, static_cast<TT*>(dst), rows, H, D, R, C))
  if (vec) APB_ROTATE(__nv_bfloat16, 4);
  APB_SERVE_DTYPE(dtype, APB_ROTATE(T, 1));
#undef APB_ROTATE
}

// bf16; C, R and ldk multiples of 8.
int apb_latent_gather(const void* cache, const int* work, int n_work, const int* page_table, int max_pages, void* latents,
                      void* rotated, int ldk, int C, int R, cudaStream_t s) {
  if (n_work <= 0) return 0;
  if (C <= 0 || R < 0 || (C & 7) || (R & 7) || (ldk & 7) || ldk < C + R || !work || !page_table) return kBadArgument;
  return static_cast<int>(launch_kernel(latent_gather_kernel<uint4>, dim3(n_work), dim3(128), 0, s,
                                        static_cast<const uint4*>(cache), work, page_table, max_pages,
                                        static_cast<uint4*>(latents), static_cast<uint4*>(rotated), ldk / 8, C / 8, R / 8));
}
}
