// Paged causal attention with sigmoid weights: key j <= i enters with weight sigmoid(scale * q_i . k_j + bias_h), no
// softmax and no normalisation over keys.  The outputs of disjoint key ranges therefore just add up.
//
// Keys and values live in pages of 16 tokens (kcache [pages, G, 16, D], vcache [pages, G, 16, E]); the step's own keys
// are already there when these kernels run, so prompts, portions of prompts and decoded tokens read the same memory.
//
//  * sigmoid_attn_kernel      any D and E up to 512, bf16 or fp32, fp32 arithmetic throughout (the fp32 engine, odd
//                             head sizes);
//  * sigmoid_attn_mma_kernel  bf16, D and E multiples of 8 up to 256: m16n8k16 tensor-core tiles whose 16 rows are
//                             (query, head of one KV head) pairs -- decoded tokens and short portions; the key range
//                             of one entry can be split over CTAs (fp32 partial sums, added by sigmoid_merge_kernel).
//
// Long portions run on tcgen05 (serve_attention_tc.cu).
#include "common.cuh"
#include "host_utils.cuh"
#include "serve_common.cuh"

namespace apb {

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }

// One CTA per (row, query head); its four warps take every fourth run of 32 keys.
constexpr int kSigThreads = 128;

template <typename T, int NV>
__global__ void __launch_bounds__(kSigThreads)
sigmoid_attn_kernel(const T* __restrict__ q, long long ldq, const int* __restrict__ row_entry, const ServeEntries e,
                    const int* __restrict__ page_table, int max_pages, const T* __restrict__ kcache,
                    const T* __restrict__ vcache, const T* __restrict__ bias, T* __restrict__ out, long long ldo, int H,
                    int G, int D, int E, float scale, float out_scale) {
  pdl_entry();
  extern __shared__ float sig_smem[];
  float* qs = sig_smem;                 // [D]
  float* red = sig_smem + D;            // [4][E]
  const int row = blockIdx.x, h = blockIdx.y, g = h / (H / G);
  const int en = row_entry ? row_entry[row] : row;
  const int r = row - e.start[en];
  if (r < 0 || r >= e.len[en]) return;
  const int n_keys = e.pos0[en] + r + 1;
  const int* pages = page_table + static_cast<long long>(en) * max_pages;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int i = threadIdx.x; i < D; i += kSigThreads)
    qs[i] = to_f32(q[static_cast<long long>(row) * ldq + static_cast<long long>(h) * D + i]);
  __syncthreads();
  const float b = to_f32(bias[h]);
  float acc[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) acc[i] = 0.f;
  for (int k0 = warp * 32; k0 < n_keys; k0 += 128) {
    const int key = k0 + lane;
    float p = 0.f;
    long long tok = 0;                  // (page, kv head, offset) row of the key
    if (key < n_keys) {
      tok = (static_cast<long long>(pages[key / kServePage]) * G + g) * kServePage + key % kServePage;
      const T* kp = kcache + tok * D;
      float s = 0.f;
      for (int d = 0; d < D; ++d) s += qs[d] * to_f32(kp[d]);
      p = sigmoid_f(s * scale + b);
    }
    const int n = min(32, n_keys - k0);
    for (int j = 0; j < n; ++j) {
      const float pj = __shfl_sync(0xffffffffu, p, j);
      const T* vp = vcache + __shfl_sync(0xffffffffu, tok, j) * E;
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (i * 32 + lane < E) acc[i] += pj * to_f32(vp[i * 32 + lane]);
    }
  }
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (i * 32 + lane < E) red[warp * E + i * 32 + lane] = acc[i];
  __syncthreads();
  for (int i = threadIdx.x; i < E; i += kSigThreads)
    out[static_cast<long long>(row) * ldo + static_cast<long long>(h) * E + i] =
        from_f32<T>((red[i] + red[E + i] + red[2 * E + i] + red[3 * E + i]) * out_scale);
}

}  // namespace apb

extern "C" {
using namespace apb;

// q [rows, H*D] (row stride ldq, already normalised), out [rows, H*E] (row stride ldo) = attention * out_scale.
// page_table [entries, max_pages]; row_entry [rows] or null (row i belongs to entry i).
int apb_sigmoid_attn(const void* q, long long ldq, const int* row_entry, const int* e_start, const int* e_len,
                     const int* e_slot, const int* e_pos0, const int* page_table, int max_pages, const void* kcache,
                     const void* vcache, const void* bias, void* out, long long ldo, int rows, int H, int G, int D,
                     int E, float scale, float out_scale, int dtype, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || D <= 0 || E <= 0 || D > 512 || E > 512) return kBadArgument;
  const ServeEntries e{e_start, e_len, e_slot, e_pos0};
  const size_t smem = (D + 4 * E) * sizeof(float);
#define APB_SIG(NVV)                                                                                                \
  return static_cast<int>(launch_kernel(sigmoid_attn_kernel<T, NVV>, dim3(rows, H), dim3(kSigThreads), smem, s,     \
                                        static_cast<const T*>(q), ldq, row_entry, e, page_table, max_pages,         \
                                        static_cast<const T*>(kcache), static_cast<const T*>(vcache),               \
                                        static_cast<const T*>(bias), static_cast<T*>(out), ldo, H, G, D, E, scale,  \
                                        out_scale))
  APB_SERVE_DTYPE(dtype, if (E <= 128) APB_SIG(4); APB_SIG(16));
#undef APB_SIG
}
}
