// Parts shared by the softmax attention kernels on m16n8k16 tensor-core tiles.
#pragma once
#include "serve_softmax.cuh"

namespace apb {

struct SoftmaxMmaParams {
  const __nv_bfloat16* q;
  long long ldq;
  ServeEntries e;
  const int* page_table;
  int max_pages;
  const __nv_bfloat16* kcache;
  const __nv_bfloat16* vcache;    // unused where the values are the first E columns of the key rows
  __nv_bfloat16* out;
  long long ldo;
  float* part;            // [entries, max_len, H, maps, splits, E + 2] fp32 (sums, maximum, weight sum) when splits > 1
  int H, G, D, E, min_len, max_len;
  SoftmaxSpec sp;
};

__device__ __forceinline__ void sx_cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void sx_ldsm_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void sx_ldsm_x4_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void sx_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// The output stage of one (query, head): `read(a, c)` gives the normalised output of map a at column c, for the columns of
// this lane.  One warp.
template <typename F>
__device__ __forceinline__ void softmax_finish(const SoftmaxSpec& sp, int E, long long row, int head, __nv_bfloat16* dst,
                                               int lane, F read) {
  if (sp.maps == 1) {
    const bool per_head = sp.gate_cols == 1;
    const float g = per_head ? output_gate<__nv_bfloat16>(sp, row, head, 0) : 1.f;
    for (int c = lane; c < E; c += 32)
      dst[c] = __float2bfloat16(read(0, c) * (per_head ? g : output_gate<__nv_bfloat16>(sp, row, head, c)));
    return;
  }
  const float lam = *sp.lambda;
  float o[8], ss = 0.f;                      // E <= 256
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int c = lane + i * 32;
    o[i] = c < E ? read(0, c) - lam * read(1, c) : 0.f;
    ss += o[i] * o[i];
  }
  const float post = sp.post_scale / sqrtf(warp_sum(ss) / E + sp.eps);
#pragma unroll
  for (int i = 0; i < 8; ++i)
    if (lane + i * 32 < E) dst[lane + i * 32] = __float2bfloat16(o[i] * post);
}

// Combines the key splits that a kernel left in p.part.
int launch_softmax_merge(const SoftmaxMmaParams& p, int n_entries, int splits, cudaStream_t s);

}  // namespace apb
