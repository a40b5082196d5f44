// Warp-level pieces of the chunked recurrences on m16n8k16 tensor-core tiles (ssm_mma.cu, retention_mma.cu, memory_mma.cu,
// delta_mma.cu, time_mix_mma.cu): copies, fragment loads, products, and the split of an fp32 operand into two bf16 parts.
#pragma once
#include "common.cuh"

namespace apb {

// 16 bytes, or zeros when `bytes` is 0
__device__ __forceinline__ void wm_cp_async16(uint32_t dst, const void* src, int bytes) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void wm_ldsm4(const __nv_bfloat16* a, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(a)));
}
__device__ __forceinline__ void wm_ldsm4_t(const __nv_bfloat16* a, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(a)));
}
__device__ __forceinline__ void wm_ldsm2(const __nv_bfloat16* a, uint32_t (&r)[2]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0, %1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(smem_u32(a)));
}
__device__ __forceinline__ void wm_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// x = hi + lo with both parts bf16; two neighbouring elements packed per word
__device__ __forceinline__ void wm_split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  const float2 h = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&hi));
  lo = pack_bf16x2(x - h.x, y - h.y);
}
__device__ __forceinline__ void wm_store_split2(__nv_bfloat16* hi, __nv_bfloat16* lo, float x, float y) {
  uint32_t h, l;
  wm_split2(x, y, h, l);
  *reinterpret_cast<uint32_t*>(hi) = h;
  *reinterpret_cast<uint32_t*>(lo) = l;
}
// 2^x, results below the normal range are zero
__device__ __forceinline__ float wm_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float2 wm_pair(const __nv_bfloat16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
__device__ __forceinline__ float4 wm_quad(const __nv_bfloat16* p) {       // 8-byte aligned
  const uint2 r = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
  return make_float4(a.x, a.y, b.x, b.y);
}

// Segments of the entries of a batch, for recurrences whose segments can be chained (serving.segment_plan).
struct ScanSegments {
  const int* seg;         // [n][6]: entry, first token, tokens, scratch index of the state before it (-1: the slot's
                          // state or zero), scratch index for its own contribution (-1: none), 1 = last of its entry
  float* carry;           // [scratch states][H][D][E]
};

// The state of a chunked recurrence, 64 columns of it: warp w holds rows [16 w, 16 w + 16) as the accumulator fragments of eight
// 8-column tiles.
struct StateTile {
  float s[8][4];

  // rows below D, columns below be; src (row stride E, already at the first column) may be null: zeros
  __device__ __forceinline__ void load(const float* src, int E, int D, int be) {
    const int r0 = (threadIdx.x >> 5) * 16 + ((threadIdx.x & 31) >> 2), c0 = (threadIdx.x & 3) * 2;
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        const int d = r0 + 8 * hh, c = c0 + nt * 8;
        float2 v = make_float2(0.f, 0.f);
        if (src && d < D && c < be) v = *reinterpret_cast<const float2*>(src + static_cast<long long>(d) * E + c);
        s[nt][2 * hh] = v.x;
        s[nt][2 * hh + 1] = v.y;
      }
  }
  __device__ __forceinline__ void store(float* dst, int E, int D, int be) const {
    const int r0 = (threadIdx.x >> 5) * 16 + ((threadIdx.x & 31) >> 2), c0 = (threadIdx.x & 3) * 2;
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        const int d = r0 + 8 * hh, c = c0 + nt * 8;
        if (d < D && c < be) *reinterpret_cast<float2*>(dst + static_cast<long long>(d) * E + c) = make_float2(s[nt][2 * hh], s[nt][2 * hh + 1]);
      }
  }
  // the operand of the next chunk's product with the state
  __device__ __forceinline__ void split_to(__nv_bfloat16* hi, __nv_bfloat16* lo, int stride) const {
    const int r0 = (threadIdx.x >> 5) * 16 + ((threadIdx.x & 31) >> 2), c0 = (threadIdx.x & 3) * 2;
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        const int o = (r0 + 8 * hh) * stride + c0 + nt * 8;
        wm_store_split2(hi + o, lo + o, s[nt][2 * hh], s[nt][2 * hh + 1]);
      }
  }
  // rows of the first and second half of the tile times f0, f1
  __device__ __forceinline__ void scale(float f0, float f1) {
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) {
      s[nt][0] *= f0;
      s[nt][1] *= f0;
      s[nt][2] *= f1;
      s[nt][3] *= f1;
    }
  }
};

}  // namespace apb
