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

// ---------------------------------------------------------------------------- tensor-core tiles for few queries
// One CTA = (entry, KV head, key split, pass group); a pass is 16 consecutive (query, head) rows of the entry: row f is
// query f / R, head f % R of the KV head's R query heads.  Each of the four warps owns every fourth page of the split's
// range, copies K and V pages with cp.async into its own 3-deep ring and runs S = Q K^T, O += sigmoid(S) V as m16n8k16
// MMAs; the warps' sums are added at the end.  Ring rows are an odd multiple of 16 bytes apart, so the 8 rows of an
// ldmatrix tile fall into different banks.
constexpr int kSmStages = 3;

struct SigmoidMmaParams {
  const __nv_bfloat16* q;
  long long ldq;
  ServeEntries e;
  const int* page_table;
  int max_pages;
  const __nv_bfloat16* kcache;
  const __nv_bfloat16* vcache;
  const __nv_bfloat16* bias;
  __nv_bfloat16* out;
  long long ldo;
  float* part;            // [entries, max_len, H, splits, E] fp32, used when splits > 1
  int H, G, D, E, min_len, max_len;
  float scale, out_scale;
};

__device__ __forceinline__ void sm_cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void sm_ldsm_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void sm_ldsm_x4_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void sm_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// N16: upper bound of D / 16 and E / 16; FULL: both are equal to it (the index arithmetic is then constant).
template <int N16, bool FULL>
__global__ void __launch_bounds__(kSigThreads)
sigmoid_attn_mma_kernel(const SigmoidMmaParams p) {
  pdl_entry();
  extern __shared__ __align__(128) uint8_t sm_ring[];
  const int en = blockIdx.x / p.G, g = blockIdx.x % p.G;
  const int len = p.e.len[en];
  if (len < p.min_len || len > p.max_len) return;
  const int D = FULL ? N16 * 16 : p.D, E = FULL ? N16 * 16 : p.E, R = p.H / p.G;
  const int d16 = (D + 15) >> 4, e16 = (E + 15) >> 4;
  const int k_row = d16 * 32 + 16, v_row = e16 * 32 + 16;            // ring row bytes
  const int stage_bytes = kServePage * (k_row + v_row);
  const int split = blockIdx.y, splits = gridDim.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int start = p.e.start[en], pos0 = p.e.pos0[en];
  const int* pages = p.page_table + static_cast<long long>(en) * p.max_pages;
  uint8_t* my_ring = sm_ring + warp * (kSmStages * stage_bytes);
  const uint32_t ring = smem_u32(my_ring);
  const int quad_row = lane >> 2, quad_col = (lane & 3) * 2;
  const int mat = lane >> 3, rowin = lane & 7;
  const int kc = D >> 3, vc = E >> 3;                                // 16-byte chunks of a cache row

  for (int f0 = blockIdx.z * 16; f0 < len * R; f0 += gridDim.z * 16) {
    const int q_last = (min(f0 + 16, len * R) - 1) / R;
    const int n_pages = (pos0 + q_last + kServePage) / kServePage;   // keys up to the last query of the pass
    const int per = (n_pages + splits - 1) / splits;
    const int p0 = split * per, p1 = min(n_pages, p0 + per);
    const int n_my = (p1 - p0 - warp + 3) / 4;
    // the half chunk that pads D to a multiple of 16 takes part in the products: zero it (copies never touch it)
    if (D & 8)
      for (int i = lane; i < kSmStages * kServePage; i += 32)
        *reinterpret_cast<uint4*>(my_ring + (i / kServePage) * stage_bytes + (i % kServePage) * k_row + D * 2) = make_uint4(0, 0, 0, 0);
    uint32_t qa[N16][4];
    int limit[2];
    float b[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int f = f0 + quad_row + 8 * h;
      const bool ok = f < len * R;
      const int qi = ok ? f / R : 0, head = g * R + (ok ? f % R : 0);
      limit[h] = ok ? pos0 + qi + 1 : 0;
      b[h] = __bfloat162float(p.bias[head]);
      const __nv_bfloat16* qp = p.q + static_cast<long long>(start + qi) * p.ldq + static_cast<long long>(head) * D;
#pragma unroll
      for (int ks = 0; ks < N16; ++ks) {
        const int c0 = ks * 16 + quad_col;
        qa[ks][h] = (ok && c0 < D) ? *reinterpret_cast<const uint32_t*>(qp + c0) : 0u;
        qa[ks][2 + h] = (ok && c0 + 8 < D) ? *reinterpret_cast<const uint32_t*>(qp + c0 + 8) : 0u;
      }
    }
    float o[2 * N16][4];
#pragma unroll
    for (int i = 0; i < 2 * N16; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;

    auto issue = [&](int j) {
      if (j < n_my) {
        const long long base = (static_cast<long long>(pages[p0 + warp + 4 * j]) * p.G + g) * kServePage;
        const uint32_t dst = ring + (j % kSmStages) * stage_bytes;
        const __nv_bfloat16* kp = p.kcache + base * D;
        const __nv_bfloat16* vp = p.vcache + base * E;
#pragma unroll
        for (int i = lane; i < kServePage * kc; i += 32) sm_cp_async16(dst + (i / kc) * k_row + (i % kc) * 16, kp + i * 8);
#pragma unroll
        for (int i = lane; i < kServePage * vc; i += 32)
          sm_cp_async16(dst + kServePage * k_row + (i / vc) * v_row + (i % vc) * 16, vp + i * 8);
      }
      asm volatile("cp.async.commit_group;" ::: "memory");
    };
#pragma unroll
    for (int j = 0; j < kSmStages - 1; ++j) issue(j);
#pragma unroll 1
    for (int j = 0; j < n_my; ++j) {
      issue(j + kSmStages - 1);
      asm volatile("cp.async.wait_group %0;" ::"n"(kSmStages - 1) : "memory");
      __syncwarp();
      const uint32_t ks_addr = ring + (j % kSmStages) * stage_bytes;
      const uint32_t vs_addr = ks_addr + kServePage * k_row;
      float sc[2][4];
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) sc[nt][0] = sc[nt][1] = sc[nt][2] = sc[nt][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < N16; ++ks)
        if (ks < d16) {
          uint32_t r[4];
          sm_ldsm_x4(ks_addr + (rowin + 8 * (mat >> 1)) * k_row + (ks * 2 + (mat & 1)) * 16, r);
          sm_mma(sc[0], qa[ks], r[0], r[1]);
          sm_mma(sc[1], qa[ks], r[2], r[3]);
        }
      const int key = (p0 + warp + 4 * j) * kServePage + quad_col;
      uint32_t pa[4];
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        float w[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float z = sc[i >> 1][2 * h + (i & 1)] * p.scale + b[h];
          w[i] = key + (i >> 1) * 8 + (i & 1) < limit[h] ? __fdividef(1.f, 1.f + __expf(-z)) : 0.f;
        }
        pa[h] = pack_bf16x2(w[0], w[1]);
        pa[2 + h] = pack_bf16x2(w[2], w[3]);
      }
#pragma unroll
      for (int dp = 0; dp < N16; ++dp)
        if (dp < e16) {
          uint32_t r[4];
          sm_ldsm_x4_t(vs_addr + (rowin + 8 * (mat & 1)) * v_row + (dp * 2 + (mat >> 1)) * 16, r);
          sm_mma(o[2 * dp], pa, r[0], r[1]);
          sm_mma(o[2 * dp + 1], pa, r[2], r[3]);
        }
      __syncwarp();
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                   // every warp is done with its ring: reuse it for the sums
    float* red = reinterpret_cast<float*>(sm_ring);    // [4][16][e16 * 16]
    const int ew = e16 * 16;
#pragma unroll
    for (int i = 0; i < 2 * N16; ++i)
      if (i < 2 * e16) {
#pragma unroll
        for (int h = 0; h < 2; ++h)
          *reinterpret_cast<float2*>(&red[(warp * 16 + quad_row + 8 * h) * ew + i * 8 + quad_col]) =
              make_float2(o[i][2 * h], o[i][2 * h + 1]);
      }
    __syncthreads();
    const int rows_valid = min(16, len * R - f0);
    for (int i = threadIdx.x; i < rows_valid * E; i += kSigThreads) {
      const int rr = i / E, c = i % E;
      const int f = f0 + rr, head = g * R + f % R;
      const long long row = start + f / R;
      const float v = (red[rr * ew + c] + red[(16 + rr) * ew + c]) + (red[(32 + rr) * ew + c] + red[(48 + rr) * ew + c]);
      if (splits > 1)
        p.part[(((static_cast<long long>(en) * p.max_len + f / R) * p.H + head) * splits + split) * E + c] = v;
      else
        p.out[row * p.ldo + static_cast<long long>(head) * E + c] = __float2bfloat16(v * p.out_scale);
    }
    __syncthreads();                                   // the ring is written again by the next pass
  }
}

// Adds the key splits of the rows handled by the kernel above.  One warp per (entry, query, head).
__global__ void __launch_bounds__(256)
sigmoid_merge_kernel(const SigmoidMmaParams p, int n_entries, int splits) {
  pdl_entry();
  const int lane = threadIdx.x & 31;
  const long long gw = (blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x) >> 5;
  if (gw >= static_cast<long long>(n_entries) * p.max_len * p.H) return;
  const int head = static_cast<int>(gw % p.H), qi = static_cast<int>(gw / p.H % p.max_len);
  const int en = static_cast<int>(gw / p.H / p.max_len), len = p.e.len[en];
  if (len < p.min_len || len > p.max_len || qi >= len) return;
  const long long row = p.e.start[en] + qi;
  const float* src = p.part + gw * splits * p.E;
  __nv_bfloat16* dst = p.out + row * p.ldo + static_cast<long long>(head) * p.E;
  for (int c = lane; c < p.E; c += 32) {
    float v = 0.f;
    for (int s = 0; s < splits; ++s) v += src[static_cast<long long>(s) * p.E + c];
    dst[c] = __float2bfloat16(v * p.out_scale);
  }
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

// bf16, D and E multiples of 8 up to 256, entries of min_len .. max_len rows (max_len: also the bound of the grid).
// part: fp32 scratch [entries, max_len, H, splits, E] when splits > 1.
int apb_sigmoid_attn_mma(const void* q, long long ldq, const int* e_start, const int* e_len,
                         const int* e_slot, const int* e_pos0, int n_entries, const int* page_table, int max_pages,
                         const void* kcache, const void* vcache, const void* bias, void* out, long long ldo, float* part,
                         int H, int G, int D, int E, int min_len, int max_len, int splits, float scale,
                         float out_scale, cudaStream_t s) {
  if (n_entries <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || D <= 0 || E <= 0 || (D % 8) || (E % 8) || D > 256 || E > 256 || (ldq % 8) ||
      (reinterpret_cast<uintptr_t>(q) & 15) || min_len < 1 || max_len < min_len || splits < 1 || (splits > 1 && !part))
    return kBadArgument;
  SigmoidMmaParams p{static_cast<const __nv_bfloat16*>(q), ldq, ServeEntries{e_start, e_len, e_slot, e_pos0}, page_table,
                     max_pages, static_cast<const __nv_bfloat16*>(kcache), static_cast<const __nv_bfloat16*>(vcache),
                     static_cast<const __nv_bfloat16*>(bias), static_cast<__nv_bfloat16*>(out), ldo, part, H, G, D, E,
                     min_len, max_len, scale, out_scale};
  const int d16 = (D + 15) / 16, e16 = (E + 15) / 16;
  const int smem = 4 * kSmStages * kServePage * (d16 * 32 + e16 * 32 + 32);
  const int passes = static_cast<int>((static_cast<long long>(max_len) * (H / G) + 15) / 16);
  const dim3 grid(n_entries * G, splits, passes < 256 ? passes : 256);
  auto run = [&](auto fn) -> int {
    if (smem > 48 * 1024) {
      const cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
      if (e != cudaSuccess) return static_cast<int>(e);
    }
    return static_cast<int>(launch_kernel(fn, grid, dim3(kSigThreads), smem, s, p));
  };
  const int n16 = d16 > e16 ? d16 : e16;
  const bool same = D == E;
  const int rc = same && D == 128 ? run(sigmoid_attn_mma_kernel<8, true>)
                 : same && D == 64 ? run(sigmoid_attn_mma_kernel<4, true>)
                 : n16 <= 4        ? run(sigmoid_attn_mma_kernel<4, false>)
                 : n16 <= 8        ? run(sigmoid_attn_mma_kernel<8, false>)
                                   : run(sigmoid_attn_mma_kernel<16, false>);
  if (rc || splits == 1) return rc;
  const int mg = static_cast<int>((static_cast<long long>(n_entries) * max_len * H * 32 + 255) / 256);
  return static_cast<int>(launch_kernel(sigmoid_merge_kernel, dim3(mg), dim3(256), 0, s, p, n_entries, splits));
}
}
