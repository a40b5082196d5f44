// Paged causal softmax attention over wide key rows whose first columns are the values (absorbed latent attention): decoded
// tokens and short portions, one map.  See SoftmaxSpec.
//
// Many query heads share one key row of up to 640 columns, so a row is read once and meets MT * 16 (query, head) rows on m16n8k16
// tensor-core tiles.  A CTA = one entry, KV head, group of rows and share of the keys; 8 warps.  Blocks of 64 keys (four pages)
// are double-buffered in shared memory and serve both products: for the scores the warps split rows and keys, for the weighted
// sums they split the value columns.  The running maximum and the weights pass through shared memory in between.
#include "common.cuh"
#include "host_utils.cuh"
#include "serve_softmax_mma.cuh"

namespace apb {

constexpr int kWideThreads = 256;
constexpr int kWideKeys = 64;
constexpr int kWideMaxDK = 640, kWideMaxE = 512;
constexpr int kWidePRow = kWideKeys * 2 + 16;          // bytes of a row of weights

template <int MT>
__global__ void __launch_bounds__(kWideThreads, 1)
softmax_attn_wide_kernel(const SoftmaxMmaParams p) {
  pdl_entry();
  extern __shared__ __align__(128) uint8_t smem[];
  constexpr int kRows = MT * 16;
  constexpr int kParts = MT == 2 ? 4 : 8;              // warps that share a row, by keys
  constexpr int kNt = MT == 2 ? 2 : 1;                 // key tiles of 8 per warp
  __shared__ float s_max[kRows][8], s_sum[kRows][8];
  const int en = blockIdx.x / p.G, g = blockIdx.x % p.G;
  const int len = p.e.len[en];
  if (len < p.min_len || len > p.max_len) return;
  const int DK = p.D, E = p.E, R = p.H / p.G;
  const int d16 = (DK + 15) >> 4, e16 = (E + 15) >> 4;
  const int row_b = d16 * 32 + 16;                     // bytes of a row of queries or keys
  const uint32_t sq = smem_u32(smem), sp = sq + kRows * row_b, sk = sp + kRows * kWidePRow;
  const int split = blockIdx.y, splits = gridDim.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int start = p.e.start[en], pos0 = p.e.pos0[en];
  const int* pages = p.page_table + static_cast<long long>(en) * p.max_pages;
  const int n_rows = len * R;
  const int mt = MT == 2 ? warp & 1 : 0, part = MT == 2 ? warp >> 1 : warp;
  const float scale = p.sp.scale * 1.4426950408889634f;

  for (int f0 = blockIdx.z * kRows; f0 < n_rows; f0 += gridDim.z * kRows) {
    const int q_first = f0 / R, q_last = (min(f0 + kRows, n_rows) - 1) / R;
    const int key_lo = visible_begin(pos0 + q_first, p.sp) / kServePage * kServePage, key_hi = pos0 + q_last + 1;
    const int blocks = (key_hi - key_lo + kWideKeys - 1) / kWideKeys, per = (blocks + splits - 1) / splits;
    const int b0 = split * per, b1 = min(blocks, b0 + per);
    const int last_page = (key_hi - 1) / kServePage;
    const int cols = d16 * 2;                          // 16-byte pieces of a row
    __syncthreads();                                   // the pass before has left the shared memory
    auto load_block = [&](int b) {
      const uint32_t dst = sk + (b & 1) * kWideKeys * row_b;
      const int k0 = key_lo + b * kWideKeys;
      for (int i = threadIdx.x; i < kWideKeys * cols; i += kWideThreads) {
        const int t = i / cols, c = i - t * cols;
        const int pg = min((k0 + t) / kServePage, last_page);            // beyond the last key: weight 0
        const __nv_bfloat16* src = p.kcache + ((static_cast<long long>(pages[pg]) * p.G + g) * kServePage + (t & (kServePage - 1))) * DK + c * 8;
        if (c * 8 < DK) sx_cp_async16(dst + t * row_b + c * 16, src);
      }
      asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (b0 < b1) load_block(b0);
    // queries; what lies behind the last column of queries and keys is zero
    for (int i = threadIdx.x; i < kRows * cols; i += kWideThreads) {
      const int r = i / cols, c = i - r * cols, f = f0 + r;
      uint4 v = make_uint4(0, 0, 0, 0);
      if (f < n_rows && c * 8 < DK)
        v = *reinterpret_cast<const uint4*>(p.q + static_cast<long long>(start + f / R) * p.ldq + static_cast<long long>(g * R + f % R) * DK + c * 8);
      *reinterpret_cast<uint4*>(smem + r * row_b + c * 16) = v;
    }
    if (cols * 8 > DK)
      for (int t = threadIdx.x; t < 2 * kWideKeys; t += kWideThreads)
        *reinterpret_cast<uint4*>(smem + (sk - sq) + t * row_b + (cols - 1) * 16) = make_uint4(0, 0, 0, 0);

    // rows of this thread, for its score tile and for all tiles of the sums
    int hi[2], lo[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int f = f0 + mt * 16 + (lane >> 2) + 8 * h;
      hi[h] = f < n_rows ? pos0 + f / R : -1;
      lo[h] = f < n_rows ? visible_begin(pos0 + f / R, p.sp) : 0;
    }
    float mx[MT][2], sum[2] = {0.f, 0.f};
    float acc[MT][4][2][4];                            // value tiles warp, warp + 8, ... of 16 columns
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      mx[m][0] = mx[m][1] = -INFINITY;
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int n = 0; n < 2; ++n) acc[m][i][n][0] = acc[m][i][n][1] = acc[m][i][n][2] = acc[m][i][n][3] = 0.f;
    }

    for (int b = b0; b < b1; ++b) {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
      __syncthreads();                                 // block b is there, block b - 1 has been used
      if (b + 1 < b1) load_block(b + 1);
      const uint32_t kb = sk + (b & 1) * kWideKeys * row_b;
      const int k0 = key_lo + b * kWideKeys;
      // ---- scores: rows of tile mt, keys [part * 8 kNt, +8 kNt)
      float sc[2][kNt][4];                             // two chains per tile
#pragma unroll
      for (int a = 0; a < 2; ++a)
#pragma unroll
        for (int n = 0; n < kNt; ++n) sc[a][n][0] = sc[a][n][1] = sc[a][n][2] = sc[a][n][3] = 0.f;
      const uint32_t qa = sq + (mt * 16 + (lane & 15)) * row_b + (lane >> 4) * 16;
      if (kNt == 2) {
        const uint32_t ka = kb + (part * 16 + (lane & 7) + ((lane >> 4) << 3)) * row_b + ((lane >> 3) & 1) * 16;
#pragma unroll 4
        for (int k = 0; k < d16; ++k) {
          uint32_t a[4], v[4];
          sx_ldsm_x4(qa + k * 32, a);
          sx_ldsm_x4(ka + k * 32, v);
          if (k & 1) {
            sx_mma(sc[1][0], a, v[0], v[1]);
            sx_mma(sc[1][kNt - 1], a, v[2], v[3]);
          } else {
            sx_mma(sc[0][0], a, v[0], v[1]);
            sx_mma(sc[0][kNt - 1], a, v[2], v[3]);
          }
        }
      } else {                                         // 8 keys: one load covers 32 columns
        const uint32_t ka = kb + (part * 8 + (lane & 7)) * row_b + (lane >> 3) * 16;
#pragma unroll 4
        for (int k = 0; k < d16; k += 2) {
          uint32_t a[4], v[4];
          sx_ldsm_x4(qa + k * 32, a);
          // an odd last step reads 32 bytes behind the row: the next row's, or the margin behind the last one
          sx_ldsm_x4(ka + k * 32, v);
          sx_mma(sc[0][0], a, v[0], v[1]);
          if (k + 1 < d16) {
            sx_ldsm_x4(qa + k * 32 + 32, a);
            sx_mma(sc[1][0], a, v[2], v[3]);
          }
        }
      }
      float top[2] = {-INFINITY, -INFINITY}, s[kNt][4];
#pragma unroll
      for (int n = 0; n < kNt; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int key = k0 + part * 8 * kNt + n * 8 + (lane & 3) * 2 + (i & 1), h = i >> 1;
          s[n][i] = key <= hi[h] && key >= lo[h] ? (sc[0][n][i] + sc[1][n][i]) * scale : -INFINITY;
          top[h] = fmaxf(top[h], s[n][i]);
        }
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        top[h] = fmaxf(top[h], __shfl_xor_sync(0xffffffffu, top[h], 1));
        top[h] = fmaxf(top[h], __shfl_xor_sync(0xffffffffu, top[h], 2));
        if ((lane & 3) == 0) s_max[mt * 16 + (lane >> 2) + 8 * h][part] = top[h];
      }
      __syncthreads();
      float fac[MT][2];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          float t = mx[m][h];
#pragma unroll
          for (int w = 0; w < kParts; ++w) t = fmaxf(t, s_max[m * 16 + (lane >> 2) + 8 * h][w]);
          fac[m][h] = t == -INFINITY ? 1.f : exp2f(mx[m][h] - t);
          mx[m][h] = t;
        }
      float ref[2], fmine[2];
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        ref[h] = MT == 2 && mt ? mx[MT - 1][h] : mx[0][h];
        fmine[h] = MT == 2 && mt ? fac[MT - 1][h] : fac[0][h];
        if (ref[h] == -INFINITY) ref[h] = 0.f;
        sum[h] *= fmine[h];
      }
#pragma unroll
      for (int n = 0; n < kNt; ++n) {
        float w[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          w[i] = exp2f(s[n][i] - ref[i >> 1]);
          sum[i >> 1] += w[i];
        }
        uint8_t* dst = smem + (sp - sq) + (mt * 16 + (lane >> 2)) * kWidePRow + (part * 8 * kNt + n * 8 + (lane & 3) * 2) * 2;
        *reinterpret_cast<uint32_t*>(dst) = pack_bf16x2(w[0], w[1]);
        *reinterpret_cast<uint32_t*>(dst + 8 * kWidePRow) = pack_bf16x2(w[2], w[3]);
      }
      __syncthreads();
      // ---- weighted sums: all rows, this warp's value tiles
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int q = 0; q < 4; ++q) acc[m][i][n][q] *= fac[m][q >> 1];
#pragma unroll
      for (int k = 0; k < kWideKeys / 16; ++k) {
        uint32_t a[MT][4];
#pragma unroll
        for (int m = 0; m < MT; ++m) sx_ldsm_x4(sp + (m * 16 + (lane & 15)) * kWidePRow + k * 32 + (lane >> 4) * 16, a[m]);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int tile = warp + 8 * i;
          if (tile >= e16) break;
          uint32_t v[4];
          sx_ldsm_x4_t(kb + (k * 16 + (lane & 15)) * row_b + tile * 32 + (lane >> 4) * 16, v);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            sx_mma(acc[m][i][0], a[m], v[0], v[1]);
            sx_mma(acc[m][i][1], a[m], v[2], v[3]);
          }
        }
      }
    }
    // ---- output
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      sum[h] += __shfl_xor_sync(0xffffffffu, sum[h], 1);
      sum[h] += __shfl_xor_sync(0xffffffffu, sum[h], 2);
      if ((lane & 3) == 0) s_sum[mt * 16 + (lane >> 2) + 8 * h][part] = sum[h];
    }
    __syncthreads();
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int rr = m * 16 + (lane >> 2) + 8 * h, f = f0 + rr;
        if (f >= n_rows) continue;
        float total = 0.f;
#pragma unroll
        for (int w = 0; w < kParts; ++w) total += s_sum[rr][w];
        const int qi = f / R, head = g * R + f % R;
        if (splits > 1) {
          float* dst = p.part + (((static_cast<long long>(en) * p.max_len + qi) * p.H + head) * splits + split) * (E + 2);
#pragma unroll
          for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int n = 0; n < 2; ++n) {
              const int c = (warp + 8 * i) * 16 + n * 8 + (lane & 3) * 2;
              if (c < E) *reinterpret_cast<float2*>(dst + c) = make_float2(acc[m][i][n][2 * h], acc[m][i][n][2 * h + 1]);
            }
          if (warp == 0 && (lane & 3) == 0) {
            dst[E] = mx[m][h];
            dst[E + 1] = total;
          }
        } else {
          const long long row = start + qi;
          const bool per_column = p.sp.gate && p.sp.gate_cols != 1;
          const float inv = inverse_sum(p.sp, head, mx[m][h], total) * (per_column ? 1.f : output_gate<__nv_bfloat16>(p.sp, row, head, 0));
          __nv_bfloat16* dst = p.out + row * p.ldo + static_cast<long long>(head) * E;
#pragma unroll
          for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int n = 0; n < 2; ++n) {
              const int c = (warp + 8 * i) * 16 + n * 8 + (lane & 3) * 2;
              if (c >= E) continue;
              float u = acc[m][i][n][2 * h] * inv, v = acc[m][i][n][2 * h + 1] * inv;
              if (per_column) {
                u *= output_gate<__nv_bfloat16>(p.sp, row, head, c);
                v *= output_gate<__nv_bfloat16>(p.sp, row, head, c + 1);
              }
              *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16x2(u, v);
            }
        }
      }
  }
}

}  // namespace apb

extern "C" {

// bf16; kcache [pages, G, 16, D] whose first E columns are the values; D and E multiples of 8, D up to 640, E up to 512; entries of
// min_len .. max_len rows.  part: fp32 scratch [entries, max_len, H, splits, E + 2] when splits > 1.
int apb_softmax_attn_wide(const void* q, long long ldq, const int* e_start, const int* e_len, const int* e_slot, const int* e_pos0,
                          int n_entries, const int* page_table, int max_pages, const void* kcache, void* out, long long ldo,
                          float* part, int H, int G, int D, int E, int min_len, int max_len, int splits, float scale, int window,
                          const float* sink, const void* gate, long long ldg, int gate_cols, cudaStream_t s) {
  using namespace apb;
  if (n_entries <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || E <= 0 || E > D || (D % 8) || (E % 8) || D > kWideMaxDK || E > kWideMaxE || (ldq % 8) || (ldo % 2) ||
      ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(kcache)) & 15) || (reinterpret_cast<uintptr_t>(out) & 3) ||
      min_len < 1 || max_len < min_len || splits < 1 || (splits > 1 && !part) || window < 0 || (gate && gate_cols != 1 && gate_cols != E))
    return kBadArgument;
  const SoftmaxMmaParams p{static_cast<const __nv_bfloat16*>(q), ldq, ServeEntries{e_start, e_len, e_slot, e_pos0}, page_table, max_pages,
                           static_cast<const __nv_bfloat16*>(kcache), nullptr, static_cast<__nv_bfloat16*>(out), ldo, part, H, G, D, E,
                           min_len, max_len, SoftmaxSpec{scale, 0.f, 0, 1, nullptr, 1.f, 0.f, window, sink, gate, ldg, gate_cols}};
  const long long rows = static_cast<long long>(max_len) * (H / G);
  const int mt = rows > 16 ? 2 : 1, row_b = (D + 15) / 16 * 32 + 16;
  const int smem = mt * 16 * (row_b + kWidePRow) + 2 * kWideKeys * row_b + 64;
  const long long passes = (rows + mt * 16 - 1) / (mt * 16);
  const dim3 grid(n_entries * G, splits, static_cast<unsigned>(passes < 1024 ? passes : 1024));
  auto run = [&](auto fn) -> int {
    const cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    return static_cast<int>(launch_kernel(fn, grid, dim3(kWideThreads), smem, s, p));
  };
  const int rc = mt == 2 ? run(softmax_attn_wide_kernel<2>) : run(softmax_attn_wide_kernel<1>);
  return rc || splits == 1 ? rc : launch_softmax_merge(p, n_entries, splits, s);
}
}
