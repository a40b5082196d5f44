// Paged causal softmax attention over wide key rows whose first columns are the values (absorbed latent attention): decoded
// tokens and short portions, one map.  See SoftmaxSpec.
//
// A key row lies in the page cache as in shared memory: its columns, zeros up to a multiple of 16 and 8 columns more, an odd number
// of 16-byte pieces, so that the rows of a page arrive by one copy and fall into different banks.
//
// Many query heads share one key row of up to 640 columns, so a row is read once and meets MT * 16 (query, head) rows on m16n8k16
// tensor-core tiles.  A CTA = one entry, KV head, group of rows and share of the keys.  13 warps: a producer that copies pages into
// a ring, four score warps and eight value warps.  A page serves both products.  The score warps take the pages in turn: each
// computes a page's scores for all rows, then -- in the order of the pages -- moves the rows' running maximum, and leaves weights
// and rescaling factors in shared memory; the value warps split the value columns and follow page by page.
#include "common.cuh"
#include "host_utils.cuh"
#include "serve_softmax_mma.cuh"

namespace apb {

constexpr int kWideThreads = 13 * 32;
constexpr int kWideScore = 4;                          // score warps
constexpr int kWideMaxStages = 12;
constexpr int kWideMaxSmem = 227 * 1024 - 3 * 1024;    // besides the static arrays
constexpr int kWideMaxDK = 640, kWideMaxE = 512;
constexpr int kWidePRow = kServePage * 2 + 16;         // bytes of a row of weights

// Contiguous bytes (a multiple of 16, both ends 16-byte aligned) to shared memory; counts on `bar`.
__device__ __forceinline__ void bulk_load(uint32_t dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src),
               "r"(bytes), "r"(smem_u32(bar))
               : "memory");
}

// A wait that runs out is recorded, and the loops go on without waiting: the block ends and frees what it holds.
struct WideWait {
  int* status;
  bool ok = true;
  __device__ __forceinline__ void operator()(uint64_t* bar, uint32_t parity, int code) {
    if (ok) ok = mbar_wait(bar, parity, status, code);
    __syncwarp();
  }
};

template <int MT>
__global__ void __launch_bounds__(kWideThreads, 1)
softmax_attn_wide_kernel(const SoftmaxMmaParams p, const int stages, int* status) {
  pdl_entry();
  extern __shared__ __align__(128) uint8_t smem[];
  constexpr int kRows = MT * 16;
  __shared__ float s_run[kRows], s_fac[kWideScore][kRows], s_sum[kWideScore][kRows], s_last[kWideScore][kRows];
  __shared__ uint64_t full[kWideMaxStages], empty[kWideMaxStages], p_full[kWideScore], p_empty[kWideScore], turn[kWideScore];
  const int en = blockIdx.x / p.G, g = blockIdx.x % p.G;
  const int len = p.e.len[en];
  if (len < p.min_len || len > p.max_len) return;
  const int DK = p.D, E = p.E, R = p.H / p.G;
  const int n_rows = len * R, f0 = blockIdx.z * kRows;
  if (f0 >= n_rows) return;
  const int d16 = (DK + 15) >> 4, e16 = (E + 15) >> 4;
  const int row_b = d16 * 32 + 16;                     // bytes of a row of queries or keys
  const uint32_t sq = smem_u32(smem), sp = sq + kRows * row_b, sk = sp + kWideScore * kRows * kWidePRow;
  const int split = blockIdx.y, splits = gridDim.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int start = p.e.start[en], pos0 = p.e.pos0[en];
  const int q_first = f0 / R, q_last = (min(f0 + kRows, n_rows) - 1) / R;
  const int page_lo = visible_begin(pos0 + q_first, p.sp) / kServePage, page_hi = (pos0 + q_last) / kServePage + 1;
  const int per = (page_hi - page_lo + splits - 1) / splits;
  const int b0 = page_lo + split * per, n = max(0, min(page_hi, b0 + per) - b0);        // pages [b0, b0 + n)
  const int cols = d16 * 2;                            // 16-byte pieces of a row

  if (threadIdx.x == 0) {
    for (int i = 0; i < stages; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 8);
    }
    for (int i = 0; i < kWideScore; ++i) {
      mbar_init(&p_full[i], 1);
      mbar_init(&p_empty[i], 8);
      mbar_init(&turn[i], 1);
    }
    mbar_fence_init();
    mbar_arrive(&turn[0]);
  }
  if (threadIdx.x < kRows) s_run[threadIdx.x] = -INFINITY;
  // queries; zeros behind the last column
  for (int i = threadIdx.x; i < kRows * cols; i += kWideThreads) {
    const int r = i / cols, c = i - r * cols, f = f0 + r;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (f < n_rows && c * 8 < DK)
      v = *reinterpret_cast<const uint4*>(p.q + static_cast<long long>(start + f / R) * p.ldq +
                                          static_cast<long long>(g * R + f % R) * DK + c * 8);
    *reinterpret_cast<uint4*>(smem + r * row_b + c * 16) = v;
  }
  __syncthreads();

  WideWait wait{status};
  if (warp == 12) {
    // ---------------------------------------------------------------- producer
    if (lane == 0) {
      const int* pages = p.page_table + static_cast<long long>(en) * p.max_pages;
      for (int i = 0, stage = 0, phase = 1; i < n; ++i) {
        const int pg = pages[b0 + i];
        if (!mbar_wait(&empty[stage], phase, status, kTimeoutEmpty)) {
          wait.ok = false;
          break;
        }
        mbar_expect_tx(&full[stage], kServePage * row_b);
        bulk_load(sk + stage * kServePage * row_b, p.kcache + (static_cast<long long>(pg) * p.G + g) * kServePage * (row_b / 2),
                  kServePage * row_b, &full[stage]);
        if (++stage == stages) stage = 0, phase ^= 1;
      }
    }
    if (!wait.ok) {                    // give copies in flight time to land before the block ends
      const uint64_t t0 = global_timer_ns();
      while (global_timer_ns() - t0 < 100000ull) {
      }
    }
  } else if (warp < kWideScore) {
    // ---------------------------------------------------------------- scores of the pages warp, warp + 4, ...; all rows
    const float scale = p.sp.scale * 1.4426950408889634f;
    int hi[MT][2], lo[MT][2];
    float last[MT][2], sum[MT][2];                     // this warp's share of the weight sums, relative to 2^last
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int f = f0 + m * 16 + (lane >> 2) + 8 * h;
        hi[m][h] = f < n_rows ? pos0 + f / R : -1;
        lo[m][h] = f < n_rows ? visible_begin(pos0 + f / R, p.sp) : 0;
        last[m][h] = -INFINITY;
        sum[m][h] = 0.f;
      }
    const uint32_t qa = sq + (lane & 15) * row_b + (lane >> 4) * 16;
    const uint32_t k_off = ((lane & 7) + ((lane >> 4) << 3)) * row_b + ((lane >> 3) & 1) * 16;
    for (int j = warp; j < n; j += kWideScore) {
      const int stage = j % stages, turns = j / kWideScore;
      wait(&full[stage], (j / stages) & 1, kTimeoutFull);
      const uint32_t ka = sk + stage * kServePage * row_b + k_off;
      float sc[2][MT][2][4];                           // two chains per tile
#pragma unroll
      for (int c = 0; c < 2; ++c)
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int t = 0; t < 2; ++t) sc[c][m][t][0] = sc[c][m][t][1] = sc[c][m][t][2] = sc[c][m][t][3] = 0.f;
      auto steps = [&](int k, int c) {
        uint32_t v[4], a[MT][4];
        sx_ldsm_x4(ka + k * 32, v);
#pragma unroll
        for (int m = 0; m < MT; ++m) sx_ldsm_x4(qa + m * 16 * row_b + k * 32, a[m]);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          sx_mma(sc[c][m][0], a[m], v[0], v[1]);
          sx_mma(sc[c][m][1], a[m], v[2], v[3]);
        }
      };
      int k = 0;
#pragma unroll 3
      for (; k + 1 < d16; k += 2) {
        steps(k, 0);
        steps(k + 1, 1);
      }
      if (k < d16) steps(k, 0);
      const int key0 = (b0 + j) * kServePage + (lane & 3) * 2;
      float s[MT][2][4], top[MT][2];
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        top[m][0] = top[m][1] = -INFINITY;
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            const int key = key0 + t * 8 + (q & 1), h = q >> 1;
            s[m][t][q] = key <= hi[m][h] && key >= lo[m][h] ? (sc[0][m][t][q] + sc[1][m][t][q]) * scale : -INFINITY;
            top[m][h] = fmaxf(top[m][h], s[m][t][q]);
          }
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          top[m][h] = fmaxf(top[m][h], __shfl_xor_sync(0xffffffffu, top[m][h], 1));
          top[m][h] = fmaxf(top[m][h], __shfl_xor_sync(0xffffffffu, top[m][h], 2));
        }
      }
      // ---- in the order of the pages: the running maximum
      wait(&turn[warp], turns & 1, kTimeoutFull);
      float before[MT][2];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          before[m][h] = s_run[m * 16 + (lane >> 2) + 8 * h];
          top[m][h] = fmaxf(top[m][h], before[m][h]);
        }
      __syncwarp();
      if ((lane & 3) == 0)
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int h = 0; h < 2; ++h) s_run[m * 16 + (lane >> 2) + 8 * h] = top[m][h];
      __syncwarp();
      if (lane == 0) mbar_arrive(&turn[(warp + 1) % kWideScore]);
      // ---- weights
      wait(&p_empty[warp], (turns & 1) ^ 1, kTimeoutEmpty);                    // this warp's last weights have been used
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        float ref[2];
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const float t = top[m][h];
          ref[h] = t == -INFINITY ? 0.f : t;
          if (t != -INFINITY) sum[m][h] *= exp2f(last[m][h] - t);
          last[m][h] = t;
          if ((lane & 3) == 0) s_fac[warp][m * 16 + (lane >> 2) + 8 * h] = t == -INFINITY ? 1.f : exp2f(before[m][h] - t);
        }
#pragma unroll
        for (int t = 0; t < 2; ++t) {
          float w[4];
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            w[q] = exp2f(s[m][t][q] - ref[q >> 1]);
            sum[m][q >> 1] += w[q];
          }
          uint8_t* dst = smem + (sp - sq) + (warp * kRows + m * 16 + (lane >> 2)) * kWidePRow + (t * 8 + (lane & 3) * 2) * 2;
          *reinterpret_cast<uint32_t*>(dst) = pack_bf16x2(w[0], w[1]);
          *reinterpret_cast<uint32_t*>(dst + 8 * kWidePRow) = pack_bf16x2(w[2], w[3]);
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[warp]);
    }
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int row = m * 16 + (lane >> 2) + 8 * h;
        float t = sum[m][h];
        t += __shfl_xor_sync(0xffffffffu, t, 1);
        t += __shfl_xor_sync(0xffffffffu, t, 2);
        if ((lane & 3) == 0) {
          s_sum[warp][row] = t;
          s_last[warp][row] = last[m][h];
        }
      }
  }
  // ------------------------------------------------------------------ weighted sums: value tiles vw, vw + 8, ... of 16 columns
  const int vw = warp - 4;
  float acc[MT][4][2][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int t = 0; t < 2; ++t) acc[m][i][t][0] = acc[m][i][t][1] = acc[m][i][t][2] = acc[m][i][t][3] = 0.f;
  if (vw >= 0 && vw < 8) {
    for (int j = 0, stage = 0, phase = 0; j < n; ++j) {
      const int buf = j % kWideScore;
      wait(&p_full[buf], (j / kWideScore) & 1, kTimeoutFull);
      // the keys are there too, but only a score warp has seen it: every reader of copied bytes observes the barrier
      wait(&full[stage], phase, kTimeoutFull);
      float fac[MT][2];
      bool same = true;
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          fac[m][h] = s_fac[buf][m * 16 + (lane >> 2) + 8 * h];
          same = same && fac[m][h] == 1.f;
        }
      uint32_t a[MT][4], v[4][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) sx_ldsm_x4(sp + (buf * kRows + m * 16 + (lane & 15)) * kWidePRow + (lane >> 4) * 16, a[m]);
      const uint32_t kb = sk + (stage * kServePage + (lane & 15)) * row_b + (lane >> 4) * 16;
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (vw + 8 * i < e16) sx_ldsm_x4_t(kb + (vw + 8 * i) * 32, v[i]);
      if (!__all_sync(0xffffffffu, same)) {
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int t = 0; t < 2; ++t)
#pragma unroll
              for (int q = 0; q < 4; ++q) acc[m][i][t][q] *= fac[m][q >> 1];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (vw + 8 * i < e16)
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            sx_mma(acc[m][i][0], a[m], v[i][0], v[i][1]);
            sx_mma(acc[m][i][1], a[m], v[i][2], v[i][3]);
          }
      __syncwarp();
      if (lane == 0) {
        mbar_arrive(&empty[stage]);
        mbar_arrive(&p_empty[buf]);
      }
      if (++stage == stages) stage = 0, phase ^= 1;
    }
  }
  __syncthreads();
  if (vw < 0 || vw >= 8) return;
  // ------------------------------------------------------------------ output
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int rr = m * 16 + (lane >> 2) + 8 * h, f = f0 + rr;
      if (f >= n_rows) continue;
      const float ref = s_run[rr];
      float total = 0.f;
#pragma unroll
      for (int w = 0; w < kWideScore; ++w)
        if (s_last[w][rr] != -INFINITY) total += s_sum[w][rr] * exp2f(s_last[w][rr] - ref);
      const int qi = f / R, head = g * R + f % R;
      if (splits > 1) {
        float* dst = p.part + (((static_cast<long long>(en) * p.max_len + qi) * p.H + head) * splits + split) * (E + 2);
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int t = 0; t < 2; ++t) {
            const int c = (vw + 8 * i) * 16 + t * 8 + (lane & 3) * 2;
            if (c < E) *reinterpret_cast<float2*>(dst + c) = make_float2(acc[m][i][t][2 * h], acc[m][i][t][2 * h + 1]);
          }
        if (vw == 0 && (lane & 3) == 0) {
          dst[E] = ref;
          dst[E + 1] = total;
        }
      } else {
        const long long row = start + qi;
        const bool per_column = p.sp.gate && p.sp.gate_cols != 1;
        const float inv = inverse_sum(p.sp, head, ref, total) * (per_column ? 1.f : output_gate<__nv_bfloat16>(p.sp, row, head, 0));
        __nv_bfloat16* dst = p.out + row * p.ldo + static_cast<long long>(head) * E;
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int t = 0; t < 2; ++t) {
            const int c = (vw + 8 * i) * 16 + t * 8 + (lane & 3) * 2;
            if (c >= E) continue;
            float u = acc[m][i][t][2 * h] * inv, v = acc[m][i][t][2 * h + 1] * inv;
            if (per_column) {
              u *= output_gate<__nv_bfloat16>(p.sp, row, head, c);
              v *= output_gate<__nv_bfloat16>(p.sp, row, head, c + 1);
            }
            *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16x2(u, v);
          }
      }
    }
}

}  // namespace apb

extern "C" {

// bf16; kcache [pages, G, 16, D rounded up to a multiple of 16, plus 8] whose first E columns are the values and whose columns behind
// D are zeros; D and E multiples of 8, D up to 640, E up to 512; entries of min_len .. max_len rows.  part: fp32 scratch
// [entries, max_len, H, splits, E + 2] when splits > 1.
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
  const int fixed = mt * 16 * (row_b + kWideScore * kWidePRow), fit = (kWideMaxSmem - fixed) / (kServePage * row_b);
  const int stages = fit < kWideMaxStages ? fit : kWideMaxStages, smem = fixed + stages * kServePage * row_b;
  const long long passes = (rows + mt * 16 - 1) / (mt * 16);
  if (passes > 65535 || stages < 2) return kBadArgument;
  const dim3 grid(n_entries * G, splits, static_cast<unsigned>(passes));
  auto run = [&](auto fn) -> int {
    const cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    return static_cast<int>(launch_kernel(fn, grid, dim3(kWideThreads), smem, s, p, stages, status_device_ptr()));
  };
  const int rc = mt == 2 ? run(softmax_attn_wide_kernel<2>) : run(softmax_attn_wide_kernel<1>);
  return rc || splits == 1 ? rc : launch_softmax_merge(p, n_entries, splits, s);
}
}
