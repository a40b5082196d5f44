// Paged causal softmax attention with two maps per head and a score cap (see serve_softmax.cu) on tcgen05 tensor cores: long
// portions of prompts.
//
// A CTA = 128 query rows of one head, none of which leaves the chunk of the first, over that chunk's key pages.  320
// threads: warp 0 TMA producer, warp 1 MMA issuer, warps 2-5 and 6-9 the weight groups, one per map.  The maps ping-pong on
// the tensor core -- while one turns its scores S_j into weights, the other's products run -- and share the value tiles.
//
// K and V tiles of 128 keys come straight from the page cache: eight 16-row boxes (one page of one KV head each) land
// 2 KB apart, which is exactly the 128-byte-swizzle layout of a contiguous 128-row tile.  A K row holds the keys of both
// maps; map g multiplies with its D columns of the tile.  Sizes that are not a multiple of 64 are padded by the zero fill
// of the boxes' out-of-range columns.
//
// The capped scores are bounded, so exp(score - ref) with a fixed reference replaces the running maximum: nothing is ever
// rescaled.  The weights overwrite S_j in tensor memory as packed bf16, feed the P V product as its TMEM operand, and the
// products of all key blocks accumulate in tensor memory; the two outputs are read once, at the end, by both groups (every
// other 32 columns each), which combine, normalise and store them.
#include "common.cuh"
#include "host_utils.cuh"
#include "serve_softmax.cuh"

namespace apb {

constexpr int kXtcThreads = 320;
constexpr int kXtcKeys = 128;                          // keys per block
constexpr int kXtcSlots = 4;                           // ring of K and V tiles
constexpr int kXtcChunk = 128 * 64 * 2;                // 64 columns of 128 rows
constexpr int kXtcTile = 2 * kXtcChunk;
constexpr int kXtcSmem = 2 * kXtcChunk + kXtcSlots * kXtcTile + 1024 + 256;

struct SoftmaxTcParams {
  const int* work;        // [n][8]: entry, KV head, head, first row, valid rows, position of the first row, first key of the
                          // walk (a multiple of the page size), first visible key
  const int* page_table;
  int max_pages;
  __nv_bfloat16* out;
  long long ldo;
  int G, D, E;
  SoftmaxSpec sp;
  int* status;
};

__device__ __forceinline__ void xtc_group_barrier() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

__global__ void __launch_bounds__(kXtcThreads, 1)
softmax_attn_tc_kernel(const __grid_constant__ CUtensorMap tma_q, const __grid_constant__ CUtensorMap tma_k,
                       const __grid_constant__ CUtensorMap tma_v, const SoftmaxTcParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* smem_q = smem;                              // [2 maps][128 rows][64 columns]
  uint8_t* smem_kv = smem + 2 * kXtcChunk;
  uint64_t* kv_full = reinterpret_cast<uint64_t*>(smem_kv + kXtcSlots * kXtcTile);
  uint64_t* kv_empty = kv_full + kXtcSlots;
  uint64_t* q_full = kv_empty + kXtcSlots;
  uint64_t* s_full = q_full + 1;    // [2] scores of a map are in tensor memory
  uint64_t* p_full = s_full + 2;    // [2] its weights are
  uint64_t* o_full = p_full + 2;    // [1] every product has completed
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(o_full + 1);
  __shared__ float s_sum[2][128], s_sq[2][128];

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int* w = p.work + static_cast<long long>(blockIdx.x) * 8;
  const int entry = w[0], kvh = w[1], head = w[2], row0 = w[3], valid = w[4], pos0 = w[5], k0 = w[6], first = w[7];
  const int n_keys = pos0 + valid - k0;                      // keys of the walk
  const int n_blocks = (n_keys + kXtcKeys - 1) / kXtcKeys;
  const int kch = (2 * p.D + 63) >> 6, vch = (p.E + 63) >> 6;    // 64-column chunks

  if (threadIdx.x == 0) {
    for (int s = 0; s < kXtcSlots; ++s) {
      mbar_init(&kv_full[s], 1);
      mbar_init(&kv_empty[s], 1);
    }
    mbar_init(q_full, 1);
    for (int g = 0; g < 2; ++g) {
      mbar_init(&s_full[g], 1);
      mbar_init(&p_full[g], 128);
    }
    mbar_init(o_full, 1);
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_holder, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_holder;
  // TMEM: S / P of map g at columns [g * 128, +128), O of map g at [256 + g * 128, +E)

  if (warp == 0) {
    // ---------------------------------------------------------------- producer (lanes 0-7: one page each)
    if (lane == 0) {
      mbar_expect_tx(q_full, 2 * kXtcChunk);
      for (int g = 0; g < 2; ++g) tma_load_2d(smem_q + g * kXtcChunk, &tma_q, q_full, (head * 2 + g) * p.D, row0);
    }
    // the blocks' tails beyond the last key repeat the last page (their weights are 0)
    const int page0 = k0 / kServePage, n_pages = (k0 + n_keys + kServePage - 1) / kServePage;
    const int* pages = p.page_table + static_cast<long long>(entry) * p.max_pages;
    bool ok = true;
    for (int n = 0; n < 2 * n_blocks && ok; ++n) {
      const int slot = n % kXtcSlots;
      const uint32_t phase = (n / kXtcSlots) & 1;
      ok = mbar_wait(&kv_empty[slot], phase ^ 1, p.status, kTimeoutEmpty);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      const bool is_v = n & 1;
      const int chunks = is_v ? vch : kch;
      if (lane == 0) mbar_expect_tx(&kv_full[slot], chunks * kXtcChunk);
      __syncwarp();
      if (lane < kXtcKeys / kServePage) {
        const int pi = min(page0 + (n >> 1) * (kXtcKeys / kServePage) + lane, n_pages - 1);
        const int row = (pages[pi] * p.G + kvh) * kServePage;
        uint8_t* dst = smem_kv + slot * kXtcTile + lane * (kServePage * 128);
        for (int c = 0; c < chunks; ++c) tma_load_2d(dst + c * kXtcChunk, is_v ? &tma_v : &tma_k, &kv_full[slot], c * 64, row);
      }
    }
    if (!ok) {                         // give copies in flight time to land before the block ends
      const uint64_t t0 = global_timer_ns();
      while (global_timer_ns() - t0 < 100000ull) {
      }
    }
  } else if (warp == 1) {
    // ---------------------------------------------------------------- MMA issuer
    if (lane == 0) {
      const uint32_t idesc_s = umma_idesc_bf16(128, kXtcKeys, 0, 0);
      const uint32_t idesc_o = umma_idesc_bf16(128, (p.E + 15) & ~15, 0, 1);
      const int k_steps = p.D >> 4;
      bool ok = mbar_wait(q_full, 0, p.status, kTimeoutFull);
      auto issue_s = [&](int g, int slot) {
        const uint32_t qa = smem_u32(smem_q + g * kXtcChunk), ka = smem_u32(smem_kv + slot * kXtcTile);
        for (int k = 0; k < k_steps; ++k) {
          const int kcol = g * p.D + k * 16;               // 16 columns never straddle a 64-column chunk
          umma_bf16_ss(tmem_base + g * 128, umma_smem_desc(qa + k * 32, 0, 1024),
                       umma_smem_desc(ka + (kcol >> 6) * kXtcChunk + (kcol & 63) * 2, 0, 1024), idesc_s, k > 0 ? 1u : 0u);
        }
        tc_commit(&s_full[g]);
      };
      auto issue_o = [&](int g, int slot, bool first_block) {
        const uint32_t va = smem_u32(smem_kv + slot * kXtcTile);
#pragma unroll
        for (int k = 0; k < kXtcKeys / 16; ++k)
          umma_bf16_ts(tmem_base + 256 + g * 128, tmem_base + g * 128 + k * 8, umma_smem_desc(va + k * 2048, kXtcChunk, 1024),
                       idesc_o, first_block && k == 0 ? 0u : 1u);
      };
      auto wait_slot = [&](int n) {    // K_j is ring item 2 j, V_j item 2 j + 1
        return mbar_wait(&kv_full[n % kXtcSlots], (n / kXtcSlots) & 1, p.status, kTimeoutFull);
      };
      if (ok) ok = wait_slot(0);
      if (ok) {
        tc_fence_after();
        for (int g = 0; g < 2; ++g) issue_s(g, 0);
        tc_commit(&kv_empty[0]);
      }
      for (int j = 0; j < n_blocks && ok; ++j) {
        const int nv = 2 * j + 1, nk = 2 * j + 2;
        const bool more = j + 1 < n_blocks;
        if (!wait_slot(nv) || (more && !wait_slot(nk))) {
          ok = false;
          break;
        }
        tc_fence_after();
        for (int g = 0; g < 2; ++g) {
          if (!mbar_wait(&p_full[g], j & 1, p.status, kTimeoutTmemEmpty)) {
            ok = false;
            break;
          }
          tc_fence_after();
          issue_o(g, nv % kXtcSlots, j == 0);
          if (more) issue_s(g, nk % kXtcSlots);      // runs after the product above has read the weights
        }
        if (!ok) break;
        tc_commit(&kv_empty[nv % kXtcSlots]);
        if (more) tc_commit(&kv_empty[nk % kXtcSlots]);
      }
      if (ok) tc_commit(o_full);
    }
  } else {
    // ---------------------------------------------------------------- weight groups, one per map
    const int g = (warp - 2) >> 2;
    const int quarter = warp & 3, row = quarter * 32 + lane;
    const uint32_t lane_off = static_cast<uint32_t>(quarter * 32) << 16;
    const uint32_t t_s = tmem_base + lane_off + g * 128;
    const float zs = p.sp.scale / p.sp.cap, gain = p.sp.cap * 1.4426950408889634f;
    const float ref = score_reference(p.sp.cap) * 1.4426950408889634f;
    // gain tanh(zs s) = s P(s^2) near zero: the series of tanh_series with the scale and the gain folded in
    const float z2 = zs * zs, c0 = gain * zs, c1 = c0 * z2 * (-1.f / 3.f), c2 = c0 * z2 * z2 * (2.f / 15.f),
                c3 = c0 * z2 * z2 * z2 * (-17.f / 315.f), c4 = c0 * z2 * z2 * z2 * z2 * (62.f / 2835.f);
    const uint64_t p0 = xtc_pair(c0, c0), p1 = xtc_pair(c1, c1), p2 = xtc_pair(c2, c2), p3 = xtc_pair(c3, c3),
                   p4 = xtc_pair(c4, c4), off = xtc_pair(-ref, -ref);
    const float small = (kSmallTanh / zs) * (kSmallTanh / zs);
    uint64_t sum2 = xtc_pair(0.f, 0.f);
    bool ok = true;
    for (int j = 0; j < n_blocks; ++j) {
      if (!mbar_wait(&s_full[g], j & 1, p.status, kTimeoutTmemFull)) {
        ok = false;
        break;
      }
      tc_fence_after();
      const int base = k0 + j * kXtcKeys;                                // position of the block's first key
      const int limit = pos0 + min(row, valid - 1) + 1 - base;           // visible keys: [skip, limit) of the block
      const int skip = first - base;
      const bool full = pos0 + 1 - base >= kXtcKeys && skip <= 0;        // ... all 128 for every row
      uint32_t ring[2][32];
      tmem_ld_32x32(t_s, ring[0]);
#pragma unroll
      for (int c = 0; c < kXtcKeys / 32; ++c) {        // the next 32 scores are on their way while these are worked on
        uint32_t(&r)[32] = ring[c & 1];
        uint32_t pk[16];
        xtc_wait_load(r);
        if (c + 1 < kXtcKeys / 32) tmem_ld_32x32(t_s + (c + 1) * 32, ring[(c + 1) & 1]);
        uint64_t v[16];                                // log2 weights of neighbouring keys
        float top = 0.f;
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const uint64_t x = xtc_pair(__uint_as_float(r[2 * i]), __uint_as_float(r[2 * i + 1]));
          const uint64_t a = xtc_mul2(x, x);
          const float2 f = xtc_unpair(a);
          top = fmaxf(fmaxf(top, f.x), f.y);
          uint64_t y = xtc_fma2(a, p4, p3);
          y = xtc_fma2(a, y, p2);
          y = xtc_fma2(a, y, p1);
          y = xtc_fma2(a, y, p0);
          v[i] = xtc_fma2(x, y, off);
        }
        if (!__all_sync(0xffffffffu, top <= small)) {  // some score lies beyond the series
#pragma unroll
          for (int i = 0; i < 16; ++i)
            v[i] = xtc_pair(fmaf(tanh_any(__uint_as_float(r[2 * i]) * zs), gain, -ref),
                            fmaf(tanh_any(__uint_as_float(r[2 * i + 1]) * zs), gain, -ref));
        }
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const float2 f = xtc_unpair(v[i]);
          float w0 = xtc_ex2(f.x), w1 = xtc_ex2(f.y);
          if (!full) {
            const int a = c * 32 + 2 * i;
            if (a >= limit || a < skip) w0 = 0.f;
            if (a + 1 >= limit || a + 1 < skip) w1 = 0.f;
          }
          sum2 = xtc_add2(sum2, xtc_pair(w0, w1));
          pk[i] = pack_bf16x2(w0, w1);
        }
        tmem_st_32x16(t_s + c * 16, pk);
      }
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(&p_full[g]);
    }
    const float2 halves = xtc_unpair(sum2);
    s_sum[g][row] = halves.x + halves.y;
    xtc_group_barrier();
    if (ok) ok = mbar_wait(o_full, 0, p.status, kTimeoutTmemFull);
    float o[2][32], sq = 0.f;
    if (ok) {
      tc_fence_after();
      const float i0 = 1.f / s_sum[0][row], i1 = *p.sp.lambda / s_sum[1][row];
#pragma unroll
      for (int n = 0; n < 2; ++n) {                      // columns [c, c + 32) of the output; E <= 128
        const int c = (2 * n + g) * 32;
        if (c < p.E) {
          uint32_t r[32];
          tmem_ld_32x32(tmem_base + lane_off + 256 + c, r);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) o[n][i] = __uint_as_float(r[i]) * i0;
          tmem_ld_32x32(tmem_base + lane_off + 384 + c, r);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            o[n][i] = c + i < p.E ? o[n][i] - __uint_as_float(r[i]) * i1 : 0.f;
            sq += o[n][i] * o[n][i];
          }
        }
      }
      tc_fence_before();
    }
    s_sq[g][row] = sq;
    xtc_group_barrier();
    if (ok && row < valid) {
      const float post = p.sp.post_scale / sqrtf((s_sq[0][row] + s_sq[1][row]) / p.E + p.sp.eps);
      __nv_bfloat16* dst = p.out + static_cast<long long>(row0 + row) * p.ldo + static_cast<long long>(head) * p.E;
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        const int c = (2 * n + g) * 32;
#pragma unroll
        for (int q = 0; q < 4; ++q)
          if (c + q * 8 < p.E) {
            uint4 v;
            v.x = pack_bf16x2(o[n][q * 8] * post, o[n][q * 8 + 1] * post);
            v.y = pack_bf16x2(o[n][q * 8 + 2] * post, o[n][q * 8 + 3] * post);
            v.z = pack_bf16x2(o[n][q * 8 + 4] * post, o[n][q * 8 + 5] * post);
            v.w = pack_bf16x2(o[n][q * 8 + 6] * post, o[n][q * 8 + 7] * post);
            *reinterpret_cast<uint4*>(dst + c + q * 8) = v;
          }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

}  // namespace apb

extern "C" {

// q: [rows, H * 2 D] columns of a row-major buffer (row stride ldq); caches [pages, G, 16, 2 D] and [pages, G, 16, E]; out
// [rows, H*E] (row stride ldo), 16-byte aligned rows.  Two maps; D a multiple of 16 up to 64, E a multiple of 8 up to 128,
// 0 < cap <= 64.  work: device int32 [n][8] (SoftmaxTcParams).
int apb_softmax_attn_tc(const void* q, long long ldq, int rows, const int* work, int n_work, const int* page_table,
                        int max_pages, const void* kcache, const void* vcache, int pages, void* out, long long ldo, int H,
                        int G, int D, int E, float scale, float cap, const float* lambda, float post_scale, float eps,
                        cudaStream_t stream) {
  using namespace apb;
  if (n_work <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || D <= 0 || E <= 0 || (D % 16) || (E % 8) || D > 64 || E > 128 || (ldq % 8) || (ldo % 8) ||
      (reinterpret_cast<uintptr_t>(q) & 15) || (reinterpret_cast<uintptr_t>(out) & 15) || pages <= 0 || !work || !page_table ||
      !lambda || !fixed_reference(cap))
    return kBadArgument;
  CUtensorMap tq, tk, tv;
  const uint64_t cache_rows = static_cast<uint64_t>(pages) * G * kServePage;
  int rc = make_tmap_2d(&tq, q, 2, rows, static_cast<uint64_t>(H) * 2 * D, ldq, 64, 128);
  if (rc) return 1000 + rc;
  rc = make_tmap_2d(&tk, kcache, 2, cache_rows, 2 * D, 2 * D, 64, kServePage);
  if (rc) return 2000 + rc;
  rc = make_tmap_2d(&tv, vcache, 2, cache_rows, E, E, 64, kServePage);
  if (rc) return 3000 + rc;
  SoftmaxTcParams p{work, page_table, max_pages, static_cast<__nv_bfloat16*>(out), ldo, G, D, E,
                    SoftmaxSpec{scale, cap, 0, 2, lambda, post_scale, eps, 0, nullptr, nullptr, 0, 0}, status_device_ptr()};
  const cudaError_t e = cudaFuncSetAttribute(softmax_attn_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kXtcSmem);
  if (e != cudaSuccess) return static_cast<int>(e);
  softmax_attn_tc_kernel<<<n_work, kXtcThreads, kXtcSmem, stream>>>(tq, tk, tv, p);
  return static_cast<int>(cudaGetLastError());
}
}
