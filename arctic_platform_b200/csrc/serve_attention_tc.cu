// Paged causal sigmoid attention (see serve_attention.cu) on tcgen05 tensor cores: long portions of prompts.
//
// A CTA walks the key pages of one sequence and KV head for up to two GROUPS of 128 query rows -- two query heads of the
// KV head on the same rows, or, when a head is left over, two consecutive row tiles of one head.  320 threads: warp 0
// TMA producer, warp 1 MMA issuer, warps 2-5 and 6-9 the weight groups.  The groups ping-pong on the tensor core: while
// one turns its scores S_j into weights, the other's products run.
//
// K and V tiles of 128 keys come straight from the page cache: eight 16-row boxes (one page of one KV head each) land
// 2 KB apart, which is exactly the 128-byte-swizzle layout of a contiguous 128-row tile.  Head sizes that are not a
// multiple of 64 are padded by the zero fill of the boxes' out-of-range columns.
//
// The weights are not normalised, so there is no running maximum and nothing to rescale: sigmoid(S_j) overwrites S_j in
// tensor memory as packed bf16, feeds the P V product as its TMEM operand, and the products of all key blocks
// accumulate in tensor memory; the output is read once, at the end.
#include "common.cuh"
#include "host_utils.cuh"
#include "serve_common.cuh"

namespace apb {

constexpr int kStcThreads = 320;
constexpr int kStcKeys = 128;                          // keys per block
constexpr int kStcSlots = 4;                           // ring of K and V tiles
constexpr int kStcTile = 2 * 128 * 64 * 2;             // up to two 64-column chunks of 128 rows
constexpr int kStcSmem = (2 + kStcSlots) * kStcTile + 1024 + 256;

struct SigmoidTcParams {
  const int* work;        // [n][12]: entry, key blocks, KV head, 0, then per group (row, valid rows, head, keys of row 0)
  const int* page_table;
  int max_pages;
  const __nv_bfloat16* bias;
  __nv_bfloat16* out;
  long long ldo;
  int G, D, E;
  float scale_l2, out_scale;
  int* status;
};

__device__ __forceinline__ float ex2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp_approx(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__global__ void __launch_bounds__(kStcThreads, 1)
sigmoid_attn_tc_kernel(const __grid_constant__ CUtensorMap tma_q, const __grid_constant__ CUtensorMap tma_k,
                       const __grid_constant__ CUtensorMap tma_v, const SigmoidTcParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* smem_q = smem;
  uint8_t* smem_kv = smem + 2 * kStcTile;
  uint64_t* kv_full = reinterpret_cast<uint64_t*>(smem_kv + kStcSlots * kStcTile);
  uint64_t* kv_empty = kv_full + kStcSlots;
  uint64_t* q_full = kv_empty + kStcSlots;
  uint64_t* s_full = q_full + 1;    // [2] scores of a group are in tensor memory
  uint64_t* p_full = s_full + 2;    // [2] its weights are
  uint64_t* o_full = p_full + 2;    // [1] every product has completed
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(o_full + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int* w = p.work + static_cast<long long>(blockIdx.x) * 12;
  const int entry = w[0], n_blocks = w[1], kvh = w[2];
  const int n_groups = w[9] > 0 ? 2 : 1;
  const int kch = (p.D + 63) >> 6, vch = (p.E + 63) >> 6;    // 64-column chunks

  if (threadIdx.x == 0) {
    for (int s = 0; s < kStcSlots; ++s) {
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
  // TMEM: S / P of group g at columns [g * 128, +128), O of group g at [256 + g * 128, +E)

  if (warp == 0) {
    // ---------------------------------------------------------------- producer (lanes 0-7: one page each)
    if (lane == 0) {
      mbar_expect_tx(q_full, n_groups * kch * 16384);
      for (int g = 0; g < n_groups; ++g)
        for (int c = 0; c < kch; ++c)
          tma_load_2d(smem_q + g * kStcTile + c * 16384, &tma_q, q_full, w[6 + 4 * g] * p.D + c * 64, w[4 + 4 * g]);
    }
    // pages of the last key any row may see; the blocks' tails beyond it repeat the last page (their weights are 0)
    const int last = w[4 + 4 * (n_groups - 1) + 3] + w[4 + 4 * (n_groups - 1) + 1] - 1;
    const int last0 = w[7] + w[5] - 1;
    const int n_pages = (max(last, last0) + kServePage - 1) / kServePage;
    const int* pages = p.page_table + static_cast<long long>(entry) * p.max_pages;
    bool ok = true;
    for (int n = 0; n < 2 * n_blocks && ok; ++n) {
      const int slot = n % kStcSlots;
      const uint32_t phase = (n / kStcSlots) & 1;
      ok = mbar_wait(&kv_empty[slot], phase ^ 1, p.status, kTimeoutEmpty);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      const bool is_v = n & 1;
      const int chunks = is_v ? vch : kch;
      if (lane == 0) mbar_expect_tx(&kv_full[slot], chunks * 16384);
      __syncwarp();
      if (lane < kStcKeys / kServePage) {
        const int pi = min((n >> 1) * (kStcKeys / kServePage) + lane, n_pages - 1);
        const int row = (pages[pi] * p.G + kvh) * kServePage;
        uint8_t* dst = smem_kv + slot * kStcTile + lane * (kServePage * 128);
        for (int c = 0; c < chunks; ++c) tma_load_2d(dst + c * 16384, is_v ? &tma_v : &tma_k, &kv_full[slot], c * 64, row);
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
      const uint32_t idesc_s = umma_idesc_bf16(128, kStcKeys, 0, 0);
      const uint32_t idesc_o = umma_idesc_bf16(128, (p.E + 15) & ~15, 0, 1);
      const int k_steps = (p.D + 15) >> 4;
      bool ok = mbar_wait(q_full, 0, p.status, kTimeoutFull);
      auto issue_s = [&](int g, int slot) {
        const uint32_t qa = smem_u32(smem_q + g * kStcTile), ka = smem_u32(smem_kv + slot * kStcTile);
        for (int k = 0; k < k_steps; ++k) {
          const uint32_t off = (k / 4) * 16384 + (k % 4) * 32;
          umma_bf16_ss(tmem_base + g * 128, umma_smem_desc(qa + off, 0, 1024), umma_smem_desc(ka + off, 0, 1024), idesc_s,
                       k > 0 ? 1u : 0u);
        }
        tc_commit(&s_full[g]);
      };
      auto issue_o = [&](int g, int slot, bool first) {
        const uint32_t va = smem_u32(smem_kv + slot * kStcTile);
#pragma unroll
        for (int k = 0; k < kStcKeys / 16; ++k)
          umma_bf16_ts(tmem_base + 256 + g * 128, tmem_base + g * 128 + k * 8, umma_smem_desc(va + k * 2048, 16384, 1024),
                       idesc_o, first && k == 0 ? 0u : 1u);
      };
      auto wait_slot = [&](int n) {    // K_j is ring item 2 j, V_j item 2 j + 1
        return mbar_wait(&kv_full[n % kStcSlots], (n / kStcSlots) & 1, p.status, kTimeoutFull);
      };
      if (ok) ok = wait_slot(0);
      if (ok) {
        tc_fence_after();
        for (int g = 0; g < n_groups; ++g) issue_s(g, 0);
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
        for (int g = 0; g < n_groups; ++g) {
          if (!mbar_wait(&p_full[g], j & 1, p.status, kTimeoutTmemEmpty)) {
            ok = false;
            break;
          }
          tc_fence_after();
          issue_o(g, nv % kStcSlots, j == 0);
          if (more) issue_s(g, nk % kStcSlots);      // runs after the product above has read the weights
        }
        if (!ok) break;
        tc_commit(&kv_empty[nv % kStcSlots]);
        if (more) tc_commit(&kv_empty[nk % kStcSlots]);
      }
      if (ok) tc_commit(o_full);
    }
  } else {
    // ---------------------------------------------------------------- weight groups
    const int g = (warp - 2) >> 2;
    if (g < n_groups) {
      const int* wg = w + 4 + 4 * g;
      const int q_row0 = wg[0], q_valid = wg[1], head = wg[2], keys0 = wg[3];
      const int quarter = warp & 3, row = quarter * 32 + lane;
      const uint32_t lane_off = static_cast<uint32_t>(quarter * 32) << 16;
      const uint32_t t_s = tmem_base + lane_off + g * 128, t_o = tmem_base + lane_off + 256 + g * 128;
      const float b_l2 = -__bfloat162float(p.bias[head]) * 1.4426950408889634f;
      bool ok = true;
      for (int j = 0; j < n_blocks; ++j) {
        if (!mbar_wait(&s_full[g], j & 1, p.status, kTimeoutTmemFull)) {
          ok = false;
          break;
        }
        tc_fence_after();
        const int limit = min(row, q_valid - 1) + keys0 - j * kStcKeys;   // visible keys of this block for this row
        const bool full = keys0 - j * kStcKeys >= kStcKeys;               // ... all 128 for every row of the tile
#pragma unroll 1
        for (int c = 0; c < kStcKeys / 32; ++c) {
          uint32_t r[32], pk[16];
          tmem_ld_32x32(t_s + c * 32, r);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            // sigmoid(z) = 1 / (1 + 2^(-z log2 e)); one reciprocal serves two weights (exponents are capped so that
            // the product of the two denominators stays finite)
            const float a0 = 1.f + ex2_approx(fminf(fmaf(__uint_as_float(r[2 * i]), -p.scale_l2, b_l2), 60.f));
            const float a1 = 1.f + ex2_approx(fminf(fmaf(__uint_as_float(r[2 * i + 1]), -p.scale_l2, b_l2), 60.f));
            const float inv = rcp_approx(a0 * a1);
            float p0 = inv * a1, p1 = inv * a0;
            if (!full) {
              if (c * 32 + 2 * i >= limit) p0 = 0.f;
              if (c * 32 + 2 * i + 1 >= limit) p1 = 0.f;
            }
            pk[i] = pack_bf16x2(p0, p1);
          }
          tmem_st_32x16(t_s + c * 16, pk);
        }
        tmem_st_wait();
        tc_fence_before();
        mbar_arrive(&p_full[g]);
      }
      if (ok) ok = mbar_wait(o_full, 0, p.status, kTimeoutTmemFull);
      if (ok) {
        tc_fence_after();
        __nv_bfloat16* dst = p.out + static_cast<long long>(q_row0 + row) * p.ldo + static_cast<long long>(head) * p.E;
#pragma unroll 1
        for (int c = 0; c < p.E; c += 32) {
          uint32_t r[32];
          tmem_ld_32x32(t_o + c, r);
          tmem_ld_wait();
          if (row < q_valid) {
#pragma unroll
            for (int q = 0; q < 4; ++q)
              if (c + q * 8 < p.E) {
                uint4 o;
                o.x = pack_bf16x2(__uint_as_float(r[q * 8]) * p.out_scale, __uint_as_float(r[q * 8 + 1]) * p.out_scale);
                o.y = pack_bf16x2(__uint_as_float(r[q * 8 + 2]) * p.out_scale, __uint_as_float(r[q * 8 + 3]) * p.out_scale);
                o.z = pack_bf16x2(__uint_as_float(r[q * 8 + 4]) * p.out_scale, __uint_as_float(r[q * 8 + 5]) * p.out_scale);
                o.w = pack_bf16x2(__uint_as_float(r[q * 8 + 6]) * p.out_scale, __uint_as_float(r[q * 8 + 7]) * p.out_scale);
                *reinterpret_cast<uint4*>(dst + c + q * 8) = o;
              }
          }
        }
        tc_fence_before();
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

// q: [rows, H*D] columns of a row-major buffer (row stride ldq); caches [pages, G, 16, D] and [pages, G, 16, E]; out
// [rows, H*E] (row stride ldo), 16-byte aligned rows.  D and E multiples of 8 up to 128.  work: device int32 [n][12]
// (SigmoidTcParams); every item has at least one key block.
int apb_sigmoid_attn_tc(const void* q, long long ldq, int rows, const int* work, int n_work, const int* page_table,
                        int max_pages, const void* kcache, const void* vcache, int pages, const void* bias, void* out,
                        long long ldo, int H, int G, int D, int E, float scale, float out_scale, cudaStream_t stream) {
  using namespace apb;
  if (n_work <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || D <= 0 || E <= 0 || (D % 8) || (E % 8) || D > 128 || E > 128 || (ldq % 8) || (ldo % 8) ||
      (reinterpret_cast<uintptr_t>(q) & 15) || (reinterpret_cast<uintptr_t>(out) & 15) || pages <= 0 || !work || !page_table)
    return kBadArgument;
  CUtensorMap tq, tk, tv;
  const uint64_t cache_rows = static_cast<uint64_t>(pages) * G * kServePage;
  int rc = make_tmap_2d(&tq, q, 2, rows, static_cast<uint64_t>(H) * D, ldq, 64, 128);
  if (rc) return 1000 + rc;
  rc = make_tmap_2d(&tk, kcache, 2, cache_rows, D, D, 64, kServePage);
  if (rc) return 2000 + rc;
  rc = make_tmap_2d(&tv, vcache, 2, cache_rows, E, E, 64, kServePage);
  if (rc) return 3000 + rc;
  SigmoidTcParams p{work, page_table, max_pages, static_cast<const __nv_bfloat16*>(bias), static_cast<__nv_bfloat16*>(out),
                    ldo, G, D, E, scale * 1.4426950408889634f, out_scale, status_device_ptr()};
  const cudaError_t e = cudaFuncSetAttribute(sigmoid_attn_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kStcSmem);
  if (e != cudaSuccess) return static_cast<int>(e);
  sigmoid_attn_tc_kernel<<<n_work, kStcThreads, kStcSmem, stream>>>(tq, tk, tv, p);
  return static_cast<int>(cudaGetLastError());
}
}
