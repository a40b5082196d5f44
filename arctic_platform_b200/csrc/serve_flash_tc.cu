// Causal softmax attention on tcgen05 tensor cores for long portions of prompts: one map, optional sliding window, sinks, output
// gates and score cap (see SoftmaxSpec), no bound on the scores needed.
//
// A CTA = two tiles of 128 query rows that share their keys: two query heads of one KV head on the same rows, or two
// consecutive row tiles of one head.  352 threads: warp 0 TMA producer, warps 2-5 and 6-9 the weight groups and warps 1 and 10 the MMA
// issuers, one per tile; the tiles ping-pong on the tensor core.
//
// Keys and values come from the page cache (16-row boxes, one page of one KV head each) or from a contiguous copy of the
// entry's context (128-row boxes; a head's columns side by side).  A key may have a second part that all heads share (the
// rotated part of latent attention), read through a tensor map of its own; queries hold both parts side by side.
//
// K and V travel in chunks of 64 columns x 128 keys through one ring.  The weights are taken relative to a reference that
// follows the running maximum only when it falls behind by more than 2^8: the products of all key blocks accumulate in tensor
// memory and are rescaled there on those rare occasions.  Under a score cap up to 64 the reference is fixed.
#include "common.cuh"
#include "host_utils.cuh"
#include "serve_softmax.cuh"

namespace apb {

constexpr int kFlThreads = 352;
constexpr int kFlKeys = 128;                           // keys per block
constexpr int kFlChunk = 128 * 64 * 2;                 // 64 columns of 128 rows
constexpr int kFlChunks = 14;                          // query chunks and ring slots together
constexpr int kFlMaxRing = 12;
constexpr int kFlSmem = kFlChunks * kFlChunk + 1024 + 512;
constexpr float kFlLag = 8.f;                          // in log2: how far the reference may lag behind the maximum

struct FlashParams {
  const int* work;        // [n][12]: entry, KV head, first key of the walk (a multiple of the page size), row of the entry's key 0 in
                          // the contiguous copy; then per tile: first row, valid rows (0: no second tile), head, position
  const int* page_table;  // null: contiguous keys
  int max_pages;
  __nv_bfloat16* out;
  long long ldo;
  int G, D, R, E;         // R: columns of the shared second part
  SoftmaxSpec sp;
  int* status;
};

// Weights 2^(score scale + off) of a row's 128 scores at t_s, packed, and their sum in two halves; top: the largest exponent.
// WHOLE: every key counts, otherwise those in [skip, limit).
template <bool WHOLE>
__device__ __forceinline__ uint64_t flash_weights(uint32_t t_s, uint64_t scale2, float off, int limit, int skip, float& top,
                                                  uint32_t (&pk)[4][16]) {
  const uint64_t off2 = xtc_pair(off, off);
  uint64_t sum[2] = {xtc_pair(0.f, 0.f), xtc_pair(0.f, 0.f)};
  float t0 = -INFINITY, t1 = -INFINITY;
  uint32_t stage[2][32];
  tmem_ld_32x32(t_s, stage[0]);
#pragma unroll
  for (int c = 0; c < 4; ++c) {                        // the next 32 scores are on their way while these are worked on
    uint32_t(&r)[32] = stage[c & 1];
    xtc_wait_load(r);
    if (c < 3) tmem_ld_32x32(t_s + (c + 1) * 32, stage[(c + 1) & 1]);
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      float2 v = xtc_unpair(xtc_fma2(xtc_pair(__uint_as_float(r[2 * i]), __uint_as_float(r[2 * i + 1])), scale2, off2));
      if (!WHOLE) {
        const int a = c * 32 + 2 * i;
        if (a >= limit || a < skip) v.x = -INFINITY;
        if (a + 1 >= limit || a + 1 < skip) v.y = -INFINITY;
      }
      t0 = fmaxf(t0, v.x);
      t1 = fmaxf(t1, v.y);
      const float w0 = xtc_ex2(v.x), w1 = xtc_ex2(v.y);
      sum[i & 1] = xtc_add2(sum[i & 1], xtc_pair(w0, w1));
      pk[c][i] = pack_bf16x2(w0, w1);
    }
  }
  top = fmaxf(t0, t1);
  return xtc_add2(sum[0], sum[1]);
}

// The same for capped scores, 2^(gain tanh(z) + off): the series of tanh_series with the scales folded into its coefficients, or the
// exponential form for a warp that holds a larger score (an exponent needs absolute accuracy only).
struct CapSeries {
  float gain, e2, small;       // e2: log2 e^(2 z) of a score; small: largest squared score of the series
  uint64_t c[5];
};
__device__ __forceinline__ CapSeries cap_series(const SoftmaxSpec& sp) {
  CapSeries k;
  const float zs = sp.scale / sp.cap, z2 = zs * zs;
  k.gain = sp.cap * 1.4426950408889634f;
  k.e2 = 2.f * 1.4426950408889634f * zs;
  k.small = (kSmallTanh / zs) * (kSmallTanh / zs);
  const float t[5] = {1.f, -1.f / 3.f, 2.f / 15.f, -17.f / 315.f, 62.f / 2835.f};
  float f = k.gain * zs;
#pragma unroll
  for (int i = 0; i < 5; ++i, f *= z2) k.c[i] = xtc_pair(f * t[i], f * t[i]);
  return k;
}
// 32 of a row's scores r as exponents v, pairs of neighbouring keys.
__device__ __forceinline__ void capped_exponents(const uint32_t (&r)[32], const CapSeries& k, float off, uint64_t (&v)[16]) {
  const uint64_t off2 = xtc_pair(off, off);
  float large = 0.f;
#pragma unroll
  for (int i = 0; i < 16; ++i) {
    const uint64_t x = xtc_pair(__uint_as_float(r[2 * i]), __uint_as_float(r[2 * i + 1])), a = xtc_mul2(x, x);
    const float2 f = xtc_unpair(a);
    large = fmaxf(fmaxf(large, f.x), f.y);
    uint64_t y = xtc_fma2(a, k.c[4], k.c[3]);
    y = xtc_fma2(a, y, k.c[2]);
    y = xtc_fma2(a, y, k.c[1]);
    y = xtc_fma2(a, y, k.c[0]);
    v[i] = xtc_fma2(x, y, off2);
  }
  if (!__all_sync(0xffffffffu, large <= k.small)) {
#pragma unroll
    for (int i = 0; i < 16; ++i)                       // gain tanh(z) = gain - 2 gain / (1 + e^(2 z))
      v[i] = xtc_pair((k.gain + off) - __fdividef(2.f * k.gain, 1.f + xtc_ex2(__uint_as_float(r[2 * i]) * k.e2)),
                      (k.gain + off) - __fdividef(2.f * k.gain, 1.f + xtc_ex2(__uint_as_float(r[2 * i + 1]) * k.e2)));
  }
}
template <bool WHOLE>
__device__ __forceinline__ uint64_t flash_capped_weights(uint32_t t_s, const CapSeries& k, float off, int limit, int skip, float& top,
                                                         uint32_t (&pk)[4][16]) {
  uint64_t sum = xtc_pair(0.f, 0.f);
  float t0 = -INFINITY;
#pragma unroll
  for (int c = 0; c < 4; ++c) {
    uint32_t r[32];
    uint64_t v[16];
    tmem_ld_32x32(t_s + c * 32, r);
    xtc_wait_load(r);
    capped_exponents(r, k, off, v);
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      float2 f = xtc_unpair(v[i]);
      if (!WHOLE) {
        const int a = c * 32 + 2 * i;
        if (a >= limit || a < skip) f.x = -INFINITY;
        if (a + 1 >= limit || a + 1 < skip) f.y = -INFINITY;
      }
      t0 = fmaxf(t0, fmaxf(f.x, f.y));
      const float w0 = xtc_ex2(f.x), w1 = xtc_ex2(f.y);
      sum = xtc_add2(sum, xtc_pair(w0, w1));
      pk[c][i] = pack_bf16x2(w0, w1);
    }
  }
  top = t0;
  return sum;
}
// With a fixed reference nothing is looked at twice: the weights replace the scores run by run (weights c lie over scores c / 2, which
// have been read).
template <bool WHOLE>
__device__ __forceinline__ uint64_t flash_fixed_weights(uint32_t t_s, const CapSeries& k, float off, int limit, int skip) {
  uint64_t sum[2] = {xtc_pair(0.f, 0.f), xtc_pair(0.f, 0.f)};
  uint32_t stage[2][32];
  tmem_ld_32x32(t_s, stage[0]);
#pragma unroll
  for (int c = 0; c < 4; ++c) {
    uint32_t(&r)[32] = stage[c & 1];
    xtc_wait_load(r);
    if (c < 3) tmem_ld_32x32(t_s + (c + 1) * 32, stage[(c + 1) & 1]);
    uint64_t v[16];
    capped_exponents(r, k, off, v);
    uint32_t pk[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      const float2 f = xtc_unpair(v[i]);
      float w0 = xtc_ex2(f.x), w1 = xtc_ex2(f.y);
      if (!WHOLE) {
        const int a = c * 32 + 2 * i;
        if (a >= limit || a < skip) w0 = 0.f;
        if (a + 1 >= limit || a + 1 < skip) w1 = 0.f;
      }
      sum[i & 1] = xtc_add2(sum[i & 1], xtc_pair(w0, w1));
      pk[i] = pack_bf16x2(w0, w1);
    }
    tmem_st_32x16(t_s + c * 16, pk);
  }
  return xtc_add2(sum[0], sum[1]);
}

enum FlashCap : int { kFlashUncapped = 0, kFlashCapped = 1, kFlashFixed = 2 };

template <int CAP>
__global__ void __launch_bounds__(kFlThreads, 1)
flash_tc_kernel(const __grid_constant__ CUtensorMap tma_q, const __grid_constant__ CUtensorMap tma_k,
                const __grid_constant__ CUtensorMap tma_k2, const __grid_constant__ CUtensorMap tma_v, const FlashParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + kFlChunks * kFlChunk);
  uint64_t* empty = full + kFlMaxRing;
  uint64_t* q_full = empty + kFlMaxRing;
  uint64_t* s_full = q_full + 1;    // [2] scores of a tile are in tensor memory
  uint64_t* p_full = s_full + 2;    // [2] its weights are
  uint64_t* o_full = p_full + 2;    // [2] every product of the tile has completed
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(o_full + 2);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int* w = p.work + static_cast<long long>(blockIdx.x) * 12;
  const int entry = w[0], kvh = w[1], k0 = w[2], base_row = w[3];
  const int n_tiles = w[9] > 0 ? 2 : 1;
  const int k1 = (p.D + 63) >> 6, kch = k1 + ((p.R + 63) >> 6), vch = (p.E + 63) >> 6;
  const int ring = min(kFlMaxRing, kFlChunks - 2 * kch), per = kch + vch;
  uint8_t* smem_q = smem;                              // [2 tiles][kch]
  uint8_t* smem_kv = smem + 2 * kch * kFlChunk;
  auto blocks_of = [&](int g) { return (w[4 + 4 * g + 3] + w[4 + 4 * g + 1] - k0 + kFlKeys - 1) / kFlKeys; };
  const int nb0 = blocks_of(0), nb1 = n_tiles == 2 ? blocks_of(1) : 0, n_blocks = max(nb0, nb1);

  if (threadIdx.x == 0) {
    for (int s = 0; s < ring; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], n_tiles);
    }
    mbar_init(q_full, 1);
    for (int g = 0; g < 2; ++g) {
      mbar_init(&s_full[g], 1);
      mbar_init(&p_full[g], 128);
      mbar_init(&o_full[g], 1);
    }
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
  // TMEM: S / P of tile g at columns [g * 128, +128), O of tile g at [256 + g * 128, +E)

  if (warp == 0) {
    // ---------------------------------------------------------------- producer (lanes 0-7: one page each)
    if (lane == 0) {
      mbar_expect_tx(q_full, n_tiles * kch * kFlChunk);
      for (int g = 0; g < n_tiles; ++g)
        for (int c = 0; c < kch; ++c)
          tma_load_2d(smem_q + (g * kch + c) * kFlChunk, &tma_q, q_full,
                      w[4 + 4 * g + 2] * (p.D + p.R) + (c < k1 ? c * 64 : p.D + (c - k1) * 64), w[4 + 4 * g]);
    }
    // paged: the blocks' tails beyond the last key repeat the last page (their weights are 0)
    const bool paged = p.page_table != nullptr;
    const int last = max(w[7] + w[5], n_tiles == 2 ? w[11] + w[9] : 0);                 // keys of the walk's end
    const int page0 = k0 / kServePage, n_pages = (last + kServePage - 1) / kServePage;
    const int* pages = p.page_table + static_cast<long long>(entry) * p.max_pages;
    bool ok = true;
    int slot = 0;
    uint32_t phase = 1;
    for (int j = 0; j < n_blocks && ok; ++j) {
      int row = 0;
      if (paged && lane < kFlKeys / kServePage)
        row = (pages[min(page0 + j * (kFlKeys / kServePage) + lane, n_pages - 1)] * p.G + kvh) * kServePage;
      for (int c = 0; c < per; ++c) {
        ok = mbar_wait(&empty[slot], phase, p.status, kTimeoutEmpty);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        if (lane == 0) mbar_expect_tx(&full[slot], kFlChunk);
        __syncwarp();
        uint8_t* dst = smem_kv + slot * kFlChunk;
        const bool second = c >= k1 && c < kch;
        const CUtensorMap* map = c < k1 ? &tma_k : second ? &tma_k2 : &tma_v;
        const int col = c < k1 ? c * 64 : second ? (c - k1) * 64 : (c - kch) * 64;
        if (paged) {
          if (lane < kFlKeys / kServePage) tma_load_2d(dst + lane * (kServePage * 128), map, &full[slot], col, row);
        } else if (lane == 0) {
          tma_load_2d(dst, map, &full[slot], second ? col : kvh * (c < k1 ? p.D : p.E) + col, base_row + k0 + j * kFlKeys);
        }
        if (++slot == ring) slot = 0, phase ^= 1;
      }
    }
    if (!ok) {                         // give copies in flight time to land before the block ends
      const uint64_t t0 = global_timer_ns();
      while (global_timer_ns() - t0 < 100000ull) {
      }
    }
  } else if (warp == 1 || warp == 10) {
    // ---------------------------------------------------------------- MMA issuers, one per tile
    const int g = warp == 10;
    if (lane == 0 && g < n_tiles) {
      const int nb = g ? nb1 : nb0, e16 = (p.E + 15) & ~15;
      const uint32_t idesc_s = umma_idesc_bf16(128, kFlKeys, 0, 0);
      const uint32_t idesc_o = umma_idesc_bf16(128, e16, 0, 1);
      const uint32_t idesc_lo = umma_idesc_bf16(128, 64, 0, 1), idesc_hi = umma_idesc_bf16(128, e16 - 64 > 0 ? e16 - 64 : 16, 0, 1);
      // descriptors differ in their address field (16-byte units) only
      const uint64_t k_desc = umma_smem_desc(0, 0, 1024), v_desc = umma_smem_desc(0, kFlChunk, 1024);
      constexpr uint32_t kChunk16 = kFlChunk >> 4;
      const uint32_t q16 = smem_u32(smem_q + g * kch * kFlChunk) >> 4, kv16 = smem_u32(smem_kv) >> 4;
      const uint32_t t_s = tmem_base + g * 128, t_o = tmem_base + 256 + g * 128;
      const int steps1 = (p.D - (k1 - 1) * 64) >> 4, steps2 = p.R ? (p.R - (kch - k1 - 1) * 64) >> 4 : 0;   // of the parts' last chunks
      int slot = 0;                                    // of the next item, and the parity of its phase
      uint32_t phase = 0;
      auto wait_items = [&](int count) {
        for (int c = 0; c < count; ++c) {
          if (!mbar_wait(&full[slot], phase, p.status, kTimeoutFull)) return false;
          if (++slot == ring) slot = 0, phase ^= 1;
        }
        return true;
      };
      auto release = [&](int first, int count) {
        for (int c = 0; c < count; ++c, first = first + 1 == ring ? 0 : first + 1) tc_commit(&empty[first]);
      };
      auto issue_s = [&](int first) {                  // slot of the block's first key chunk
        uint64_t qd = k_desc + q16;
        uint32_t more = 0;
        for (int c = 0; c < kch; ++c) {
          const uint64_t kd = k_desc + (kv16 + first * kChunk16);
          const int steps = c == k1 - 1 ? steps1 : c == kch - 1 ? steps2 : 4;
#pragma unroll
          for (int k = 0; k < 4; ++k)
            if (k < steps) {
              umma_bf16_ss(t_s, qd + k * 2, kd + k * 2, idesc_s, more);
              more = 1;
            }
          qd += kChunk16;
          first = first + 1 == ring ? 0 : first + 1;
        }
        tc_commit(&s_full[g]);
      };
      auto issue_o = [&](int first, bool first_block) {
        const uint64_t vd = v_desc + (kv16 + first * kChunk16);
        const bool split = vch == 2 && first + 1 == ring;                // the value chunks lie at both ends of the ring
        const uint32_t idesc = split ? idesc_lo : idesc_o;
#pragma unroll
        for (int k = 0; k < kFlKeys / 16; ++k) umma_bf16_ts(t_o, t_s + k * 8, vd + k * 128, idesc, first_block && k == 0 ? 0u : 1u);
        if (split) {
          const uint64_t v2 = v_desc + kv16;
#pragma unroll
          for (int k = 0; k < kFlKeys / 16; ++k) umma_bf16_ts(t_o + 64, t_s + k * 8, v2 + k * 128, idesc_hi, first_block && k == 0 ? 0u : 1u);
        }
      };
      bool ok = mbar_wait(q_full, 0, p.status, kTimeoutFull) && wait_items(kch);
      if (ok) {
        tc_fence_after();
        issue_s(0);
        release(0, kch);
      }
      for (int j = 0; j < n_blocks && ok; ++j) {
        const bool more = j + 1 < n_blocks;            // of the other tile, perhaps
        const int sv = slot;
        if (!wait_items(vch)) break;
        if (j < nb) {
          if (!mbar_wait(&p_full[g], j & 1, p.status, kTimeoutTmemEmpty)) break;
          tc_fence_after();
          issue_o(sv, j == 0);
          if (more) release(sv, vch);
          if (j + 1 == nb) tc_commit(&o_full[g]);
        } else if (more) {
          for (int c = 0, at = sv; c < vch; ++c, at = at + 1 == ring ? 0 : at + 1) mbar_arrive(&empty[at]);
        }
        if (!more) break;
        const int sk = slot;
        if (!wait_items(kch)) break;
        if (j + 1 < nb) {                              // these scores run after the product above has read the weights
          tc_fence_after();
          issue_s(sk);
          release(sk, kch);
        } else {
          for (int c = 0, at = sk; c < kch; ++c, at = at + 1 == ring ? 0 : at + 1) mbar_arrive(&empty[at]);
        }
      }
    }
  } else if (warp < 10 && ((warp - 2) >> 2) < n_tiles) {
    // ---------------------------------------------------------------- weight groups, one per tile
    const int g = (warp - 2) >> 2;
    const int quarter = warp & 3, row = quarter * 32 + lane;
    const int row0 = w[4 + 4 * g], valid = w[4 + 4 * g + 1], head = w[4 + 4 * g + 2], pos0 = w[4 + 4 * g + 3];
    const int nb = g ? nb1 : nb0, window = p.sp.window;
    const uint32_t lane_off = static_cast<uint32_t>(quarter * 32) << 16;
    const uint32_t t_s = tmem_base + lane_off + g * 128, t_o = tmem_base + lane_off + 256 + g * 128;
    const float scale = p.sp.scale * 1.4426950408889634f;
    const uint64_t scale2 = xtc_pair(scale, scale);
    const int pos = pos0 + min(row, valid - 1);
    CapSeries cs = {};
    if (CAP != kFlashUncapped) cs = cap_series(p.sp);
    float ref = CAP == kFlashFixed ? score_reference(p.sp.cap) * 1.4426950408889634f : -INFINITY;      // reference of the weights (log2)
    uint64_t sum2 = xtc_pair(0.f, 0.f);
    bool ok = true;
    for (int j = 0; j < nb; ++j) {
      if (!mbar_wait(&s_full[g], j & 1, p.status, kTimeoutTmemFull)) {
        ok = false;
        break;
      }
      tc_fence_after();
      const int base = k0 + j * kFlKeys;                                 // position of the block's first key
      const int limit = pos + 1 - base;                                  // visible keys: [skip, limit) of the block
      const int skip = window > 0 ? pos + 1 - window - base : 0;
      const bool whole = pos0 + 1 - base >= kFlKeys && (window <= 0 || pos0 + valid - window - base <= 0);   // all 128 for every row
      if constexpr (CAP == kFlashFixed) {
        sum2 = xtc_add2(sum2, whole ? flash_fixed_weights<true>(t_s, cs, -ref, limit, skip) : flash_fixed_weights<false>(t_s, cs, -ref, limit, skip));
        tmem_st_wait();
        tc_fence_before();
        mbar_arrive(&p_full[g]);
        continue;
      }
      uint32_t pk[4][16];
      for (int pass = 0; pass < 2; ++pass) {           // a second time if the reference had to move
        const float off = ref == -INFINITY ? 0.f : -ref;
        float top;                                     // largest score relative to the reference
        uint64_t block2;
        if constexpr (CAP != kFlashUncapped)
          block2 = whole ? flash_capped_weights<true>(t_s, cs, off, limit, skip, top, pk) : flash_capped_weights<false>(t_s, cs, off, limit, skip, top, pk);
        else
          block2 = whole ? flash_weights<true>(t_s, scale2, off, limit, skip, top, pk) : flash_weights<false>(t_s, scale2, off, limit, skip, top, pk);
        const bool behind = top > kFlLag || (ref == -INFINITY && top > -INFINITY);
        if (pass == 1 || !__any_sync(0xffffffffu, behind)) {
          sum2 = xtc_add2(sum2, block2);
          break;
        }
        const float next = fmaxf(ref, top - off);
        const float f = ref == next ? 1.f : xtc_ex2(ref - next);         // 0 while nothing has been seen
        ref = next;
        sum2 = xtc_mul2(sum2, xtc_pair(f, f));
        if (j > 0) {                                   // the products of the blocks before have completed: S_j came behind them
          for (int c = 0; c < p.E; c += 32) {
            uint32_t o[32];
            tmem_ld_32x32(t_o + c, o);
            xtc_wait_load(o);
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * f);
            tmem_st_32x32(t_o + c, o);
          }
        }
      }
#pragma unroll
      for (int c = 0; c < 4; ++c) tmem_st_32x16(t_s + c * 16, pk[c]);
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(&p_full[g]);
    }
    if (p.sp.gate && row < valid) {                    // the row's gates come closer while the last products run
      const __nv_bfloat16* gate = static_cast<const __nv_bfloat16*>(p.sp.gate) + (static_cast<long long>(row0) + row) * p.sp.ldg +
                                  static_cast<long long>(head) * p.sp.gate_cols;
      for (int c = 0; c < p.sp.gate_cols; c += 64) asm volatile("prefetch.global.L1 [%0];" ::"l"(gate + c));
    }
    __syncwarp();
    if (ok) ok = mbar_wait(&o_full[g], 0, p.status, kTimeoutTmemFull);
    if (ok) {
      tc_fence_after();
      const float2 halves = xtc_unpair(sum2);
      const long long t = static_cast<long long>(row0) + row;
      const bool live = row < valid, per_column = p.sp.gate && p.sp.gate_cols != 1;
      const float inv = live ? inverse_sum(p.sp, head, ref, halves.x + halves.y) * (per_column ? 1.f : output_gate<__nv_bfloat16>(p.sp, t, head, 0))
                             : 0.f;
      __nv_bfloat16* dst = p.out + t * p.ldo + static_cast<long long>(head) * p.E;
      const __nv_bfloat16* gate = static_cast<const __nv_bfloat16*>(p.sp.gate) + t * p.sp.ldg + static_cast<long long>(head) * p.E;
#pragma unroll 1
      for (int c = 0; c < p.E; c += 32) {
        uint32_t o[32];
        tmem_ld_32x32(t_o + c, o);
        xtc_wait_load(o);
        if (!live) continue;
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          if (c + q * 8 >= p.E) continue;
          float v[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) v[i] = __uint_as_float(o[q * 8 + i]) * inv;
          if (per_column) {
            const uint4 raw = *reinterpret_cast<const uint4*>(gate + c + q * 8);
            const uint32_t gw[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
            for (int i = 0; i < 4; ++i) {
              const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gw[i]));
              v[2 * i] = __fdividef(v[2 * i], 1.f + __expf(-f.x));
              v[2 * i + 1] = __fdividef(v[2 * i + 1], 1.f + __expf(-f.y));
            }
          }
          *reinterpret_cast<uint4*>(dst + c + q * 8) =
              make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
        }
      }
      tc_fence_before();
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

// q: [rows, H * (D + R)] columns of a row-major buffer (row stride ldq); out [rows, H * E] (row stride ldo), 16-byte aligned rows.
// With a page table: k [pages, G, 16, D], v [pages, G, 16, E], key_rows = pages * G * 16, R = 0.  Without: k [key_rows, G * D]
// (row stride ldk), k2 [key_rows, R] (contiguous, R > 0), v [key_rows, G * E] (ldv).  D and R multiples of 16, at most 4 chunks of
// 64 columns together, E a multiple of 8 up to 128; cap > 0: capped scores; gate (if any): rows of 16-byte aligned columns.
int apb_flash_tc(const void* q, long long ldq, int rows, const int* work, int n_work, const int* page_table, int max_pages,
                 const void* k, long long ldk, const void* k2, const void* v, long long ldv, long long key_rows, void* out,
                 long long ldo, int H, int G, int D, int R, int E, float scale, float cap, int window, const float* sink,
                 const void* gate, long long ldg, int gate_cols, cudaStream_t stream) {
  using namespace apb;
  if (n_work <= 0) return 0;
  const int kch = (D + 63) / 64 + (R + 63) / 64;
  if (H <= 0 || G <= 0 || H % G || D <= 0 || R < 0 || E <= 0 || (D % 16) || (R % 16) || (E % 8) || kch > 4 || E > 128 ||
      (ldq % 8) || (ldo % 8) || (ldk % 8) || (ldv % 8) || key_rows <= 0 || !work || (page_table && R) || (R && !k2) || window < 0 ||
      ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(k) |
        reinterpret_cast<uintptr_t>(k2) | reinterpret_cast<uintptr_t>(v)) & 15) ||
      (gate && gate_cols != 1 && (gate_cols != E || (ldg % 8) || (reinterpret_cast<uintptr_t>(gate) & 15))))
    return kBadArgument;
  CUtensorMap tq, tk, tk2, tv;
  const int box = page_table ? kServePage : kFlKeys, heads = page_table ? 1 : G;
  int rc = make_tmap_2d(&tq, q, 2, rows, static_cast<uint64_t>(H) * (D + R), ldq, 64, 128);
  if (rc) return 1000 + rc;
  rc = make_tmap_2d(&tk, k, 2, key_rows, static_cast<uint64_t>(heads) * D, ldk, 64, box);
  if (rc) return 2000 + rc;
  rc = R ? make_tmap_2d(&tk2, k2, 2, key_rows, R, R, 64, box) : 0;
  if (rc) return 3000 + rc;
  if (!R) tk2 = tk;
  rc = make_tmap_2d(&tv, v, 2, key_rows, static_cast<uint64_t>(heads) * E, ldv, 64, box);
  if (rc) return 4000 + rc;
  const FlashParams p{work, page_table, max_pages, static_cast<__nv_bfloat16*>(out), ldo, G, D, R, E,
                      SoftmaxSpec{scale, cap, 0, 1, nullptr, 1.f, 0.f, window, sink, gate, ldg, gate_cols}, status_device_ptr()};
  auto run = [&](auto fn) -> int {
    const cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, kFlSmem);
    if (e != cudaSuccess) return static_cast<int>(e);
    fn<<<n_work, kFlThreads, kFlSmem, stream>>>(tq, tk, tk2, tv, p);
    return static_cast<int>(cudaGetLastError());
  };
  return fixed_reference(cap) ? run(flash_tc_kernel<kFlashFixed>) : cap > 0.f ? run(flash_tc_kernel<kFlashCapped>) : run(flash_tc_kernel<kFlashUncapped>);
}
}
