// Small kernels of a serving step over a RAGGED batch: several sequences, each with its own run of new tokens (a
// portion of a prompt, or one decoded token), share one packed row axis.
//
// A batch is described by per-entry arrays: e_start / e_len (rows of the entry), e_slot (state slot of its sequence)
// and e_pos0 (position of its first row, i.e. tokens of the sequence before this step).  A decode step is the special
// case "entry i = row i = slot i, e_len 0 or 1", with every array living in device buffers, so that it can be captured
// in a CUDA graph.
//
// Per-sequence state that a step reads at the entry's first rows and replaces at its last rows (the previous token,
// the convolution history) is double buffered: `parity[slot]` names the half that is read, the other half is written,
// and serve_commit flips the parity once at the end of the step.  A position-0 entry ignores whatever its slot holds.
//
// The kernels take bf16 or fp32 activations (dtype argument: 0 = bf16, 1 = fp32); the residual stream, norms and
// convolution histories are fp32 in both.
#include "common.cuh"
#include "host_utils.cuh"
#include "serve_common.cuh"

namespace apb {

// ---------------------------------------------------------------------------- embedding
// x[row] = (embed[token] (+ bigram[hash(previous token, token)])) * scale, fp32, written `copies` times (parallel residual
// streams start equal); `x0` (optional) receives the same row in the activation type (the right half of the loop-input
// operand), `kv_slot` the row's cache slot (page * 16 + offset, -1 for an entry without tokens).
template <typename T>
__global__ void __launch_bounds__(128)
embed_hash_kernel(const int* __restrict__ tokens, const int* __restrict__ row_entry, const ServeEntries e,
                  const int* __restrict__ prev, const T* __restrict__ embed, const T* __restrict__ bigram,
                  long long buckets, long long mul_prev, long long mul_cur, int vocab, int W, float scale, int copies,
                  float* __restrict__ x, T* __restrict__ x0, long long ld0, const int* __restrict__ page_table, int max_pages,
                  int* __restrict__ kv_slot) {
  pdl_entry();
  const int row = blockIdx.x;
  const int en = row_entry ? row_entry[row] : row;
  if (kv_slot && threadIdx.x == 0) {
    const int r = row - e.start[en], pos = e.pos0[en] + r;
    const bool live = r >= 0 && r < e.len[en] && pos >= 0 && pos / kServePage < max_pages;
    kv_slot[row] = live ? page_table[static_cast<long long>(en) * max_pages + pos / kServePage] * kServePage + pos % kServePage : -1;
  }
  int tok = tokens[row];
  tok = tok < 0 ? 0 : (tok >= vocab ? vocab - 1 : tok);
  const T* big = nullptr;
  if (bigram) {
    const int r = row - e.start[en];
    long long b = buckets;                        // first token of a sequence
    if (e.pos0[en] + r > 0) {
      int pt = r > 0 ? tokens[row - 1] : prev[e.slot[en]];
      pt = pt < 0 ? 0 : (pt >= vocab ? vocab - 1 : pt);
      b = (static_cast<long long>(pt) * mul_prev + static_cast<long long>(tok) * mul_cur) % buckets;
      if (b < 0) b += buckets;
    }
    big = bigram + b * W;
  }
  const T* src = embed + static_cast<long long>(tok) * W;
  for (int i = threadIdx.x; i < W; i += blockDim.x) {
    float v = to_f32(src[i]);
    if (big) v += to_f32(big[i]);
    v *= scale;
    for (int c = 0; c < copies; ++c) x[(static_cast<long long>(row) * copies + c) * W + i] = v;
    if (x0) x0[static_cast<long long>(row) * ld0 + i] = from_f32<T>(v);
  }
}

// Start of a pass over looped layers: the left half of the loop-input operand receives the residual stream in the
// activation type, and the stream itself restarts from `init` (the pass's step vector), onto which the loop-input
// projection is then accumulated.
template <typename T>
__global__ void __launch_bounds__(256)
loop_begin_kernel(float* __restrict__ x, const T* __restrict__ init, int W, T* __restrict__ out, long long ld,
                  long long n) {
  pdl_entry();
  for (long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i < n;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const int c = static_cast<int>(i % W);
    out[(i / W) * ld + c] = from_f32<T>(x[i]);
    x[i] = to_f32(init[c]);
  }
}

// ---------------------------------------------------------------------------- norm + input convolutions
// h = x / rms(x) * g  (one gain for the whole row), then up to two causal depth-wise convolutions over time that share
// h:  out_k[t] = h[t] + sum_j w_k[j] h[t - taps + 1 + j].  w_k is [taps, W]; a null w_k copies h.  The history of h
// before the entry's first row comes from the slot's state [2][taps - 1][W]; the last taps - 1 rows of h replace it.
// One block = up to kNormRows consecutive rows of one entry (tiles[2 i] = entry, tiles[2 i + 1] = first row; without a
// table block i is entry i, which then has at most one row).
constexpr int kNormRows = 8;
constexpr int kNormThreads = 256;

template <typename T>
__global__ void __launch_bounds__(kNormThreads)
norm_conv_kernel(const float* __restrict__ x, const T* __restrict__ gain, const T* __restrict__ w1,
                 const T* __restrict__ w2, T* __restrict__ out1, T* __restrict__ out2, float* __restrict__ state,
                 const int* __restrict__ parity, const ServeEntries e, const int* __restrict__ tiles, int W, int taps,
                 float eps) {
  pdl_entry();
  extern __shared__ float rs[];                    // [hist + kNormRows] row factors g / rms, rows r0 - hist ...
  const int en = tiles ? tiles[2 * blockIdx.x] : blockIdx.x;
  const int r0 = tiles ? tiles[2 * blockIdx.x + 1] : 0;
  const int len = e.len[en];
  if (r0 >= len) return;
  const int nr = min(kNormRows, len - r0);
  const int hist = taps - 1;
  const int start = e.start[en], pos0 = e.pos0[en];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float g = to_f32(*gain);
  for (int i = warp; i < hist + nr; i += kNormThreads / 32) {
    const int r = r0 - hist + i;
    float ss = 0.f;
    if (r >= 0) {
      const float* xr = x + static_cast<long long>(start + r) * W;
      if ((W & 3) == 0) {
        for (int c = lane * 4; c < W; c += 128) {
          const float4 v = *reinterpret_cast<const float4*>(xr + c);
          ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
      } else {
        for (int c = lane; c < W; c += 32) ss += xr[c] * xr[c];
      }
      ss = warp_sum(ss);
    }
    if (lane == 0) rs[i] = g / sqrtf(ss / W + eps);
  }
  __syncthreads();
  const int slot = e.slot[en];
  const float* old_h = nullptr;
  float* new_h = nullptr;
  if (hist > 0 && slot >= 0) {
    const int par = parity[slot] & 1;
    old_h = state + (static_cast<long long>(slot) * 2 + par) * hist * W;
    new_h = state + (static_cast<long long>(slot) * 2 + (par ^ 1)) * hist * W;
  }
  // h of row r (relative to the entry; negative rows come from the state or lie before the sequence)
  auto h_at = [&](int r, int c) -> float {
    if (r >= 0) return x[static_cast<long long>(start + r) * W + c] * rs[r - r0 + hist];
    return (pos0 + r >= 0 && old_h) ? old_h[static_cast<long long>(hist + r) * W + c] : 0.f;
  };
  for (int c = threadIdx.x; c < W; c += kNormThreads) {
    for (int i = 0; i < nr; ++i) {
      const int r = r0 + i;
      const float h = h_at(r, c);
      float a1 = h, a2 = h;
      if (w1 || w2) {
#pragma unroll 4
        for (int j = 0; j < taps; ++j) {
          const float hv = j == hist ? h : h_at(r - hist + j, c);
          if (w1) a1 += to_f32(w1[j * W + c]) * hv;
          if (w2) a2 += to_f32(w2[j * W + c]) * hv;
        }
      }
      const long long o = static_cast<long long>(start + r) * W + c;
      out1[o] = from_f32<T>(a1);
      if (out2) out2[o] = from_f32<T>(a2);
    }
    if (new_h && r0 + nr == len)
      for (int i = 0; i < hist; ++i) new_h[static_cast<long long>(i) * W + c] = h_at(len - hist + i, c);
  }
}

template <typename T>
__device__ __forceinline__ float2 load2(const T* p) {
  if constexpr (sizeof(T) == 2)
    return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
  else
    return *reinterpret_cast<const float2*>(p);
}
template <typename T>
__device__ __forceinline__ void store2(T* p, float2 v) {
  if constexpr (sizeof(T) == 2)
    *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(v.x, v.y);
  else
    *reinterpret_cast<float2*>(p) = v;
}
__device__ __forceinline__ void fma2(float2& a, const float2& w, const float2& h) {
  a.x += w.x * h.x;
  a.y += w.y * h.y;
}

// The same for a compile-time number of taps and W a multiple of 4: two channels per thread, the rows of the tile
// loaded at once, the window in registers.  ROWS = 1 (decoded tokens) is for launches without a tile table.
template <typename T, int TAPS, int ROWS>
__global__ void __launch_bounds__(kNormThreads, ROWS == 1 ? 4 : 2)
norm_conv_vec_kernel(const float* __restrict__ x, const T* __restrict__ gain, const T* __restrict__ w1,
                     const T* __restrict__ w2, T* __restrict__ out1, T* __restrict__ out2, float* __restrict__ state,
                     const int* __restrict__ parity, const ServeEntries e, const int* __restrict__ tiles, int W,
                     float eps) {
  pdl_entry();
  constexpr int kHist = TAPS - 1;
  __shared__ float rs[kHist + ROWS];
  __shared__ float red[kNormThreads / 32];
  const int en = tiles ? tiles[2 * blockIdx.x] : blockIdx.x;
  const int r0 = tiles ? tiles[2 * blockIdx.x + 1] : 0;
  const int len = e.len[en];
  if (r0 >= len) return;
  const int nr = min(ROWS, len - r0);
  const int start = e.start[en], pos0 = e.pos0[en];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float g = to_f32(*gain);
  if (len == 1) {                                  // a decoded token: the whole block sums its row
    const float* xr = x + static_cast<long long>(start) * W;
    float ss = 0.f;
#pragma unroll 4
    for (int c = threadIdx.x * 4; c < W; c += kNormThreads * 4) {
      const float4 v = *reinterpret_cast<const float4*>(xr + c);
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    if (threadIdx.x == 0) {
      ss = 0.f;
      for (int i = 0; i < kNormThreads / 32; ++i) ss += red[i];
      rs[kHist] = g / sqrtf(ss / W + eps);
    }
  } else {
    for (int i = warp; i < kHist + nr; i += kNormThreads / 32) {
      const int r = r0 - kHist + i;
      if (r < 0) continue;
      const float* xr = x + static_cast<long long>(start + r) * W;
      float ss = 0.f;
#pragma unroll 8
      for (int c = lane * 4; c < W; c += 128) {
        const float4 v = *reinterpret_cast<const float4*>(xr + c);
        ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
      }
      ss = warp_sum(ss);
      if (lane == 0) rs[i] = g / sqrtf(ss / W + eps);
    }
  }
  __syncthreads();
  const int slot = e.slot[en];
  const float* old_h = nullptr;
  float* new_h = nullptr;
  if (kHist > 0 && slot >= 0) {
    const int par = parity[slot] & 1;
    old_h = state + (static_cast<long long>(slot) * 2 + par) * kHist * W;
    new_h = state + (static_cast<long long>(slot) * 2 + (par ^ 1)) * kHist * W;
  }
  const float2 zero = make_float2(0.f, 0.f);
#pragma unroll (ROWS == 1 ? 2 : 1)
  for (int c = threadIdx.x * 2; c < W; c += kNormThreads * 2) {
    float2 h[kHist + ROWS];                   // rows r0 - hist .. r0 + ROWS - 1
    const float* xp = x + static_cast<long long>(start + r0 - kHist) * W + c;
#pragma unroll
    for (int i = 0; i < kHist + ROWS; ++i, xp += W) {
      const int r = r0 - kHist + i;
      h[i] = zero;
      if (r >= 0 && i < kHist + nr)
        h[i] = *reinterpret_cast<const float2*>(xp);
      else if (r < 0 && pos0 + r >= 0 && old_h)
        h[i] = *reinterpret_cast<const float2*>(old_h + static_cast<long long>(kHist + r) * W + c);
    }
    float2 a[TAPS], b[TAPS];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      a[j] = w1 ? load2(w1 + static_cast<long long>(j) * W + c) : zero;
      b[j] = w2 ? load2(w2 + static_cast<long long>(j) * W + c) : zero;
    }
#pragma unroll
    for (int i = 0; i < kHist + ROWS; ++i)
      if (r0 - kHist + i >= 0 && i < kHist + nr) {
        const float f = rs[i];
        h[i] = make_float2(h[i].x * f, h[i].y * f);
      }
    long long o = static_cast<long long>(start + r0) * W + c;
#pragma unroll
    for (int i = 0; i < ROWS; ++i, o += W)
      if (i < nr) {
        float2 y1 = h[i + kHist], y2 = y1;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
          fma2(y1, a[j], h[i + j]);
          fma2(y2, b[j], h[i + j]);
        }
        store2(out1 + o, y1);
        if (out2) store2(out2 + o, y2);
      }
    if (new_h && r0 + nr == len) {
#pragma unroll
      for (int i = 0; i < kHist + ROWS; ++i)  // rows len - hist .. len - 1
        if (i >= nr && i < nr + kHist) *reinterpret_cast<float2*>(new_h + static_cast<long long>(i - nr) * W + c) = h[i];
    }
  }
}

// Final norm of selected rows: out[i] = x[rows[i]] / rms * (offset + g) (rows == null: row i), with one gain (gain_step 0) or
// one per channel (gain_step 1).  One block per row.
template <typename T>
__global__ void __launch_bounds__(256)
gain_norm_rows_kernel(const float* __restrict__ x, const int* __restrict__ rows, const T* __restrict__ gain,
                      int gain_step, float offset, T* __restrict__ out, int W, int groups, float eps) {
  pdl_entry();
  extern __shared__ float gn_sums[];           // [max(8, groups)]
  const float* xr = x + static_cast<long long>(rows ? rows[blockIdx.x] : static_cast<int>(blockIdx.x)) * W;
  const int size = W / groups, parts = group_parts(groups);
  group_sums(groups, size, gn_sums, [&](int c) { return xr[c]; });
  __syncthreads();
  float f = groups == 1 ? group_rms_inverse(gn_sums, 0, parts, size, eps) : 0.f;
  for (int c = threadIdx.x; c < W; c += 256) {
    if (groups > 1) f = group_rms_inverse(gn_sums, c / size, parts, size, eps);
    out[static_cast<long long>(blockIdx.x) * W + c] = from_f32<T>(xr[c] * f * (offset + to_f32(gain[c * gain_step])));
  }
}

// ---------------------------------------------------------------------------- q/k norm + paged cache write
// p [rows, ld]: q heads at column q_col, k heads at k_col, v heads at v_col.  q and k heads are divided by their root
// mean square (no weight); q goes back in place, k and v go to their cache slot (page * 16 + offset, < 0: nothing is
// written) of kcache [pages, G, 16, D] and vcache [pages, G, 16, E].  One warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(256)
qk_norm_cache_kernel(T* __restrict__ p, long long ld, int q_col, int k_col, int v_col, const int* __restrict__ kv_slot,
                     T* __restrict__ kcache, T* __restrict__ vcache, int rows, int H, int G, int D, int E, float eps) {
  pdl_entry();
  const int lane = threadIdx.x & 31;
  const long long gw = (blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x) >> 5;
  const int units = H + 2 * G;
  if (gw >= static_cast<long long>(rows) * units) return;
  const int row = static_cast<int>(gw / units), u = static_cast<int>(gw % units);
  T* pr = p + static_cast<long long>(row) * ld;
  const bool is_q = u < H, is_v = u >= H + G;
  const int hk = is_q ? u : (is_v ? u - H - G : u - H);
  const int n = is_v ? E : D;
  T* src = pr + (is_q ? q_col : is_v ? v_col : k_col) + static_cast<long long>(hk) * n;
  T* dst = src;
  if (!is_q) {
    const int slot = kv_slot[row];
    if (slot < 0) return;
    dst = (is_v ? vcache : kcache) + ((static_cast<long long>(slot / kServePage) * G + hk) * kServePage + slot % kServePage) * n;
  }
  const bool vec = sizeof(T) == 2 && (n & 7) == 0 && n <= 256 && (reinterpret_cast<uintptr_t>(src) & 15) == 0;
  if (vec) {                                       // 8 elements per lane, one 16-byte access each way
    uint4 raw = make_uint4(0u, 0u, 0u, 0u);
    const bool mine = lane * 8 < n;
    if (mine) raw = *reinterpret_cast<const uint4*>(src + lane * 8);
    if (!is_v) {
      __nv_bfloat162* h2 = reinterpret_cast<__nv_bfloat162*>(&raw);
      float f[8], ss = 0.f;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 t = __bfloat1622float2(h2[i]);
        f[2 * i] = t.x;
        f[2 * i + 1] = t.y;
        ss += t.x * t.x + t.y * t.y;
      }
      const float r = 1.f / sqrtf(warp_sum(ss) / n + eps);
      raw.x = pack_bf16x2(f[0] * r, f[1] * r);
      raw.y = pack_bf16x2(f[2] * r, f[3] * r);
      raw.z = pack_bf16x2(f[4] * r, f[5] * r);
      raw.w = pack_bf16x2(f[6] * r, f[7] * r);
    }
    if (mine) *reinterpret_cast<uint4*>(dst + lane * 8) = raw;
    return;
  }
  float r = 1.f;
  if (!is_v) {
    float ss = 0.f;
    for (int i = lane; i < n; i += 32) {
      const float v = to_f32(src[i]);
      ss += v * v;
    }
    r = 1.f / sqrtf(warp_sum(ss) / n + eps);
  }
  for (int i = lane; i < n; i += 32) dst[i] = is_v ? src[i] : from_f32<T>(to_f32(src[i]) * r);
}

// ---------------------------------------------------------------------------- rotation + paged cache write
// Rotary positions on neighbouring pairs: of every head of D columns the first `rot` are rotated, dimension 2i with 2i + 1,
// by the angles of the row's position (tables [positions, rot / 2]).  q (HQ heads at q_col) is rotated in place; k (HK
// heads at k_col) goes to kcache [pages, G, 16, HK / G * D], v (G heads of E at v_col) to vcache [pages, G, 16, E].  HK = 0:
// q only.  One thread handles V neighbouring columns (8 bf16, or one pair).
template <typename T, int V>
__global__ void __launch_bounds__(256)
rope_cache_kernel(T* __restrict__ p, long long ld, int q_col, int k_col, int v_col, const int* __restrict__ row_entry,
                  const ServeEntries e, const int* __restrict__ kv_slot, const float* __restrict__ cos_t,
                  const float* __restrict__ sin_t, int rot, T* __restrict__ kcache, T* __restrict__ vcache, int rows,
                  int HQ, int HK, int G, int D, int E) {
  pdl_entry();
  const int du = (D + V - 1) / V, eu = (E + V - 1) / V;             // units of a head
  const int nq = HQ * du, nk = HK * du, units = nq + nk + (HK ? G * eu : 0);
  const long long idx = blockIdx.x * 256LL + threadIdx.x;
  if (idx >= static_cast<long long>(rows) * units) return;
  const int row = static_cast<int>(idx / units);
  int u = static_cast<int>(idx % units);
  const int en = row_entry ? row_entry[row] : row;
  const int r = row - e.start[en];
  if (r < 0 || r >= e.len[en]) return;
  const bool is_q = u < nq, is_v = u >= nq + nk;
  u -= is_q ? 0 : (is_v ? nq + nk : nq);
  const int w = is_v ? E : D, per = is_v ? eu : du;
  const int head = u / per, c0 = (u % per) * V;
  const int n = V == 8 ? 8 : min(V, w - c0);
  T* src = p + static_cast<long long>(row) * ld + (is_q ? q_col : is_v ? v_col : k_col) + static_cast<long long>(head) * w + c0;
  T* dst = src;
  if (!is_q) {
    const int slot = kv_slot[row];
    if (slot < 0) return;
    const int maps = HK / G;                                         // key heads side by side in one cache row
    const int g = is_v ? head : head / maps;
    const long long tok = (static_cast<long long>(slot / kServePage) * G + g) * kServePage + slot % kServePage;
    dst = is_v ? vcache + tok * E + c0 : kcache + (tok * maps + head % maps) * D + c0;
  }
  const long long tr = static_cast<long long>(e.pos0[en] + r) * (rot >> 1);
  if constexpr (V == 8) {
    uint4 raw = *reinterpret_cast<const uint4*>(src);
    if (!is_v && c0 < rot) {
      uint32_t* w2 = reinterpret_cast<uint32_t*>(&raw);
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (c0 + 2 * i < rot) {
          const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w2[i]));
          const float c = cos_t[tr + (c0 >> 1) + i], s = sin_t[tr + (c0 >> 1) + i];
          w2[i] = pack_bf16x2(f.x * c - f.y * s, f.y * c + f.x * s);
        }
    }
    *reinterpret_cast<uint4*>(dst) = raw;
  } else {
    T a = src[0], b = n > 1 ? src[1] : src[0];
    if (!is_v && c0 + 1 < rot) {
      const float c = cos_t[tr + (c0 >> 1)], s = sin_t[tr + (c0 >> 1)];
      const float x = to_f32(a), y = to_f32(b);
      a = from_f32<T>(x * c - y * s);
      b = from_f32<T>(y * c + x * s);
    }
    dst[0] = a;
    if (n > 1) dst[1] = b;
  }
}

// ---------------------------------------------------------------------------- norm of whole projections + rotation + page write
// p [rows, ld]: H query heads of D columns at q_col, G key heads at k_col, G value heads of E at v_col.  All query columns are
// divided by their common root mean square and multiplied by wq [H D], the key columns likewise (wk [G D]); then the first
// `rot` columns of every head are rotated, dimension i with i + rot / 2, by the angles of the row's position.  q goes back in
// place, k and v to their cache slot.  One block per row; a thread owns V neighbouring columns and their partners.
constexpr int kRowNormThreads = 256;

template <typename T, int V>
__device__ __forceinline__ void load_cols(const T* p, float (&v)[V]) {
  if constexpr (V == 8) {
    const uint4 r = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w[i]));
      v[2 * i] = f.x;
      v[2 * i + 1] = f.y;
    }
  } else if constexpr (V == 2) {
    const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
    v[0] = f.x;
    v[1] = f.y;
  } else {
    v[0] = to_f32(*p);
  }
}
template <typename T, int V>
__device__ __forceinline__ void store_cols(T* p, const float (&v)[V]) {
  if constexpr (V == 8)
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
  else if constexpr (V == 2)
    *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(v[0], v[1]);
  else
    *p = from_f32<T>(v[0]);
}

template <typename T, int V>
__global__ void __launch_bounds__(kRowNormThreads)
row_norm_rope_cache_kernel(T* __restrict__ p, long long ld, int q_col, int k_col, int v_col, const T* __restrict__ wq,
                           const T* __restrict__ wk, const int* __restrict__ row_entry, const ServeEntries e,
                           const int* __restrict__ kv_slot, const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                           int rot, T* __restrict__ kcache, T* __restrict__ vcache, int H, int G, int D, int E, float eps) {
  pdl_entry();
  __shared__ float red[2][kRowNormThreads / 32];
  const int row = blockIdx.x;
  const int en = row_entry ? row_entry[row] : row;
  const int at = row - e.start[en];
  if (at < 0 || at >= e.len[en]) return;
  T* pr = p + static_cast<long long>(row) * ld;
  float s[2] = {0.f, 0.f};
  for (int i = threadIdx.x * V; i < (H + G) * D; i += kRowNormThreads * V) {
    float v[V];
    const bool k = i >= H * D;
    load_cols<T, V>(k ? pr + k_col + (i - H * D) : pr + q_col + i, v);
#pragma unroll
    for (int j = 0; j < V; ++j) s[k ? 1 : 0] += v[j] * v[j];
  }
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    s[k] = warp_sum(s[k]);
    if ((threadIdx.x & 31) == 0) red[k][threadIdx.x >> 5] = s[k];
  }
  __syncthreads();
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    s[k] = 0.f;
#pragma unroll
    for (int i = 0; i < kRowNormThreads / 32; ++i) s[k] += red[k][i];
    s[k] = 1.f / sqrtf(s[k] / ((k ? G : H) * D) + eps);
  }
  const int slot = kv_slot[row];
  const long long page = slot / kServePage, off = slot % kServePage;
  const int half = rot >> 1, per = (D - half) / V;              // units of a head: pairs of runs, then runs that are not rotated
  const long long tr = static_cast<long long>(e.pos0[en] + at) * half;
  for (int u = threadIdx.x; u < (H + G) * per; u += kRowNormThreads) {
    const int hh = u / per, c = (u % per) * V;
    const bool k = hh >= H;
    const int head = k ? hh - H : hh;
    if (k && slot < 0) continue;
    const T* src = pr + (k ? k_col : q_col) + head * D;
    const T* w = (k ? wk : wq) + head * D;
    T* dst = k ? kcache + ((page * G + head) * kServePage + off) * D : pr + q_col + head * D;
    const float r = s[k ? 1 : 0];
    const int c0 = c < half ? c : c + half;
    float a[V], g[V];
    load_cols<T, V>(src + c0, a);
    load_cols<T, V>(w + c0, g);
#pragma unroll
    for (int j = 0; j < V; ++j) a[j] *= r * g[j];
    if (c < half) {
      float b[V];
      load_cols<T, V>(src + c0 + half, b);
      load_cols<T, V>(w + c0 + half, g);
#pragma unroll
      for (int j = 0; j < V; ++j) {
        b[j] *= r * g[j];
        const float cs = cos_t[tr + c0 + j], sn = sin_t[tr + c0 + j], x = a[j];
        a[j] = x * cs - b[j] * sn;
        b[j] = b[j] * cs + x * sn;
      }
      store_cols<T, V>(dst + c0 + half, b);
    }
    store_cols<T, V>(dst + c0, a);
  }
  if (slot < 0) return;
  for (int i = threadIdx.x * V; i < G * E; i += kRowNormThreads * V) {
    float v[V];
    load_cols<T, V>(pr + v_col + i, v);
    store_cols<T, V>(vcache + ((page * G + i / E) * kServePage + off) * E + i % E, v);
  }
}

// ---------------------------------------------------------------------------- half-split rotation + value norm + page write
// p [rows, ld]: H query heads of D columns at q_col, G key heads at k_col, G value heads of E at v_col.  The first `rot` columns of
// every query and key head are rotated, dimension i with i + rot / 2, by the angles of the row's position; with v_eps >= 0 every
// value head is divided by its root mean square.  q goes back in place, k and v to their cache slot.  One warp per (row, head).
template <typename T, int V>
__global__ void __launch_bounds__(256)
half_rope_cache_kernel(T* __restrict__ p, long long ld, int q_col, int k_col, int v_col, const int* __restrict__ row_entry,
                       const ServeEntries e, const int* __restrict__ kv_slot, const float* __restrict__ cos_t,
                       const float* __restrict__ sin_t, int rot, T* __restrict__ kcache, T* __restrict__ vcache, int rows, int H,
                       int G, int D, int E, float v_eps) {
  pdl_entry();
  const int lane = threadIdx.x & 31;
  const unsigned heads = H + 2 * G, gw = blockIdx.x * 8u + (threadIdx.x >> 5);       // rows * heads fits: the entry point checks
  if (gw >= rows * heads) return;
  const int row = static_cast<int>(gw / heads), hh = static_cast<int>(gw % heads);
  const int en = row_entry ? row_entry[row] : row;
  const int at = row - e.start[en];
  if (at < 0 || at >= e.len[en]) return;
  const bool is_q = hh < H, is_v = hh >= H + G;
  const int head = is_q ? hh : is_v ? hh - H - G : hh - H;
  const int slot = is_q ? 0 : kv_slot[row];
  if (slot < 0) return;
  T* pr = p + static_cast<long long>(row) * ld;
  const long long tok = (static_cast<long long>(slot / kServePage) * G + head) * kServePage + slot % kServePage;
  if (is_v) {
    const T* src = pr + v_col + head * E;
    T* dst = vcache + tok * E;
    float r = 1.f;
    if (v_eps >= 0.f) {
      float ss = 0.f;
      for (int c = lane * V; c < E; c += 32 * V) {
        float a[V];
        load_cols<T, V>(src + c, a);
#pragma unroll
        for (int i = 0; i < V; ++i) ss += a[i] * a[i];
      }
      r = 1.f / sqrtf(warp_sum(ss) / E + v_eps);
    }
    for (int c = lane * V; c < E; c += 32 * V) {
      float a[V];
      load_cols<T, V>(src + c, a);
#pragma unroll
      for (int i = 0; i < V; ++i) a[i] *= r;
      store_cols<T, V>(dst + c, a);
    }
    return;
  }
  T* src = pr + (is_q ? q_col : k_col) + head * D;
  T* dst = is_q ? src : kcache + tok * D;
  const int half = rot >> 1;
  const long long tr = static_cast<long long>(e.pos0[en] + at) * half;
  for (int c = lane * V; c < half; c += 32 * V) {
    float a[V], b[V];
    load_cols<T, V>(src + c, a);
    load_cols<T, V>(src + c + half, b);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      const float cs = cos_t[tr + c + i], sn = sin_t[tr + c + i], u = a[i];
      a[i] = u * cs - b[i] * sn;
      b[i] = b[i] * cs + u * sn;
    }
    store_cols<T, V>(dst + c, a);
    store_cols<T, V>(dst + c + half, b);
  }
  if (!is_q)
    for (int c = rot + lane * V; c < D; c += 32 * V) {
      float a[V];
      load_cols<T, V>(src + c, a);
      store_cols<T, V>(dst + c, a);
    }
}

// ---------------------------------------------------------------------------- end of a step
// Every entry that fed tokens: remember its last token and flip the parity of its double-buffered state.
__global__ void __launch_bounds__(128)
serve_commit_kernel(const int* __restrict__ tokens, const ServeEntries e, int n_entries, int* __restrict__ prev,
                    int* __restrict__ parity) {
  pdl_entry();
  const int en = blockIdx.x * blockDim.x + threadIdx.x;
  if (en >= n_entries) return;
  const int len = e.len[en], slot = e.slot[en];
  if (len <= 0 || slot < 0) return;
  prev[slot] = tokens[e.start[en] + len - 1];
  parity[slot] ^= 1;
}

}  // namespace apb

extern "C" {
using namespace apb;

int apb_embed_hash(const int* tokens, const int* row_entry, const int* e_start, const int* e_len, const int* e_slot,
                   const int* e_pos0, const int* prev, const void* embed, const void* bigram, long long buckets,
                   long long mul_prev, long long mul_cur, int vocab, int W, float scale, int copies, float* x, void* x0,
                   long long ld0, const int* page_table, int max_pages, int* kv_slot, int rows, int dtype,
                   cudaStream_t s) {
  if (rows <= 0) return 0;
  if (!tokens || !embed || !x || copies < 1 || (bigram && (buckets <= 0 || !prev)) || (kv_slot && !page_table)) return kBadArgument;
  const ServeEntries e{e_start, e_len, e_slot, e_pos0};
  APB_SERVE_DTYPE(dtype, return static_cast<int>(launch_kernel(
                             embed_hash_kernel<T>, dim3(rows), dim3(128), 0, s, tokens, row_entry, e, prev,
                             static_cast<const T*>(embed), static_cast<const T*>(bigram), buckets, mul_prev, mul_cur,
                             vocab, W, scale, copies, x, static_cast<T*>(x0), ld0, page_table, max_pages, kv_slot)));
}

int apb_loop_begin(float* x, const void* init, int rows, int W, void* out, long long ld, int dtype, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (!x || !init || !out) return kBadArgument;
  const long long n = static_cast<long long>(rows) * W;
  const int grid = static_cast<int>(n / 256 + 1 < sm_count() * 8 ? n / 256 + 1 : sm_count() * 8);
  APB_SERVE_DTYPE(dtype, return static_cast<int>(launch_kernel(loop_begin_kernel<T>, dim3(grid), dim3(256), 0, s, x,
                                                               static_cast<const T*>(init), W, static_cast<T*>(out), ld,
                                                               n)));
}

// tiles: device int32 [n_tiles][2] or null (then n_tiles is the number of entries, none longer than one row).
int apb_norm_conv(const float* x, const void* gain, const void* w1, const void* w2, void* out1, void* out2,
                  float* state, const int* parity, const int* e_start, const int* e_len, const int* e_slot,
                  const int* e_pos0, const int* tiles, int n_tiles, int W, int taps, float eps, int dtype,
                  cudaStream_t s) {
  if (n_tiles <= 0) return 0;
  if (taps < 1 || taps > 1024 || !x || !gain || !out1 || (taps > 1 && (!state || !parity))) return kBadArgument;
  const ServeEntries e{e_start, e_len, e_slot, e_pos0};
  if ((W & 3) == 0 && taps <= 5) {
#define APB_NORM_CONV(TT)                                                                                             \
  return static_cast<int>(launch_kernel(tiles ? norm_conv_vec_kernel<T, TT, kNormRows> : norm_conv_vec_kernel<T, TT, 1>, \
                                        dim3(n_tiles), dim3(kNormThreads), 0, s, x,                                   \
                                        static_cast<const T*>(gain), static_cast<const T*>(w1),                       \
                                        static_cast<const T*>(w2), static_cast<T*>(out1), static_cast<T*>(out2),      \
                                        state, parity, e, tiles, W, eps))
    APB_SERVE_DTYPE(dtype, if (taps == 1) APB_NORM_CONV(1); if (taps == 2) APB_NORM_CONV(2); if (taps == 3) APB_NORM_CONV(3);
                    if (taps == 4) APB_NORM_CONV(4); APB_NORM_CONV(5));
#undef APB_NORM_CONV
  }
  const size_t smem = (taps - 1 + kNormRows) * sizeof(float);
  APB_SERVE_DTYPE(dtype, return static_cast<int>(launch_kernel(
                             norm_conv_kernel<T>, dim3(n_tiles), dim3(kNormThreads), smem, s, x,
                             static_cast<const T*>(gain), static_cast<const T*>(w1), static_cast<const T*>(w2),
                             static_cast<T*>(out1), static_cast<T*>(out2), state, parity, e, tiles, W, taps, eps)));
}

int apb_gain_norm_rows(const float* x, const int* rows, const void* gain, int gain_step, float offset, void* out, int n, int W,
                       int groups, float eps, int dtype, cudaStream_t s) {
  if (n <= 0) return 0;
  if (W <= 0 || groups < 1 || W % groups || groups > 8192) return kBadArgument;
  const size_t smem = (groups > 8 ? groups : 8) * sizeof(float);
  APB_SERVE_DTYPE(dtype, return static_cast<int>(launch_kernel(gain_norm_rows_kernel<T>, dim3(n), dim3(256), smem, s, x, rows,
                                                               static_cast<const T*>(gain), gain_step, offset,
                                                               static_cast<T*>(out), W, groups, eps)));
}

int apb_qk_norm_cache(void* p, long long ld, int q_col, int k_col, int v_col, const int* kv_slot, void* kcache,
                      void* vcache, int rows, int H, int G, int D, int E, float eps, int dtype, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (H <= 0 || G <= 0 || D <= 0 || E <= 0 || H % G) return kBadArgument;
  const long long warps = static_cast<long long>(rows) * (H + 2 * G);
  const int grid = static_cast<int>((warps * 32 + 255) / 256);
  APB_SERVE_DTYPE(dtype, return static_cast<int>(launch_kernel(
                             qk_norm_cache_kernel<T>, dim3(grid), dim3(256), 0, s, static_cast<T*>(p), ld, q_col, k_col,
                             v_col, kv_slot, static_cast<T*>(kcache), static_cast<T*>(vcache), rows, H, G, D, E, eps)));
}

// row_entry [rows] or null (row i belongs to entry i).  HK = 0: only q is rotated (a layer that reads another layer's cache).
int apb_rope_cache(void* p, long long ld, int q_col, int k_col, int v_col, const int* row_entry, const int* e_start,
                   const int* e_len, const int* e_slot, const int* e_pos0, const int* kv_slot, const float* cos_t,
                   const float* sin_t, int rot, void* kcache, void* vcache, int rows, int HQ, int HK, int G, int D, int E,
                   int dtype, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (HQ <= 0 || HK < 0 || G <= 0 || HK % G || D <= 0 || E <= 0 || rot < 0 || (rot & 1) || rot > D ||
      (rot && (!cos_t || !sin_t)) || (HK && (!kcache || !vcache || !kv_slot)))
    return kBadArgument;
  const ServeEntries e{e_start, e_len, e_slot, e_pos0};
  const bool vec = dtype == 0 && !((D | E | q_col | (HK ? k_col | v_col : 0)) & 7) && !(ld & 7) &&
                   !((reinterpret_cast<uintptr_t>(p) | reinterpret_cast<uintptr_t>(kcache) | reinterpret_cast<uintptr_t>(vcache)) & 15);
  const int V = vec ? 8 : 2;
  const int du = (D + V - 1) / V, eu = (E + V - 1) / V;
  const long long n = static_cast<long long>(rows) * (static_cast<long long>(HQ + HK) * du + (HK ? G * eu : 0));
  const int grid = static_cast<int>((n + 255) / 256);
#define APB_ROPE(TT, VV)                                                                                              \
  return static_cast<int>(launch_kernel(rope_cache_kernel<TT, VV>, dim3(grid), dim3(256), 0, s, static_cast<TT*>(p), ld, \
                                        q_col, k_col, v_col, row_entry, e, kv_slot, cos_t, sin_t, rot,                \
                                        static_cast<TT*>(kcache), static_cast<TT*>(vcache), rows, HQ, HK, G, D, E))
  if (vec) APB_ROPE(__nv_bfloat16, 8);
  APB_SERVE_DTYPE(dtype, APB_ROPE(T, 2));
#undef APB_ROPE
}

// row_entry [rows] or null (row i belongs to entry i); wq [H D], wk [G D].
int apb_row_norm_rope_cache(void* p, long long ld, int q_col, int k_col, int v_col, const void* wq, const void* wk,
                            const int* row_entry, const int* e_start, const int* e_len, const int* e_slot, const int* e_pos0,
                            const int* kv_slot, const float* cos_t, const float* sin_t, int rot, void* kcache, void* vcache,
                            int rows, int H, int G, int D, int E, float eps, int dtype, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (H <= 0 || G <= 0 || D <= 0 || E <= 0 || rot < 0 || (rot & 1) || rot > D || (rot && (!cos_t || !sin_t)) || !kv_slot)
    return kBadArgument;
  const ServeEntries e{e_start, e_len, e_slot, e_pos0};
  const bool vec = dtype == 0 && !((D | E | q_col | k_col | v_col) & 7) && !(rot & 15) && !(ld & 7) &&
                   !((reinterpret_cast<uintptr_t>(p) | reinterpret_cast<uintptr_t>(kcache) | reinterpret_cast<uintptr_t>(vcache) |
                      reinterpret_cast<uintptr_t>(wq) | reinterpret_cast<uintptr_t>(wk)) & 15);
#define APB_ROW_NORM(TT, VV)                                                                                               \
  return static_cast<int>(launch_kernel(row_norm_rope_cache_kernel<TT, VV>, dim3(rows), dim3(kRowNormThreads), 0, s,       \
                                        static_cast<TT*>(p), ld, q_col, k_col, v_col, static_cast<const TT*>(wq),          \
                                        static_cast<const TT*>(wk), row_entry, e, kv_slot, cos_t, sin_t, rot,              \
                                        static_cast<TT*>(kcache), static_cast<TT*>(vcache), H, G, D, E, eps))
  if (vec) APB_ROW_NORM(__nv_bfloat16, 8);
  APB_SERVE_DTYPE(dtype, APB_ROW_NORM(T, 1));
#undef APB_ROW_NORM
}

// row_entry [rows] or null (row i belongs to entry i); v_eps < 0: values are stored as they are.
int apb_half_rope_cache(void* p, long long ld, int q_col, int k_col, int v_col, const int* row_entry, const int* e_start,
                        const int* e_len, const int* e_slot, const int* e_pos0, const int* kv_slot, const float* cos_t,
                        const float* sin_t, int rot, void* kcache, void* vcache, int rows, int H, int G, int D, int E, float v_eps,
                        int dtype, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (H <= 0 || G <= 0 || D <= 0 || E <= 0 || rot < 0 || (rot & 1) || rot > D || (rot && (!cos_t || !sin_t)) || !kv_slot || !kcache ||
      !vcache)
    return kBadArgument;
  const ServeEntries e{e_start, e_len, e_slot, e_pos0};
  const uintptr_t at = reinterpret_cast<uintptr_t>(p) | reinterpret_cast<uintptr_t>(kcache) | reinterpret_cast<uintptr_t>(vcache);
  const bool vec = dtype == 0 && !((D | E | q_col | k_col | v_col) & 1) && !(rot & 3) && !(ld & 1) && !(at & 3);
  const long long warps = static_cast<long long>(rows) * (H + 2 * G);
  if (warps > 0x7fffffffLL) return kBadArgument;
  const dim3 grid(static_cast<unsigned>((warps + 7) / 8));
#define APB_HALF_ROPE(TT, VV)                                                                                             \
  return static_cast<int>(launch_kernel(half_rope_cache_kernel<TT, VV>, grid, dim3(256), 0, s, static_cast<TT*>(p), ld,   \
                                        q_col, k_col, v_col, row_entry, e, kv_slot, cos_t, sin_t, rot,                    \
                                        static_cast<TT*>(kcache), static_cast<TT*>(vcache), rows, H, G, D, E, v_eps))
  if (vec) APB_HALF_ROPE(__nv_bfloat16, 2);
  APB_SERVE_DTYPE(dtype, APB_HALF_ROPE(T, 1));
#undef APB_HALF_ROPE
}

int apb_serve_commit(const int* tokens, const int* e_start, const int* e_len, const int* e_slot, const int* e_pos0,
                     int n_entries, int* prev, int* parity, cudaStream_t s) {
  if (n_entries <= 0) return 0;
  const ServeEntries e{e_start, e_len, e_slot, e_pos0};
  return static_cast<int>(launch_kernel(serve_commit_kernel, dim3((n_entries + 127) / 128), dim3(128), 0, s, tokens, e,
                                        n_entries, prev, parity));
}
}
