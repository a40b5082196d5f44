// Retention over long entries on tensor cores, with fp32-class products.
//
// Same recurrence as retention_chunk_kernel (retention.cu), chunks of 32 tokens.  Every fp32 operand x (rotated q and k,
// decayed scores, the carried state) is split into two bf16 numbers, x = hi + lo, and a product takes the three
// significant cross terms as m16n8k16 MMAs with fp32 accumulation, which keeps 16 bits of every factor; v is bf16 to
// begin with.  The state itself stays in fp32 registers (the accumulator fragments of the update product), its hi / lo
// copy in shared memory is only the operand of the next chunk's q S product.
//
// q and k are rotated, scaled and split once per (row, head) by retention_split_kernel; the chunk kernel copies the
// halves to shared memory while the previous chunk is being computed.
//
// One CTA = (segment of an entry, head, 64-column slice of E), two CTAs per SM.  An entry is one segment when there are
// enough entries to fill the GPU.  Otherwise it is cut into several: a first launch (state_only) computes what each
// segment adds to the state, retention_carry_kernel chains them into the state before each segment, and the second
// launch runs all segments at once.
#include "common.cuh"
#include "host_utils.cuh"
#include "retention.cuh"
#include "warp_mma.cuh"

namespace apb {

constexpr int kRmThreads = 256;
constexpr int kRmC = 32;                  // tokens per chunk
constexpr int kRmBE = 64;                 // E columns per CTA
constexpr int kRmVS = kRmBE + 8;          // row strides (elements): odd multiples of 16 bytes
constexpr int kRmAS = kRmC + 8;
constexpr int kRmMaxD = 128;

struct RetentionSegments {
  const int* seg;         // [n][6]: entry, first token, tokens, scratch index of the state before it (-1: the slot's
                          // state or zero), scratch index for its own contribution (-1: none), 1 = last of its entry
  float* carry;           // [scratch states][H][D][E]
};

// qk [rows][H][4][dp]: hi and lo of the rotated q, hi and lo of the rotated and scaled k; dp = D rounded up to 16, the
// padding zero.  Rows of one-token entries are skipped.  One warp per (row, head).
__global__ void __launch_bounds__(256)
retention_split_kernel(const RetentionParams p, const int* __restrict__ row_entry, int rows, __nv_bfloat16* __restrict__ qk) {
  pdl_entry();
  const int lane = threadIdx.x & 31;
  const long long gw = (blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x) >> 5;
  if (gw >= static_cast<long long>(rows) * p.H) return;
  const int row = static_cast<int>(gw / p.H), h = static_cast<int>(gw % p.H);
  const int en = row_entry ? row_entry[row] : row;
  if (p.e.len[en] <= 1) return;
  const int D = p.D, dp = (D + 15) & ~15, half = p.rot_dims >> 1;
  const long long tr = static_cast<long long>(p.e.pos0[en] + row - p.e.start[en]) * half;
  const __nv_bfloat16* pr = static_cast<const __nv_bfloat16*>(p.p) + static_cast<long long>(row) * p.ld;
  const __nv_bfloat16* q = pr + p.q_col + h * D;
  const __nv_bfloat16* k = pr + p.k_col + h * D;
  __nv_bfloat16* out = qk + gw * 4 * dp;
  auto put = [&](int part, int d, float x, float y) {
    uint32_t hi, lo;
    wm_split2(x, y, hi, lo);
    *reinterpret_cast<uint32_t*>(out + part * dp + d) = hi;
    *reinterpret_cast<uint32_t*>(out + (part + 1) * dp + d) = lo;
  };
  int d_done = 0;                                  // dimensions covered by the paired loop
  if ((half & 1) == 0) {                           // two neighbouring rotation pairs (d, d + half), (d + 1, d + 1 + half)
    d_done = p.rot_dims;
    for (int d = lane * 2; d < half; d += 64) {
      const float2 c = *reinterpret_cast<const float2*>(p.cos_t + tr + d);
      const float2 sn = *reinterpret_cast<const float2*>(p.sin_t + tr + d);
      const float2 qu = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(q + d));
      const float2 qv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(q + d + half));
      const float2 ku = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(k + d));
      const float2 kv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(k + d + half));
      put(0, d, qu.x * c.x - qv.x * sn.x, qu.y * c.y - qv.y * sn.y);
      put(0, d + half, qv.x * c.x + qu.x * sn.x, qv.y * c.y + qu.y * sn.y);
      put(2, d, (ku.x * c.x - kv.x * sn.x) * p.k_scale, (ku.y * c.y - kv.y * sn.y) * p.k_scale);
      put(2, d + half, (kv.x * c.x + ku.x * sn.x) * p.k_scale, (kv.y * c.y + ku.y * sn.y) * p.k_scale);
    }
  }
  for (int d = d_done + lane * 2; d < dp; d += 64) {     // unrotated dimensions and padding, or odd rotations
    float2 a = make_float2(0.f, 0.f), b = a;
    if (d < D) {
      a = make_float2(rotated(q, d, p.rot_dims, p.cos_t + tr, p.sin_t + tr), rotated(q, d + 1, p.rot_dims, p.cos_t + tr, p.sin_t + tr));
      b = make_float2(rotated(k, d, p.rot_dims, p.cos_t + tr, p.sin_t + tr) * p.k_scale,
                      rotated(k, d + 1, p.rot_dims, p.cos_t + tr, p.sin_t + tr) * p.k_scale);
    }
    put(0, d, a.x, a.y);
    put(2, d, b.x, b.y);
  }
}

__host__ __device__ inline int rm_smem_bytes(int D) {
  const int dp = (D + 15) / 16 * 16, ds = dp + 8;
  return 2 * (6 * kRmC * ds + 4 * kRmC * kRmVS + 2 * kRmC * kRmAS + 2 * dp * kRmVS) + 256;
}

// DP: D rounded up to 16 when known at compile time, else 0.
template <int DP>
__global__ void __launch_bounds__(kRmThreads, 2)
retention_mma_kernel(const RetentionParams p, const RetentionSegments sg, const __nv_bfloat16* __restrict__ qk,
                     int state_only) {
  pdl_entry();
  extern __shared__ __align__(128) uint8_t rm_smem[];
  const int* w = sg.seg + blockIdx.x * 6;
  const int en = w[0], t_begin = w[1], n_tok = w[2], carry_in = w[3], carry_out = w[4], is_last = w[5];
  if (state_only && carry_out < 0) return;
  const int h = blockIdx.y, e0 = blockIdx.z * kRmBE;
  const int D = p.D, E = p.E, dp = DP ? DP : (D + 15) & ~15, ds = dp + 8, d16 = dp >> 4;
  const int be = min(kRmBE, E - e0);
  const int start = p.e.start[en] + t_begin, pos0 = p.e.pos0[en] + t_begin, slot = p.e.slot[en];
  __nv_bfloat16* Qh = reinterpret_cast<__nv_bfloat16*>(rm_smem);
  __nv_bfloat16* Ql = Qh + kRmC * ds;
  __nv_bfloat16* K2 = Ql + kRmC * ds;            // two buffers of (hi, lo) [32][ds]
  __nv_bfloat16* V2 = K2 + 4 * kRmC * ds;        // two buffers of values [32][72]
  __nv_bfloat16* Wh = V2 + 2 * kRmC * kRmVS;     // values times decay^(n - 1 - j), hi / lo
  __nv_bfloat16* Wl = Wh + kRmC * kRmVS;
  __nv_bfloat16* Ah = Wl + kRmC * kRmVS;         // [32][40] decayed scores
  __nv_bfloat16* Al = Ah + kRmC * kRmAS;
  __nv_bfloat16* Sh = Al + kRmC * kRmAS;         // [dp][72] carried state
  __nv_bfloat16* Sl = Sh + dp * kRmVS;
  float* pw = reinterpret_cast<float*>(Sl + dp * kRmVS);     // decay powers 0 .. 32
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int quad_row = lane >> 2, quad_col = (lane & 3) * 2;
  const int mat = lane >> 3, rowin = lane & 7;
  const __nv_bfloat16* pb = static_cast<const __nv_bfloat16*>(p.p);

  if (threadIdx.x <= kRmC) pw[threadIdx.x] = decay_pow(p.log2_decay[h], threadIdx.x);

  // rows beyond the segment are filled with zeros
  const int pc = dp >> 3;                        // 16-byte chunks of one part
  auto fetch_part = [&](int t0, int part, __nv_bfloat16* dst) {         // hi and lo of q (part 0) or k (part 2)
#pragma unroll
    for (int i = threadIdx.x; i < kRmC * 2 * pc; i += kRmThreads) {
      const int r = i / (2 * pc), c = i % (2 * pc), ok = t0 + r < n_tok;
      const __nv_bfloat16* src = qk + ((static_cast<long long>(start + (ok ? t0 + r : 0)) * p.H + h) * 4 + part) * dp + c * 8;
      wm_cp_async16(smem_u32(dst + (c / pc) * (kRmC * ds) + r * ds + (c % pc) * 8), src, ok ? 16 : 0);
    }
  };
  auto fetch_kv = [&](int t0, int buf) {
    fetch_part(t0, 2, K2 + buf * 2 * kRmC * ds);
    const int r = threadIdx.x >> 3, c = threadIdx.x & 7, ok = t0 + r < n_tok && c * 8 < be;
    const __nv_bfloat16* src = pb + static_cast<long long>(start + (ok ? t0 + r : 0)) * p.ld + p.v_col + h * E + e0 + (ok ? c * 8 : 0);
    wm_cp_async16(smem_u32(V2 + buf * kRmC * kRmVS + r * kRmVS + c * 8), src, ok ? 16 : 0);
  };
  static_assert(kRmThreads == kRmC * kRmBE / 8, "one 16-byte chunk of the values per thread");
  if (!state_only) fetch_part(0, 0, Qh);
  fetch_kv(0, 0);
  asm volatile("cp.async.commit_group;" ::: "memory");

  // the warp's 16 state rows, fp32: accumulator fragments over eight 8-column tiles
  float s[8][4];
  const float* s_in = nullptr;
  if (!state_only) {
    if (carry_in >= 0)
      s_in = sg.carry + (static_cast<long long>(carry_in) * p.H + h) * D * E;
    else if (pos0 > 0)
      s_in = p.state + (static_cast<long long>(slot) * p.H + h) * D * E;
  }
  const int sr = warp * 16 + quad_row;
  auto store_state_operand = [&]() {
    if (warp < d16) {
#pragma unroll
      for (int nt = 0; nt < 8; ++nt)
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
          uint32_t hi, lo;
          wm_split2(s[nt][2 * hh], s[nt][2 * hh + 1], hi, lo);
          const int o = (sr + 8 * hh) * kRmVS + nt * 8 + quad_col;
          *reinterpret_cast<uint32_t*>(Sh + o) = hi;
          *reinterpret_cast<uint32_t*>(Sl + o) = lo;
        }
    }
  };
#pragma unroll
  for (int nt = 0; nt < 8; ++nt)
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      const int d = sr + 8 * hh, c = nt * 8 + quad_col;
      float2 v = make_float2(0.f, 0.f);
      if (s_in && d < D && c < be) v = *reinterpret_cast<const float2*>(s_in + static_cast<long long>(d) * E + e0 + c);
      s[nt][2 * hh] = v.x;
      s[nt][2 * hh + 1] = v.y;
    }
  bool have_state = s_in != nullptr;
  if (have_state) store_state_operand();

  for (int t0 = 0, buf = 0; t0 < n_tok; t0 += kRmC, buf ^= 1) {
    const int n = min(kRmC, n_tok - t0);
    const bool more = t0 + kRmC < n_tok;
    const __nv_bfloat16* Kh = K2 + buf * 2 * kRmC * ds;
    const __nv_bfloat16* Kl = Kh + kRmC * ds;
    const __nv_bfloat16* V = V2 + buf * kRmC * kRmVS;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                               // this chunk has landed; everybody is done with the last one
    if (more) fetch_kv(t0 + kRmC, buf ^ 1);
    for (int i = threadIdx.x; i < kRmC * (kRmBE / 2); i += kRmThreads) {
      const int r = i / (kRmBE / 2), o = r * kRmVS + (i % (kRmBE / 2)) * 2;
      const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(V + o));
      const float g = r < n ? pw[n - 1 - r] : 0.f;
      uint32_t wh, wl;
      wm_split2(f.x * g, f.y * g, wh, wl);
      *reinterpret_cast<uint32_t*>(Wh + o) = wh;
      *reinterpret_cast<uint32_t*>(Wl + o) = wl;
    }
    const int r0 = (warp & 1) * 16, c0 = (warp >> 1) * 16;     // this warp's tile of the output
    float o[2][4];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) o[nt][0] = o[nt][1] = o[nt][2] = o[nt][3] = 0.f;
    if (!state_only) {
      // ---- scores: 16 queries x 8 keys per warp
      const int k0 = (warp >> 1) * 8;
      float a[4] = {0.f, 0.f, 0.f, 0.f};
      const bool live = k0 <= r0 + 15;
#pragma unroll 4
      for (int ks = 0; ks < d16; ++ks) {
        uint32_t qh[4], ql[4];
        const int ao = (r0 + rowin + (mat & 1) * 8) * ds + ks * 16 + (mat >> 1) * 8;
        wm_ldsm4(Qh + ao, qh);
        wm_ldsm4(Ql + ao, ql);
        if (live) {
          uint32_t kh[2], kl[2];
          const int bo = (k0 + rowin) * ds + ks * 16 + (mat & 1) * 8;
          wm_ldsm2(Kh + bo, kh);
          wm_ldsm2(Kl + bo, kl);
          wm_mma(a, ql, kh[0], kh[1]);
          wm_mma(a, qh, kl[0], kl[1]);
          wm_mma(a, qh, kh[0], kh[1]);
        }
        if (have_state) {                          // q S of the carried state
          uint32_t sh[4], sl[4];
          const int so = (ks * 16 + rowin + 8 * (mat & 1)) * kRmVS + c0 + (mat >> 1) * 8;
          wm_ldsm4_t(Sh + so, sh);
          wm_ldsm4_t(Sl + so, sl);
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            wm_mma(o[nt], ql, sh[2 * nt], sh[2 * nt + 1]);
            wm_mma(o[nt], qh, sl[2 * nt], sl[2 * nt + 1]);
            wm_mma(o[nt], qh, sh[2 * nt], sh[2 * nt + 1]);
          }
        }
      }
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        const int i = r0 + quad_row + 8 * hh, j = k0 + quad_col;
        uint32_t hi, lo;
        wm_split2(j <= i ? a[2 * hh] * pw[i - j] : 0.f, j + 1 <= i ? a[2 * hh + 1] * pw[i - j - 1] : 0.f, hi, lo);
        *reinterpret_cast<uint32_t*>(Ah + i * kRmAS + j) = hi;
        *reinterpret_cast<uint32_t*>(Al + i * kRmAS + j) = lo;
        const float g = pw[i + 1];
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          o[nt][2 * hh] *= g;
          o[nt][2 * hh + 1] *= g;
        }
      }
    }
    __syncthreads();                               // scores and W visible; nobody reads q or the state operand any more
    if (more && !state_only) fetch_part(t0 + kRmC, 0, Qh);
    asm volatile("cp.async.commit_group;" ::: "memory");
    if (!state_only) {
      for (int ks = 0; ks < (r0 + 16) / 16; ++ks) {
        uint32_t ah[4], al[4], v[4];
        const int ao = (r0 + rowin + (mat & 1) * 8) * kRmAS + ks * 16 + (mat >> 1) * 8;
        wm_ldsm4(Ah + ao, ah);
        wm_ldsm4(Al + ao, al);
        wm_ldsm4_t(V + (ks * 16 + rowin + 8 * (mat & 1)) * kRmVS + c0 + (mat >> 1) * 8, v);
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          wm_mma(o[nt], al, v[2 * nt], v[2 * nt + 1]);
          wm_mma(o[nt], ah, v[2 * nt], v[2 * nt + 1]);
        }
      }
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        const int i = r0 + quad_row + 8 * hh;
        if (i < n) {
          float* dst = p.o + (static_cast<long long>(start + t0 + i) * p.H + h) * E + e0;
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            const int c = c0 + nt * 8 + quad_col;
            if (c < be) *reinterpret_cast<float2*>(dst + c) = make_float2(o[nt][2 * hh], o[nt][2 * hh + 1]);
          }
        }
      }
    }
    // ---- S = decay^n S + sum_j k_j (decay^(n - 1 - j) v_j)^T
    if (warp < d16) {
      const float dn = pw[n];
#pragma unroll
      for (int nt = 0; nt < 8; ++nt)
#pragma unroll
        for (int i = 0; i < 4; ++i) s[nt][i] *= dn;
#pragma unroll
      for (int ks = 0; ks < kRmC / 16; ++ks) {
        uint32_t kh[4], kl[4];
        const int ao = (ks * 16 + rowin + (mat >> 1) * 8) * ds + warp * 16 + (mat & 1) * 8;
        wm_ldsm4_t(Kh + ao, kh);
        wm_ldsm4_t(Kl + ao, kl);
#pragma unroll
        for (int n2 = 0; n2 < 4; ++n2) {
          uint32_t wh[4], wl[4];
          const int bo = (ks * 16 + rowin + 8 * (mat & 1)) * kRmVS + n2 * 16 + (mat >> 1) * 8;
          wm_ldsm4_t(Wh + bo, wh);
          wm_ldsm4_t(Wl + bo, wl);
#pragma unroll
          for (int k = 0; k < 2; ++k) {
            wm_mma(s[2 * n2 + k], kl, wh[2 * k], wh[2 * k + 1]);
            wm_mma(s[2 * n2 + k], kh, wl[2 * k], wl[2 * k + 1]);
            wm_mma(s[2 * n2 + k], kh, wh[2 * k], wh[2 * k + 1]);
          }
        }
      }
    }
    if (!state_only && more) store_state_operand();
    have_state = true;
  }
  // ---- the state after the segment
  float* s_out = state_only ? sg.carry + (static_cast<long long>(carry_out) * p.H + h) * D * E
                            : (is_last ? p.state + (static_cast<long long>(slot) * p.H + h) * D * E : nullptr);
  if (s_out && warp < d16) {
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        const int d = sr + 8 * hh, c = nt * 8 + quad_col;
        if (d < D && c < be)
          *reinterpret_cast<float2*>(s_out + static_cast<long long>(d) * E + e0 + c) = make_float2(s[nt][2 * hh], s[nt][2 * hh + 1]);
      }
  }
}

// Chains the contributions of an entry's segments: scratch[base] becomes the state before the entry, scratch[base + i]
// the state before its i-th segment.  chains [n][4]: entry, base, segments, index of its first segment.
__global__ void __launch_bounds__(256)
retention_carry_kernel(const RetentionParams p, const RetentionSegments sg, const int* __restrict__ chains) {
  pdl_entry();
  const int* c = chains + blockIdx.x * 4;
  const int en = c[0], base = c[1], n_seg = c[2], first = c[3], h = blockIdx.y;
  const int size = p.D * p.E;
  const int i = blockIdx.z * 256 + threadIdx.x;
  if (i >= size) return;
  const long long stride = static_cast<long long>(p.H) * size;
  float* x = sg.carry + static_cast<long long>(base) * stride + static_cast<long long>(h) * size + i;
  float s = p.e.pos0[en] > 0 ? p.state[static_cast<long long>(p.e.slot[en]) * stride + static_cast<long long>(h) * size + i] : 0.f;
  x[0] = s;
  for (int k = 0; k + 1 < n_seg; ++k) {
    s = s * decay_pow(p.log2_decay[h], sg.seg[(first + k) * 6 + 2]) + x[(k + 1) * stride];
    x[(k + 1) * stride] = s;
  }
}

}  // namespace apb

extern "C" {
using namespace apb;

// bf16; D a multiple of 8 up to 128, E a multiple of 8; every column offset and ld a multiple of 8.  Writes o [rows, H, E]
// (fp32) for the segments' rows and the entries' states.  n_chains > 0: some entries have several segments (carry is
// scratch for their states).  qk: bf16 scratch [rows, H, 4, D rounded up to 16].
int apb_retention_mma(const void* p, long long ld, int q_col, int k_col, int v_col, const float* cos_t, const float* sin_t,
                      int rot_dims, const float* log2_decay, float k_scale, float* state, float* o, const int* e_start,
                      const int* e_len, const int* e_slot, const int* e_pos0, const int* seg, int n_seg, float* carry,
                      const int* chains, int n_chains, const int* row_entry, void* qk, int rows, int H, int D, int E,
                      cudaStream_t s) {
  if (n_seg <= 0) return 0;
  if (H <= 0 || D <= 0 || E <= 0 || (D % 8) || (E % 8) || D > kRmMaxD || (ld % 8) || (q_col % 8) || (k_col % 8) || (v_col % 8) ||
      (reinterpret_cast<uintptr_t>(p) & 15) || (rot_dims & 1) || rot_dims > D || rot_dims < 0 || !seg || !o || !qk ||
      (n_chains > 0 && (!carry || !chains)))
    return kBadArgument;
  RetentionParams a{};
  a.e = ServeEntries{e_start, e_len, e_slot, e_pos0};
  a.p = p;
  a.ld = ld;
  a.q_col = q_col;
  a.k_col = k_col;
  a.v_col = v_col;
  a.cos_t = cos_t;
  a.sin_t = sin_t;
  a.rot_dims = rot_dims;
  a.log2_decay = log2_decay;
  a.k_scale = k_scale;
  a.state = state;
  a.o = o;
  a.H = H;
  a.D = D;
  a.E = E;
  const RetentionSegments sg{seg, carry};
  const int smem = rm_smem_bytes(D), dp = (D + 15) / 16 * 16;
  const dim3 grid(n_seg, H, (E + kRmBE - 1) / kRmBE);
  const int sgrid = static_cast<int>((static_cast<long long>(rows) * H * 32 + 255) / 256);
  __nv_bfloat16* qkp = static_cast<__nv_bfloat16*>(qk);
  cudaError_t e = launch_kernel(retention_split_kernel, dim3(sgrid), dim3(256), 0, s, a, row_entry, rows, qkp);
  if (e != cudaSuccess) return static_cast<int>(e);
  auto run = [&](auto fn) -> cudaError_t {
    cudaError_t r = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (r != cudaSuccess) return r;
    if (n_chains > 0) {
      r = launch_kernel(fn, grid, dim3(kRmThreads), smem, s, a, sg, qkp, 1);
      if (r != cudaSuccess) return r;
      r = launch_kernel(retention_carry_kernel, dim3(n_chains, H, (D * E + 255) / 256), dim3(256), 0, s, a, sg, chains);
      if (r != cudaSuccess) return r;
    }
    return launch_kernel(fn, grid, dim3(kRmThreads), smem, s, a, sg, qkp, 0);
  };
  return static_cast<int>(dp == 128 ? run(retention_mma_kernel<128>) : dp == 64 ? run(retention_mma_kernel<64>) : run(retention_mma_kernel<0>));
}
}
