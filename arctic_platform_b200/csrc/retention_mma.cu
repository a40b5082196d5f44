// Retention over long entries on tensor cores, with fp32-class products.
//
// Same recurrence as retention_chunk_kernel (retention.cu), chunks of 32 tokens.  Every fp32 operand x (rotated q and k,
// decayed scores, the carried state) is split into two bf16 numbers, x = hi + lo, and a product takes the three
// significant cross terms as m16n8k16 MMAs with fp32 accumulation, which keeps 16 bits of every factor; v is bf16 to
// begin with.  The state itself stays in fp32 registers (the accumulator fragments of the update product), its hi / lo
// copy in shared memory is only the operand of the next chunk's q S product.
//
// One CTA = (segment of an entry, head, 64-column slice of E), two CTAs per SM.  An entry is one segment when there are
// enough entries to fill the GPU.  Otherwise it is cut into several: a first launch (state_only) computes what each
// segment adds to the state, retention_carry_kernel chains them into the state before each segment, and the second
// launch runs all segments at once.
#include "common.cuh"
#include "host_utils.cuh"
#include "retention.cuh"

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

__device__ __forceinline__ void rm_cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void rm_ldsm4(const __nv_bfloat16* a, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(a)));
}
__device__ __forceinline__ void rm_ldsm4_t(const __nv_bfloat16* a, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(a)));
}
__device__ __forceinline__ void rm_ldsm2(const __nv_bfloat16* a, uint32_t (&r)[2]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0, %1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(smem_u32(a)));
}
__device__ __forceinline__ void rm_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// x = hi + lo with both parts bf16; two neighbouring elements packed per word
__device__ __forceinline__ void rm_split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  const float2 h = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&hi));
  lo = pack_bf16x2(x - h.x, y - h.y);
}

__host__ __device__ inline int rm_smem_bytes(int D) {
  const int dp = (D + 15) / 16 * 16, ds = dp + 8;
  return 2 * (4 * kRmC * ds + 3 * kRmC * kRmVS + 2 * kRmC * kRmAS + 2 * dp * kRmVS + kRmC * (2 * dp + kRmBE)) + 256;
}

__global__ void __launch_bounds__(kRmThreads, 2)
retention_mma_kernel(const RetentionParams p, const RetentionSegments sg, int state_only) {
  pdl_entry();
  extern __shared__ __align__(128) uint8_t rm_smem[];
  const int* w = sg.seg + blockIdx.x * 6;
  const int en = w[0], t_begin = w[1], n_tok = w[2], carry_in = w[3], carry_out = w[4], is_last = w[5];
  if (state_only && carry_out < 0) return;
  const int h = blockIdx.y, e0 = blockIdx.z * kRmBE;
  const int D = p.D, E = p.E, dp = (D + 15) & ~15, ds = dp + 8, d16 = dp >> 4;
  const int be = min(kRmBE, E - e0);
  const int start = p.e.start[en] + t_begin, pos0 = p.e.pos0[en] + t_begin, slot = p.e.slot[en];
  __nv_bfloat16* Qh = reinterpret_cast<__nv_bfloat16*>(rm_smem);
  __nv_bfloat16* Ql = Qh + kRmC * ds;
  __nv_bfloat16* Kh = Ql + kRmC * ds;
  __nv_bfloat16* Kl = Kh + kRmC * ds;
  __nv_bfloat16* V = Kl + kRmC * ds;             // [32][72] values
  __nv_bfloat16* Wh = V + kRmC * kRmVS;          // values times decay^(n - 1 - j), hi / lo
  __nv_bfloat16* Wl = Wh + kRmC * kRmVS;
  __nv_bfloat16* Ah = Wl + kRmC * kRmVS;         // [32][40] decayed scores
  __nv_bfloat16* Al = Ah + kRmC * kRmAS;
  __nv_bfloat16* Sh = Al + kRmC * kRmAS;         // [dp][72] carried state
  __nv_bfloat16* Sl = Sh + dp * kRmVS;
  __nv_bfloat16* raw = Sl + dp * kRmVS;          // [32][dp] q, [32][dp] k, [32][64] v as they come from memory
  float* pw = reinterpret_cast<float*>(raw + kRmC * (2 * dp + kRmBE));   // decay powers 0 .. 32
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int quad_row = lane >> 2, quad_col = (lane & 3) * 2;
  const int mat = lane >> 3, rowin = lane & 7;
  const __nv_bfloat16* pb = static_cast<const __nv_bfloat16*>(p.p);

  if (threadIdx.x <= kRmC) pw[threadIdx.x] = decay_pow(p.log2_decay[h], threadIdx.x);

  auto fetch = [&](int t0) {
    const int n = min(kRmC, n_tok - t0), dc = D >> 3, vc = be >> 3;
    for (int i = threadIdx.x; i < n * (2 * dc + vc); i += kRmThreads) {
      const int r = i / (2 * dc + vc), c = i % (2 * dc + vc);
      const __nv_bfloat16* row = pb + static_cast<long long>(start + t0 + r) * p.ld;
      if (c < dc)
        rm_cp_async16(smem_u32(raw + r * dp + c * 8), row + p.q_col + h * D + c * 8);
      else if (c < 2 * dc)
        rm_cp_async16(smem_u32(raw + (kRmC + r) * dp + (c - dc) * 8), row + p.k_col + h * D + (c - dc) * 8);
      else
        rm_cp_async16(smem_u32(raw + 2 * kRmC * dp + r * kRmBE + (c - 2 * dc) * 8), row + p.v_col + h * E + e0 + (c - 2 * dc) * 8);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0);

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
          rm_split2(s[nt][2 * hh], s[nt][2 * hh + 1], hi, lo);
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

  for (int t0 = 0; t0 < n_tok; t0 += kRmC) {
    const int n = min(kRmC, n_tok - t0);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                               // raw rows have landed; everybody is done with the last chunk
    // ---- rotate, scale, split
    auto put = [&](__nv_bfloat16* hi_t, __nv_bfloat16* lo_t, int o, float x, float y) {
      uint32_t hi, lo;
      rm_split2(x, y, hi, lo);
      *reinterpret_cast<uint32_t*>(hi_t + o) = hi;
      *reinterpret_cast<uint32_t*>(lo_t + o) = lo;
    };
    const int half = p.rot_dims >> 1;
    int d_done = 0;                                // dimensions covered by the paired loop
    if ((half & 1) == 0) {                         // two neighbouring rotation pairs (d, d + half), (d + 1, d + 1 + half)
      d_done = p.rot_dims;
      const int q2 = half >> 1;
#pragma unroll 4
      for (int i = threadIdx.x; i < kRmC * q2; i += kRmThreads) {
        const int r = i / q2, d = (i - r * q2) * 2, o = r * ds + d;
        float2 qu = make_float2(0.f, 0.f), qv = qu, ku = qu, kv = qu, c = qu, sn = qu;
        if (r < n) {
          const long long tr = static_cast<long long>(pos0 + t0 + r) * half + d;
          c = *reinterpret_cast<const float2*>(p.cos_t + tr);
          sn = *reinterpret_cast<const float2*>(p.sin_t + tr);
          const __nv_bfloat16* rq = raw + r * dp + d;
          const __nv_bfloat16* rk = rq + kRmC * dp;
          qu = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(rq));
          qv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(rq + half));
          ku = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(rk));
          kv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(rk + half));
        }
        if (!state_only) {
          put(Qh, Ql, o, qu.x * c.x - qv.x * sn.x, qu.y * c.y - qv.y * sn.y);
          put(Qh, Ql, o + half, qv.x * c.x + qu.x * sn.x, qv.y * c.y + qu.y * sn.y);
        }
        put(Kh, Kl, o, (ku.x * c.x - kv.x * sn.x) * p.k_scale, (ku.y * c.y - kv.y * sn.y) * p.k_scale);
        put(Kh, Kl, o + half, (kv.x * c.x + ku.x * sn.x) * p.k_scale, (kv.y * c.y + ku.y * sn.y) * p.k_scale);
      }
    }
    const int pairs = (dp - d_done) >> 1;          // unrotated dimensions (and the padding), or odd rotations
    for (int i = threadIdx.x; i < kRmC * pairs; i += kRmThreads) {
      const int r = i / pairs, d = d_done + (i % pairs) * 2, o = r * ds + d;
      float2 qv = make_float2(0.f, 0.f), kv = qv;
      if (r < n && d < D) {
        const long long tr = static_cast<long long>(pos0 + t0 + r) * half;
        const float* c = p.cos_t + tr;
        const float* sn = p.sin_t + tr;
        const __nv_bfloat16* rq = raw + r * dp;
        const __nv_bfloat16* rk = raw + (kRmC + r) * dp;
        qv = make_float2(rotated(rq, d, p.rot_dims, c, sn), rotated(rq, d + 1, p.rot_dims, c, sn));
        kv = make_float2(rotated(rk, d, p.rot_dims, c, sn) * p.k_scale, rotated(rk, d + 1, p.rot_dims, c, sn) * p.k_scale);
      }
      if (!state_only) put(Qh, Ql, o, qv.x, qv.y);
      put(Kh, Kl, o, kv.x, kv.y);
    }
    for (int i = threadIdx.x; i < kRmC * (kRmBE / 2); i += kRmThreads) {
      const int r = i / (kRmBE / 2), c = (i % (kRmBE / 2)) * 2;
      uint32_t v = 0, wh = 0, wl = 0;
      if (r < n && c < be) {
        v = *reinterpret_cast<const uint32_t*>(raw + 2 * kRmC * dp + r * kRmBE + c);
        const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v));
        const float g = pw[n - 1 - r];
        rm_split2(f.x * g, f.y * g, wh, wl);
      }
      const int o = r * kRmVS + c;
      *reinterpret_cast<uint32_t*>(V + o) = v;
      *reinterpret_cast<uint32_t*>(Wh + o) = wh;
      *reinterpret_cast<uint32_t*>(Wl + o) = wl;
    }
    __syncthreads();
    if (t0 + kRmC < n_tok) fetch(t0 + kRmC);        // the raw rows are free again: overlap the next chunk's loads
    const int r0 = (warp & 1) * 16, c0 = (warp >> 1) * 16;     // this warp's tile of the output
    float o[2][4];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) o[nt][0] = o[nt][1] = o[nt][2] = o[nt][3] = 0.f;
    if (!state_only) {
      // ---- scores: 16 queries x 8 keys per warp
      const int k0 = (warp >> 1) * 8;
      float a[4] = {0.f, 0.f, 0.f, 0.f};
      const bool live = k0 <= r0 + 15;
      for (int ks = 0; ks < d16; ++ks) {
        uint32_t qh[4], ql[4];
        const int ao = (r0 + rowin + (mat & 1) * 8) * ds + ks * 16 + (mat >> 1) * 8;
        rm_ldsm4(Qh + ao, qh);
        rm_ldsm4(Ql + ao, ql);
        if (live) {
          uint32_t kh[2], kl[2];
          const int bo = (k0 + rowin) * ds + ks * 16 + (mat & 1) * 8;
          rm_ldsm2(Kh + bo, kh);
          rm_ldsm2(Kl + bo, kl);
          rm_mma(a, ql, kh[0], kh[1]);
          rm_mma(a, qh, kl[0], kl[1]);
          rm_mma(a, qh, kh[0], kh[1]);
        }
        if (have_state) {                          // q S of the carried state
          uint32_t sh[4], sl[4];
          const int so = (ks * 16 + rowin + 8 * (mat & 1)) * kRmVS + c0 + (mat >> 1) * 8;
          rm_ldsm4_t(Sh + so, sh);
          rm_ldsm4_t(Sl + so, sl);
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            rm_mma(o[nt], ql, sh[2 * nt], sh[2 * nt + 1]);
            rm_mma(o[nt], qh, sl[2 * nt], sl[2 * nt + 1]);
            rm_mma(o[nt], qh, sh[2 * nt], sh[2 * nt + 1]);
          }
        }
      }
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        const int i = r0 + quad_row + 8 * hh, j = k0 + quad_col;
        uint32_t hi, lo;
        rm_split2(j <= i ? a[2 * hh] * pw[i - j] : 0.f, j + 1 <= i ? a[2 * hh + 1] * pw[i - j - 1] : 0.f, hi, lo);
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
    __syncthreads();                               // scores visible; nobody reads the state operand any more
    if (!state_only) {
      for (int ks = 0; ks < (r0 + 16) / 16; ++ks) {
        uint32_t ah[4], al[4], v[4];
        const int ao = (r0 + rowin + (mat & 1) * 8) * kRmAS + ks * 16 + (mat >> 1) * 8;
        rm_ldsm4(Ah + ao, ah);
        rm_ldsm4(Al + ao, al);
        rm_ldsm4_t(V + (ks * 16 + rowin + 8 * (mat & 1)) * kRmVS + c0 + (mat >> 1) * 8, v);
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          rm_mma(o[nt], al, v[2 * nt], v[2 * nt + 1]);
          rm_mma(o[nt], ah, v[2 * nt], v[2 * nt + 1]);
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
        rm_ldsm4_t(Kh + ao, kh);
        rm_ldsm4_t(Kl + ao, kl);
#pragma unroll
        for (int n2 = 0; n2 < 4; ++n2) {
          uint32_t wh[4], wl[4];
          const int bo = (ks * 16 + rowin + 8 * (mat & 1)) * kRmVS + n2 * 16 + (mat >> 1) * 8;
          rm_ldsm4_t(Wh + bo, wh);
          rm_ldsm4_t(Wl + bo, wl);
#pragma unroll
          for (int k = 0; k < 2; ++k) {
            rm_mma(s[2 * n2 + k], kl, wh[2 * k], wh[2 * k + 1]);
            rm_mma(s[2 * n2 + k], kh, wl[2 * k], wl[2 * k + 1]);
            rm_mma(s[2 * n2 + k], kh, wh[2 * k], wh[2 * k + 1]);
          }
        }
      }
    }
    if (!state_only && t0 + kRmC < n_tok) store_state_operand();
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
// scratch for their states).
int apb_retention_mma(const void* p, long long ld, int q_col, int k_col, int v_col, const float* cos_t, const float* sin_t,
                      int rot_dims, const float* log2_decay, float k_scale, float* state, float* o, const int* e_start,
                      const int* e_len, const int* e_slot, const int* e_pos0, const int* seg, int n_seg, float* carry,
                      const int* chains, int n_chains, int H, int D, int E, cudaStream_t s) {
  if (n_seg <= 0) return 0;
  if (H <= 0 || D <= 0 || E <= 0 || (D % 8) || (E % 8) || D > kRmMaxD || (ld % 8) || (q_col % 8) || (k_col % 8) || (v_col % 8) ||
      (reinterpret_cast<uintptr_t>(p) & 15) || (rot_dims & 1) || rot_dims > D || rot_dims < 0 || !seg || !o ||
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
  const int smem = rm_smem_bytes(D);
  cudaError_t e = cudaFuncSetAttribute(retention_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return static_cast<int>(e);
  const dim3 grid(n_seg, H, (E + kRmBE - 1) / kRmBE);
  if (n_chains > 0) {
    e = launch_kernel(retention_mma_kernel, grid, dim3(kRmThreads), smem, s, a, sg, 1);
    if (e != cudaSuccess) return static_cast<int>(e);
    e = launch_kernel(retention_carry_kernel, dim3(n_chains, H, (D * E + 255) / 256), dim3(256), 0, s, a, sg, chains);
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  return static_cast<int>(launch_kernel(retention_mma_kernel, grid, dim3(kRmThreads), smem, s, a, sg, 0));
}
}
