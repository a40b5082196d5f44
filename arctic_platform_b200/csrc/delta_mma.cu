// Gated delta rule (see recurrent.cuh) over long entries on tensor cores, with fp32-class products.
//
// Chunks of 32 tokens.  With G_i the running sum of the log decays inside the chunk, k^ and q^ the unit vectors and S the state
// before it, the written values solve a triangular system, whose inverse T does not depend on S:
//     u = T (diag(beta) V - diag(beta e^G) K^ S),         T^-1 = I + [beta_i e^(G_i - G_j) (k^_i . k^_j)]_{j < i}
//     o_i = e^(G_i) S^T q^_i + sum_{j <= i} A_ij u_j,     A_ij = e^(G_i - G_j) (q^_i . k^_j)
//     S <- e^(G_n) S + sum_j k^_j (e^(G_n - G_j) u_j)^T
// delta_chunk_kernel computes T, A and the scalars of all chunks at once; delta_mma_kernel walks the chunks with the state.  The
// operands q, k, v are the bf16 convolved columns; the norms of q and k are fp32 scalars applied to rows of the results, and every
// fp32 operand is split into two bf16 parts, hi + lo (the significant cross products).  One CTA = (entry, head, 64 columns of E).
#include "common.cuh"
#include "host_utils.cuh"
#include "recurrent.cuh"
#include "warp_mma.cuh"

namespace apb {

constexpr int kDlThreads = 256;
constexpr int kDlPrep = 128;
constexpr int kDlC = 32;
constexpr int kDlBE = 64;
constexpr int kDlVS = kDlBE + 8;
constexpr int kDlAS = kDlC + 8;
constexpr int kDlMaxD = 128;
constexpr int kDlSquare = kDlC * kDlC;
// scalars of a chunk: [0] beta, [1] beta e^G / |k|, [2] e^G D^-1/2 / |q|, [3] e^(G_n - G) / |k|, [4][0] e^(G_n)
constexpr int kDlScalars = 4 * kDlC + 4;

struct DeltaChunks {
  const int* tiles;          // [n][2] entry, first row of every chunk
  const int* heads;          // [m][2] entry, its first chunk
  __nv_bfloat16* square;     // [n][H][4][32][32]: T hi, T lo, A hi, A lo
  float* scalars;            // [n][H][kDlScalars]
};

__global__ void __launch_bounds__(kDlPrep)
delta_chunk_kernel(const RecurrentParams p, const DeltaChunks dc) {
  pdl_entry();
  extern __shared__ __align__(128) uint8_t dl_smem[];
  __shared__ __align__(16) float s_mat[kDlC][kDlC + 4];
  __shared__ float s_l[kDlC], s_beta[kDlC], s_k[kDlC], s_q[kDlC];
  const int tile = blockIdx.x, h = blockIdx.y, en = dc.tiles[2 * tile], t0 = dc.tiles[2 * tile + 1];
  const int n = min(kDlC, p.e.len[en] - t0);
  const int D = p.D, np = (D + 15) & ~15, ns = np + 8, n16 = np >> 4, kh = h / (p.H / p.KH), pc = np >> 3;
  const long long row0 = p.e.start[en] + t0;
  __nv_bfloat16* Q = reinterpret_cast<__nv_bfloat16*>(dl_smem);
  __nv_bfloat16* K = Q + kDlC * ns;
  const __nv_bfloat16* xb = static_cast<const __nv_bfloat16*>(p.xc);
  for (int i = threadIdx.x; i < 2 * kDlC * pc; i += kDlPrep) {
    const int m = i / (kDlC * pc), r = i / pc % kDlC, c = i % pc, ok = r < n && c * 8 < D;
    wm_cp_async16(smem_u32(Q + (m * kDlC + r) * ns + c * 8),
                  xb + (row0 + (ok ? r : 0)) * p.ldx + static_cast<long long>(m * p.KH + kh) * D + (ok ? c * 8 : 0), ok ? 16 : 0);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int quad_row = lane >> 2, quad_col = (lane & 3) * 2, mat = lane >> 3, rowin = lane & 7;
  if (warp == 3) {
    float2 g = make_float2(0.f, 0.f);
    if (lane < n) g = delta_gates<__nv_bfloat16>(p, row0 + lane, h);
    float l = fmaxf(g.x * 1.4426950408889634f, -kMaxLogDecay);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, l, o);
      if (lane >= o) l += v;
    }
    s_l[lane] = l;
    s_beta[lane] = g.y;
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  // ---- norms: a warp takes 8 rows of q and of k, four lanes per row
  {
    const int r = warp * 8 + (lane >> 2);
    float qq = 0.f, kk = 0.f;
    for (int d = (lane & 3) * 2; d < np; d += 8) {
      const float2 a = wm_pair(Q + r * ns + d), b = wm_pair(K + r * ns + d);
      qq += a.x * a.x + a.y * a.y;
      kk += b.x * b.x + b.y * b.y;
    }
#pragma unroll
    for (int o = 1; o < 4; o <<= 1) {
      qq += __shfl_xor_sync(0xffffffffu, qq, o);
      kk += __shfl_xor_sync(0xffffffffu, kk, o);
    }
    if ((lane & 3) == 0) {
      s_q[r] = 1.f / (sqrtf(qq + 1e-6f) * sqrtf(static_cast<float>(D)));
      s_k[r] = 1.f / sqrtf(kk + 1e-6f);
    }
  }
  const int r0 = (warp & 1) * 16, c0 = (warp >> 1) * 16;
  float kk[2][4] = {}, qk[2][4] = {};
  if (c0 <= r0)
    for (int ks = 0; ks < n16; ++ks) {
      uint32_t a[4], q[4], b[4];
      const int ro = (r0 + rowin + (mat & 1) * 8) * ns + ks * 16 + (mat >> 1) * 8;
      wm_ldsm4(K + ro, a);
      wm_ldsm4(Q + ro, q);
      wm_ldsm4(K + (c0 + rowin + (mat >> 1) * 8) * ns + ks * 16 + (mat & 1) * 8, b);
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        wm_mma(kk[nt], a, b[2 * nt], b[2 * nt + 1]);
        wm_mma(qk[nt], q, b[2 * nt], b[2 * nt + 1]);
      }
    }
  __syncthreads();
  __nv_bfloat16* out = dc.square + (static_cast<long long>(tile) * p.H + h) * 4 * kDlSquare;
#pragma unroll
  for (int nt = 0; nt < 2; ++nt)
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      const int i = r0 + quad_row + 8 * hh, j = c0 + nt * 8 + quad_col;
      float a[2];
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const float f = j + x <= i ? wm_ex2(s_l[i] - s_l[j + x]) * s_k[j + x] : 0.f;
        a[x] = qk[nt][2 * hh + x] * f * s_q[i];
        s_mat[i][j + x] = j + x < i ? kk[nt][2 * hh + x] * f * s_k[i] * s_beta[i] : 0.f;
      }
      wm_store_split2(out + 2 * kDlSquare + i * kDlC + j, out + 3 * kDlSquare + i * kDlC + j, a[0], a[1]);
    }
  __syncthreads();
  if (warp == 0) {                               // forward substitution, one column of T per lane
    float t[kDlC];
#pragma unroll
    for (int i = 0; i < kDlC; ++i) {
      float x = i == lane ? 1.f : 0.f;
#pragma unroll
      for (int j = 0; j < i; ++j) x -= s_mat[i][j] * t[j];
      t[i] = x;
      const __nv_bfloat16 hi = __float2bfloat16(x);
      out[i * kDlC + lane] = hi;
      out[kDlSquare + i * kDlC + lane] = __float2bfloat16(x - __bfloat162float(hi));
    }
  } else if (warp == 1) {
    float* sc = dc.scalars + (static_cast<long long>(tile) * p.H + h) * kDlScalars;
    const float l = s_l[lane], end = s_l[kDlC - 1], e = wm_ex2(l);
    sc[lane] = s_beta[lane];
    sc[kDlC + lane] = s_beta[lane] * e * s_k[lane];
    sc[2 * kDlC + lane] = e * s_q[lane];
    sc[3 * kDlC + lane] = lane < n ? wm_ex2(end - l) * s_k[lane] : 0.f;
    if (lane == 0) sc[4 * kDlC] = wm_ex2(end);
  }
}

__host__ __device__ inline int delta_smem_bytes(int D) {
  const int np = (D + 15) / 16 * 16, ns = np + 8;
  return 2 * (4 * kDlC * ns + 2 * kDlC * kDlVS + 8 * kDlC * kDlAS + 6 * kDlC * kDlVS + 2 * np * kDlVS) + 2 * kDlScalars * 4;
}

template <int NP>
__global__ void __launch_bounds__(kDlThreads)
delta_mma_kernel(const RecurrentParams p, const DeltaChunks dc) {
  pdl_entry();
  extern __shared__ __align__(128) uint8_t dl_smem[];
  const int en = dc.heads[2 * blockIdx.x], tile0 = dc.heads[2 * blockIdx.x + 1];
  const int h = blockIdx.y, e0 = blockIdx.z * kDlBE, kh = h / (p.H / p.KH);
  const int D = p.D, E = p.E, np = NP ? NP : (D + 15) & ~15, ns = np + 8, n16 = np >> 4, pc = np >> 3;
  const int be = min(kDlBE, E - e0), len = p.e.len[en], pos0 = p.e.pos0[en], slot = p.e.slot[en];
  const long long start = p.e.start[en];
  __nv_bfloat16* KQ2 = reinterpret_cast<__nv_bfloat16*>(dl_smem);    // two buffers [64][ns]: k, then q
  __nv_bfloat16* V2 = KQ2 + 4 * kDlC * ns;                           // two buffers [32][72]
  __nv_bfloat16* X2 = V2 + 2 * kDlC * kDlVS;                         // two buffers [4][32][40]: T hi, T lo, A hi, A lo
  __nv_bfloat16* Rh = X2 + 8 * kDlC * kDlAS;                         // [32][72] each, hi / lo: right-hand sides,
  __nv_bfloat16* Rl = Rh + kDlC * kDlVS;
  __nv_bfloat16* Uh = Rl + kDlC * kDlVS;                             // u,
  __nv_bfloat16* Ul = Uh + kDlC * kDlVS;
  __nv_bfloat16* Wh = Ul + kDlC * kDlVS;                             // u times its weight in the state after the chunk
  __nv_bfloat16* Wl = Wh + kDlC * kDlVS;
  __nv_bfloat16* Sh = Wl + kDlC * kDlVS;                             // [np][72] state before the chunk
  __nv_bfloat16* Sl = Sh + np * kDlVS;
  float* sc2 = reinterpret_cast<float*>(Sl + np * kDlVS);            // two buffers of scalars
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int quad_row = lane >> 2, quad_col = (lane & 3) * 2, mat = lane >> 3, rowin = lane & 7;
  const __nv_bfloat16* xb = static_cast<const __nv_bfloat16*>(p.xc);

  auto fetch = [&](int t0, int buf) {
#pragma unroll
    for (int i = threadIdx.x; i < 2 * kDlC * pc; i += kDlThreads) {
      const int m = i / (kDlC * pc), r = i / pc % kDlC, c = i % pc, ok = t0 + r < len && c * 8 < D;      // m 0: k, 1: q
      wm_cp_async16(smem_u32(KQ2 + ((buf * 2 + m) * kDlC + r) * ns + c * 8),
                    xb + (start + (ok ? t0 + r : 0)) * p.ldx + static_cast<long long>((1 - m) * p.KH + kh) * D + (ok ? c * 8 : 0), ok ? 16 : 0);
    }
    {
      const int r = threadIdx.x >> 3, c = threadIdx.x & 7, ok = t0 + r < len && c * 8 < be;
      wm_cp_async16(smem_u32(V2 + (buf * kDlC + r) * kDlVS + c * 8),
                    xb + (start + (ok ? t0 + r : 0)) * p.ldx + 2LL * p.KH * D + static_cast<long long>(h) * E + e0 + (ok ? c * 8 : 0), ok ? 16 : 0);
    }
    const long long at = static_cast<long long>(tile0 + t0 / kDlC) * p.H + h;
    const __nv_bfloat16* sq = dc.square + at * 4 * kDlSquare;
#pragma unroll
    for (int i = threadIdx.x; i < 4 * kDlC * 4; i += kDlThreads)     // 16-byte pieces: matrix, row, quarter
      wm_cp_async16(smem_u32(X2 + ((buf * 4 + i / (kDlC * 4)) * kDlC + i / 4 % kDlC) * kDlAS + (i & 3) * 8), sq + i * 8, 16);
    if (threadIdx.x < kDlScalars / 4) wm_cp_async16(smem_u32(sc2 + buf * kDlScalars + threadIdx.x * 4), dc.scalars + at * kDlScalars + threadIdx.x * 4, 16);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  static_assert(kDlThreads == kDlC * kDlBE / 8 && kDlScalars % 4 == 0, "one 16-byte piece of v per thread");
  fetch(0, 0);
  const float* s_in = pos0 > 0 ? p.state + (static_cast<long long>(slot) * p.H + h) * D * E + e0 : nullptr;
  StateTile st;
  st.load(s_in, E, D, be);
  bool have_state = s_in != nullptr;
  if (have_state && warp < n16) st.split_to(Sh, Sl, kDlVS);

  for (int t0 = 0, buf = 0; t0 < len; t0 += kDlC, buf ^= 1) {
    const int n = min(kDlC, len - t0);
    const bool more = t0 + kDlC < len;
    const __nv_bfloat16* K = KQ2 + buf * 2 * kDlC * ns;
    const __nv_bfloat16* V = V2 + buf * kDlC * kDlVS;
    const __nv_bfloat16* X = X2 + buf * 4 * kDlC * kDlAS;
    const float* sc = sc2 + buf * kDlScalars;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                               // this chunk has landed, the state operand is there
    if (more) fetch(t0 + kDlC, buf ^ 1);
    // ---- [K; Q] S: warps 0, 1, 4, 5 the rows of k, the others those of q; 16 rows x 32 columns each
    const int rt = warp & 3, ch = (warp >> 2) * 32;
    float o[4][4];
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) o[nt][0] = o[nt][1] = o[nt][2] = o[nt][3] = 0.f;
    if (have_state) {
#pragma unroll 4
      for (int ks = 0; ks < n16; ++ks) {
        uint32_t a[4];
        wm_ldsm4(K + (rt * 16 + rowin + (mat & 1) * 8) * ns + ks * 16 + (mat >> 1) * 8, a);
#pragma unroll
        for (int n2 = 0; n2 < 2; ++n2) {
          uint32_t sh[4], sl[4];
          const int so = (ks * 16 + rowin + 8 * (mat & 1)) * kDlVS + ch + n2 * 16 + (mat >> 1) * 8;
          wm_ldsm4_t(Sh + so, sh);
          wm_ldsm4_t(Sl + so, sl);
#pragma unroll
          for (int q = 0; q < 2; ++q) {
            wm_mma(o[2 * n2 + q], a, sl[2 * q], sl[2 * q + 1]);
            wm_mma(o[2 * n2 + q], a, sh[2 * q], sh[2 * q + 1]);
          }
        }
      }
    }
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      const int i = (rt & 1) * 16 + quad_row + 8 * hh;
      if (rt < 2) {                                // right-hand sides
        const float beta = sc[i], f = sc[kDlC + i];
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
          const int x = i * kDlVS + ch + nt * 8 + quad_col;
          const float2 v = wm_pair(V + x);
          wm_store_split2(Rh + x, Rl + x, beta * v.x - f * o[nt][2 * hh], beta * v.y - f * o[nt][2 * hh + 1]);
        }
      } else {
        const float f = sc[2 * kDlC + i];
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
          o[nt][2 * hh] *= f;
          o[nt][2 * hh + 1] *= f;
        }
      }
    }
    __syncthreads();
    // ---- u = T R: 16 x 16 per warp
    {
      const int r0 = (warp & 1) * 16, c0 = (warp >> 1) * 16;
      float u[2][4];
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) u[nt][0] = u[nt][1] = u[nt][2] = u[nt][3] = 0.f;
      for (int ks = 0; ks < (r0 + 16) / 16; ++ks) {
        uint32_t th[4], tl[4], rh[4], rl[4];
        const int to = (r0 + rowin + (mat & 1) * 8) * kDlAS + ks * 16 + (mat >> 1) * 8;
        const int ro = (ks * 16 + rowin + 8 * (mat & 1)) * kDlVS + c0 + (mat >> 1) * 8;
        wm_ldsm4(X + to, th);
        wm_ldsm4(X + kDlC * kDlAS + to, tl);
        wm_ldsm4_t(Rh + ro, rh);
        wm_ldsm4_t(Rl + ro, rl);
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          wm_mma(u[nt], tl, rh[2 * nt], rh[2 * nt + 1]);
          wm_mma(u[nt], th, rl[2 * nt], rl[2 * nt + 1]);
          wm_mma(u[nt], th, rh[2 * nt], rh[2 * nt + 1]);
        }
      }
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        const int i = r0 + quad_row + 8 * hh;
        const float wt = sc[3 * kDlC + i];
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          const int x = i * kDlVS + c0 + nt * 8 + quad_col;
          wm_store_split2(Uh + x, Ul + x, u[nt][2 * hh], u[nt][2 * hh + 1]);
          wm_store_split2(Wh + x, Wl + x, u[nt][2 * hh] * wt, u[nt][2 * hh + 1] * wt);
        }
      }
    }
    __syncthreads();
    // ---- o += A u (the warps that hold rows of q)
    if (rt >= 2) {
      const int r0 = (rt - 2) * 16;
      for (int ks = 0; ks < (r0 + 16) / 16; ++ks) {
        uint32_t ah[4], al[4];
        const int ao = (2 * kDlC + r0 + rowin + (mat & 1) * 8) * kDlAS + ks * 16 + (mat >> 1) * 8;
        wm_ldsm4(X + ao, ah);
        wm_ldsm4(X + kDlC * kDlAS + ao, al);
#pragma unroll
        for (int n2 = 0; n2 < 2; ++n2) {
          uint32_t uh[4], ul[4];
          const int uo = (ks * 16 + rowin + 8 * (mat & 1)) * kDlVS + ch + n2 * 16 + (mat >> 1) * 8;
          wm_ldsm4_t(Uh + uo, uh);
          wm_ldsm4_t(Ul + uo, ul);
#pragma unroll
          for (int q = 0; q < 2; ++q) {
            wm_mma(o[2 * n2 + q], al, uh[2 * q], uh[2 * q + 1]);
            wm_mma(o[2 * n2 + q], ah, ul[2 * q], ul[2 * q + 1]);
            wm_mma(o[2 * n2 + q], ah, uh[2 * q], uh[2 * q + 1]);
          }
        }
      }
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        const int i = r0 + quad_row + 8 * hh;
        if (i < n) {
          float* dst = p.y + (start + t0 + i) * p.H * E + static_cast<long long>(h) * E + e0;
#pragma unroll
          for (int nt = 0; nt < 4; ++nt) {
            const int c = ch + nt * 8 + quad_col;
            if (c < be) *reinterpret_cast<float2*>(dst + c) = make_float2(o[nt][2 * hh], o[nt][2 * hh + 1]);
          }
        }
      }
    }
    // ---- S = e^(G_n) S + K^T W
    if (warp < n16) {
      const float dn = sc[4 * kDlC];
      st.scale(dn, dn);
#pragma unroll
      for (int ks = 0; ks < kDlC / 16; ++ks) {
        uint32_t k[4];
        wm_ldsm4_t(K + (ks * 16 + rowin + (mat >> 1) * 8) * ns + warp * 16 + (mat & 1) * 8, k);
#pragma unroll
        for (int n2 = 0; n2 < 4; ++n2) {
          uint32_t wh[4], wl[4];
          const int bo = (ks * 16 + rowin + 8 * (mat & 1)) * kDlVS + n2 * 16 + (mat >> 1) * 8;
          wm_ldsm4_t(Wh + bo, wh);
          wm_ldsm4_t(Wl + bo, wl);
#pragma unroll
          for (int q = 0; q < 2; ++q) {
            wm_mma(st.s[2 * n2 + q], k, wl[2 * q], wl[2 * q + 1]);
            wm_mma(st.s[2 * n2 + q], k, wh[2 * q], wh[2 * q + 1]);
          }
        }
      }
      if (more) st.split_to(Sh, Sl, kDlVS);
    }
    have_state = true;
  }
  if (warp < n16) st.store(p.state + (static_cast<long long>(slot) * p.H + h) * D * E + e0, E, D, be);
}

}  // namespace apb

extern "C" {
using namespace apb;

// bf16; D a multiple of 8 up to 128, E a multiple of 8; xc as apb_short_conv leaves it, ldx a multiple of 8.  tiles [n_tiles, 2]: the
// chunks of 32 rows of the entries longer than one token, in order; heads [n_heads, 2]: those entries and their first chunks.
// square, scalars: scratch (see DeltaChunks).  Writes y and the entries' states.
int apb_delta_mma(const RecurrentParams* params, const int* tiles, int n_tiles, const int* heads, int n_heads, void* square,
                  float* scalars, cudaStream_t s) {
  if (n_tiles <= 0 || n_heads <= 0) return 0;
  const RecurrentParams& a = *params;
  if (!recurrent_params_ok(kRuleDelta, a) || (a.D % 8) || (a.E % 8) || a.D > kDlMaxD || !a.y || !a.xc || (a.ldx % 8) ||
      (reinterpret_cast<uintptr_t>(a.xc) & 15) || !tiles || !heads || !square || !scalars)
    return kBadArgument;
  const DeltaChunks dc{tiles, heads, static_cast<__nv_bfloat16*>(square), scalars};
  const int np = (a.D + 15) / 16 * 16;
  cudaError_t r = launch_kernel(delta_chunk_kernel, dim3(n_tiles, a.H), dim3(kDlPrep), 4 * kDlC * (np + 8), s, a, dc);
  if (r != cudaSuccess) return static_cast<int>(r);
  const int smem = delta_smem_bytes(a.D);
  const dim3 grid(n_heads, a.H, (a.E + kDlBE - 1) / kDlBE);
  auto run = [&](auto fn) -> cudaError_t {
    const cudaError_t r = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    return r != cudaSuccess ? r : launch_kernel(fn, grid, dim3(kDlThreads), smem, s, a, dc);
  };
  return static_cast<int>(np == 128 ? run(delta_mma_kernel<128>) : np == 64 ? run(delta_mma_kernel<64>) : run(delta_mma_kernel<0>));
}
}
