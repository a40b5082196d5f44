// Time mixing (see recurrent.cuh) over long entries on tensor cores, with fp32-class products.
//
// Chunks of 32 tokens in two halves of 16.  With L_i [D] the running sum of the log decays inside the chunk (L before its first token
// is 0), S the state before it and all products of vectors per channel,
//     o_i = S^T (r_i e^(L_(i-1))) + sum_{j < i} A_ij v_j + (sum_d r_i u k_i) v_i,   A_ij = sum_d r_i k_j e^(L_(i-1) - L_j)
//     S  <- diag(e^(L_n)) S + sum_j (k_j e^(L_n - L_j)) v_j^T
// Decays may be arbitrarily strong, so no exponential of a positive number is taken: inside a half A is summed directly, and between
// the halves it is the product of r_i e^(L_(i-1) - L_15) with k_j e^(L_15 - L_j).  r, k, v are bf16 to begin with; decayed vectors,
// A and the state are fp32 operands, split into two bf16 parts, hi + lo (the significant cross products of m16n8k16 MMAs).
//
// time_mix_chunk_kernel computes A (the bonus on its diagonal) of all chunks at once; time_mix_mma_kernel walks the chunks with the
// state, one CTA = (segment of an entry, head, 64 columns of E).  As in ssm_mma.cu, few long entries are cut into segments that a
// first launch reduces to their contributions, chained before the second.
#include "common.cuh"
#include "host_utils.cuh"
#include "recurrent.cuh"
#include "warp_mma.cuh"

namespace apb {

constexpr int kTmThreads = 256;
constexpr int kTmC = 32, kTmHalf = 16;
constexpr int kTmBE = 64;
constexpr int kTmVS = kTmBE + 8;
constexpr int kTmAS = kTmC + 8;
constexpr int kTmMaxD = 128;
constexpr int kTmPairs = kTmHalf * (kTmHalf + 1) / 2;

constexpr int kTmSquare = kTmC * kTmC;

struct TimeMixScan {
  ScanSegments sg;
  float* decay;           // [n][H][D] log2 decay over a segment
  const int* tiles;       // [chunks][2] entry, first row
  const int* seg_tile;    // [n] first chunk of a segment
  __nv_bfloat16* square;  // [chunks][H][2][32][32]: A hi, A lo
};

// L [32][np + 4] holds a chunk's decay projections (rows from n on: anything) and receives the running sums of its log2 decays; all
// threads, two barriers inside, one needed behind.  part: [4][np] scratch.  Returns a channel's sum over the chunk (threads below np).
__device__ __forceinline__ float decay_sums(float* L, int ls, const float* w0, float* part, int np, int n) {
  const int lanes = np <= 64 ? 64 : 128, runs = kTmThreads / lanes, len = kTmC / runs;     // a thread: one channel, one run of tokens
  const int ch = threadIdx.x % lanes, run = threadIdx.x / lanes;
  if (ch < np) {
    float sum = 0.f;
    for (int i = run * len; i < (run + 1) * len; ++i) {
      if (i < n) sum -= fminf(wm_ex2((L[i * ls + ch] + w0[ch]) * 1.4426950408889634f) * 1.4426950408889634f, kMaxLogDecay);
      L[i * ls + ch] = sum;
    }
    part[run * np + ch] = sum;
  }
  __syncthreads();
  float before = 0.f, total = 0.f;
  if (ch < np) {
    for (int x = 0; x < runs; ++x) {
      if (x == run) before = total;
      total += part[x * np + ch];
    }
    if (run > 0)
      for (int i = run * len; i < (run + 1) * len; ++i) L[i * ls + ch] += before;
  }
  return total;
}

__host__ __device__ inline int time_mix_chunk_smem(int D) {
  const int np = (D + 15) / 16 * 16, ns = np + 8;
  return 2 * (2 * kTmC * ns + 4 * kTmHalf * ns + 2 * kTmSquare) + 4 * (kTmC * (np + 4) + 6 * np);
}

__global__ void __launch_bounds__(kTmThreads)
time_mix_chunk_kernel(const RecurrentParams p, const TimeMixScan ts) {
  pdl_entry();
  extern __shared__ __align__(128) uint8_t tm_smem[];
  __shared__ uint8_t s_pair[kTmPairs];           // (i, j <= i) of a half, i in the upper four bits
  const int tile = blockIdx.x, h = blockIdx.y, en = ts.tiles[2 * tile], t0 = ts.tiles[2 * tile + 1];
  const int n = min(kTmC, p.e.len[en] - t0);
  const int D = p.D, np = (D + 15) & ~15, ns = np + 8, ls = np + 4, n16 = np >> 4, pc = np >> 3, kh = h / (p.H / p.KH);
  const long long row0 = p.e.start[en] + t0;
  __nv_bfloat16* R = reinterpret_cast<__nv_bfloat16*>(tm_smem);      // [32][ns]
  __nv_bfloat16* K = R + kTmC * ns;
  __nv_bfloat16* Xh = K + kTmC * ns;                                 // [16][ns] second half's r e^(L before - L_15)
  __nv_bfloat16* Xl = Xh + kTmHalf * ns;
  __nv_bfloat16* Yh = Xl + kTmHalf * ns;                             // [16][ns] first half's k e^(L_15 - L)
  __nv_bfloat16* Yl = Yh + kTmHalf * ns;
  __nv_bfloat16* Ah = Yl + kTmHalf * ns;                             // [32][32]
  __nv_bfloat16* Al = Ah + kTmSquare;
  float* L = reinterpret_cast<float*>(Al + kTmSquare);               // [32][np + 4]
  float* bonus = L + kTmC * ls;                                      // [np]
  float* w0 = bonus + np;                                            // [np]
  float* part = w0 + np;                                             // [4][np]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int quad_row = lane >> 2, quad_col = (lane & 3) * 2, mat = lane >> 3, rowin = lane & 7;
  const __nv_bfloat16* pb = static_cast<const __nv_bfloat16*>(p.p);
  for (int i = threadIdx.x; i < 2 * kTmC * pc; i += kTmThreads) {
    const int m = i / (kTmC * pc), r = i / pc % kTmC, c = i % pc, ok = r < n && c * 8 < D;
    wm_cp_async16(smem_u32(R + (m * kTmC + r) * ns + c * 8),
                  pb + (row0 + (ok ? r : 0)) * p.ld + (m ? p.k_off : p.q_off) + static_cast<long long>(kh) * D + (ok ? c * 8 : 0), ok ? 16 : 0);
  }
  const int zc = np >> 2;
  for (int i = threadIdx.x; i < kTmC * zc; i += kTmThreads) {
    const int r = i / zc, c = i % zc, ok = r < n && c * 4 < D;
    wm_cp_async16(smem_u32(L + r * ls + c * 4), p.z + (row0 + (ok ? r : 0)) * p.ldz + static_cast<long long>(h) * D + (ok ? c * 4 : 0), ok ? 16 : 0);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  for (int i = threadIdx.x; i < np; i += kTmThreads) {
    bonus[i] = i < D ? __bfloat162float(static_cast<const __nv_bfloat16*>(p.w1)[h * D + i]) : 0.f;
    w0[i] = i < D ? __bfloat162float(static_cast<const __nv_bfloat16*>(p.w0)[h * D + i]) : 0.f;
  }
  if (threadIdx.x < kTmHalf)
    for (int j = 0; j <= threadIdx.x; ++j) s_pair[threadIdx.x * (threadIdx.x + 1) / 2 + j] = threadIdx.x << 4 | j;
  for (int i = threadIdx.x; i < 2 * kTmSquare / 8; i += kTmThreads) reinterpret_cast<uint4*>(Ah)[i] = make_uint4(0, 0, 0, 0);
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  decay_sums(L, ls, w0, part, np, n);
  __syncthreads();
  // ---- factors between the halves
  for (int i = threadIdx.x; i < kTmHalf * (np >> 1); i += kTmThreads) {
    const int r = i / (np >> 1), c = (i % (np >> 1)) * 2, o = r * ns + c;
    const float2 lm = *reinterpret_cast<const float2*>(L + (kTmHalf - 1) * ls + c), lj = *reinterpret_cast<const float2*>(L + r * ls + c);
    const float2 lp = *reinterpret_cast<const float2*>(L + (kTmHalf + r - 1) * ls + c);
    const float2 k = wm_pair(K + o), q = wm_pair(R + o + kTmHalf * ns);
    wm_store_split2(Yh + o, Yl + o, k.x * wm_ex2(lm.x - lj.x), k.y * wm_ex2(lm.y - lj.y));
    wm_store_split2(Xh + o, Xl + o, q.x * wm_ex2(lp.x - lm.x), q.y * wm_ex2(lp.y - lm.y));
  }
  // ---- A inside the halves: 2 x kTmPairs pairs (i, j <= i), four lanes each
  for (int task = warp * 8 + (lane >> 2); task < 2 * kTmPairs; task += 64) {          // 272 = 4 * 64 + 16: whole warps stay together
    const int half = task >= kTmPairs, pair = s_pair[half ? task - kTmPairs : task];
    const int i = half * kTmHalf + (pair >> 4), j = half * kTmHalf + (pair & 15);
    float sum = 0.f;
    for (int d = (lane & 3) * 4; d < np; d += 16) {
      const float4 q = wm_quad(R + i * ns + d), k = wm_quad(K + j * ns + d);
      float4 f;
      if (i == j) {
        f = *reinterpret_cast<const float4*>(bonus + d);
      } else {
        const float4 a = *reinterpret_cast<const float4*>(L + (i - 1) * ls + d), b = *reinterpret_cast<const float4*>(L + j * ls + d);
        f = make_float4(wm_ex2(a.x - b.x), wm_ex2(a.y - b.y), wm_ex2(a.z - b.z), wm_ex2(a.w - b.w));
      }
      sum += q.x * k.x * f.x + q.y * k.y * f.y + q.z * k.z * f.z + q.w * k.w * f.w;
    }
    const unsigned mask = __activemask();
    sum += __shfl_xor_sync(mask, sum, 1);
    sum += __shfl_xor_sync(mask, sum, 2);
    if ((lane & 3) == 0) {
      const __nv_bfloat16 hi = __float2bfloat16(sum);
      Ah[i * kTmC + j] = hi;
      Al[i * kTmC + j] = __float2bfloat16(sum - __bfloat162float(hi));
    }
  }
  __syncthreads();
  // ---- A between the halves: 8 keys each of two warps
  if (warp < 2) {
    const int k0 = warp * 8;
    float a[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
    for (int ks = 0; ks < n16; ++ks) {
      uint32_t xh[4], xl[4], yh[2], yl[2];
      const int xo = (rowin + (mat & 1) * 8) * ns + ks * 16 + (mat >> 1) * 8, yo = (k0 + rowin) * ns + ks * 16 + (mat & 1) * 8;
      wm_ldsm4(Xh + xo, xh);
      wm_ldsm4(Xl + xo, xl);
      wm_ldsm2(Yh + yo, yh);
      wm_ldsm2(Yl + yo, yl);
      wm_mma(a, xl, yh[0], yh[1]);
      wm_mma(a, xh, yl[0], yl[1]);
      wm_mma(a, xh, yh[0], yh[1]);
    }
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      const int x = (kTmHalf + quad_row + 8 * hh) * kTmC + k0 + quad_col;
      wm_store_split2(Ah + x, Al + x, a[2 * hh], a[2 * hh + 1]);
    }
  }
  __syncthreads();
  uint4* out = reinterpret_cast<uint4*>(ts.square + (static_cast<long long>(tile) * p.H + h) * 2 * kTmSquare);
  out[threadIdx.x] = reinterpret_cast<const uint4*>(Ah)[threadIdx.x];
  static_assert(kTmThreads * 8 == 2 * kTmSquare, "16 bytes of A per thread");
}

__host__ __device__ inline int time_mix_smem_bytes(int D) {
  const int np = (D + 15) / 16 * 16, ns = np + 8;
  // r, k twice; v twice; A twice; decayed r and k; state | L twice, w0, partial sums
  return 2 * (4 * kTmC * ns + 2 * kTmC * kTmVS + 4 * kTmC * kTmAS + 4 * kTmC * ns + 2 * np * kTmVS) + 4 * (2 * kTmC * (np + 4) + 5 * np);
}

template <int NP>
__global__ void __launch_bounds__(kTmThreads, NP == 128 || NP == 0 ? 1 : 2)
time_mix_mma_kernel(const RecurrentParams p, const TimeMixScan ts, int state_only) {
  pdl_entry();
  extern __shared__ __align__(128) uint8_t tm_smem[];
  const ScanSegments& sg = ts.sg;
  const int* w = sg.seg + blockIdx.x * 6;
  const int en = w[0], t_begin = w[1], n_tok = w[2], carry_in = w[3], carry_out = w[4], is_last = w[5];
  if (state_only && carry_out < 0) return;
  const int h = blockIdx.y, e0 = blockIdx.z * kTmBE, kh = h / (p.H / p.KH), tile0 = ts.seg_tile[blockIdx.x];
  const int D = p.D, E = p.E, np = NP ? NP : (D + 15) & ~15, ns = np + 8, ls = np + 4, n16 = np >> 4, pc = np >> 3;
  const int be = min(kTmBE, E - e0);
  const long long start = p.e.start[en] + t_begin;
  const int pos0 = p.e.pos0[en] + t_begin, slot = p.e.slot[en];
  __nv_bfloat16* RK2 = reinterpret_cast<__nv_bfloat16*>(tm_smem);    // two buffers [64][ns]: r, then k
  __nv_bfloat16* V2 = RK2 + 4 * kTmC * ns;                           // two buffers [32][72]
  __nv_bfloat16* A2 = V2 + 2 * kTmC * kTmVS;                         // two buffers [2][32][40]: A hi, A lo
  __nv_bfloat16* Rh = A2 + 4 * kTmC * kTmAS;                         // [32][ns] r e^L before the token
  __nv_bfloat16* Rl = Rh + kTmC * ns;
  __nv_bfloat16* Kh = Rl + kTmC * ns;                                // [32][ns] k e^(L_n - L)
  __nv_bfloat16* Kl = Kh + kTmC * ns;
  __nv_bfloat16* Sh = Kl + kTmC * ns;                                // [np][72] state before the chunk
  __nv_bfloat16* Sl = Sh + np * kTmVS;
  float* L2 = reinterpret_cast<float*>(Sl + np * kTmVS);             // two buffers [32][np + 4]: decay projections, then L
  float* w0 = L2 + 2 * kTmC * ls;                                    // [np]
  float* part = w0 + np;                                             // [4][np]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int quad_row = lane >> 2, quad_col = (lane & 3) * 2, mat = lane >> 3, rowin = lane & 7;
  const __nv_bfloat16* pb = static_cast<const __nv_bfloat16*>(p.p);

  auto fetch = [&](int t0, int buf) {
#pragma unroll
    for (int i = threadIdx.x; i < 2 * kTmC * pc; i += kTmThreads) {
      const int m = i / (kTmC * pc), r = i / pc % kTmC, c = i % pc, ok = t0 + r < n_tok && c * 8 < D;
      wm_cp_async16(smem_u32(RK2 + ((buf * 2 + m) * kTmC + r) * ns + c * 8),
                    pb + (start + (ok ? t0 + r : 0)) * p.ld + (m ? p.k_off : p.q_off) + static_cast<long long>(kh) * D + (ok ? c * 8 : 0), ok ? 16 : 0);
    }
    {
      const int r = threadIdx.x >> 3, c = threadIdx.x & 7, ok = t0 + r < n_tok && c * 8 < be;
      wm_cp_async16(smem_u32(V2 + (buf * kTmC + r) * kTmVS + c * 8),
                    pb + (start + (ok ? t0 + r : 0)) * p.ld + p.v_off + static_cast<long long>(h) * E + e0 + (ok ? c * 8 : 0), ok ? 16 : 0);
    }
    const int zc = np >> 2;
#pragma unroll
    for (int i = threadIdx.x; i < kTmC * zc; i += kTmThreads) {
      const int r = i / zc, c = i % zc, ok = t0 + r < n_tok && c * 4 < D;
      wm_cp_async16(smem_u32(L2 + (buf * kTmC + r) * ls + c * 4),
                    p.z + (start + (ok ? t0 + r : 0)) * p.ldz + static_cast<long long>(h) * D + (ok ? c * 4 : 0), ok ? 16 : 0);
    }
    if (!state_only) {                             // 16-byte pieces: matrix, row, quarter
      const __nv_bfloat16* sq = ts.square + (static_cast<long long>(tile0 + t0 / kTmC) * p.H + h) * 2 * kTmSquare;
      const int i = threadIdx.x;
      wm_cp_async16(smem_u32(A2 + ((buf * 2 + i / (kTmC * 4)) * kTmC + i / 4 % kTmC) * kTmAS + (i & 3) * 8), sq + i * 8, 16);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  static_assert(kTmThreads == kTmC * kTmBE / 8, "one 16-byte piece of v per thread");
  fetch(0, 0);
  for (int i = threadIdx.x; i < np; i += kTmThreads) w0[i] = i < D ? __bfloat162float(static_cast<const __nv_bfloat16*>(p.w0)[h * D + i]) : 0.f;
  const float* s_in = nullptr;
  if (!state_only) {
    if (carry_in >= 0)
      s_in = sg.carry + (static_cast<long long>(carry_in) * p.H + h) * D * E;
    else if (pos0 > 0)
      s_in = p.state + (static_cast<long long>(slot) * p.H + h) * D * E;
  }
  StateTile st;
  st.load(s_in ? s_in + e0 : nullptr, E, D, be);
  bool have_state = s_in != nullptr;
  if (have_state && warp < n16) st.split_to(Sh, Sl, kTmVS);
  float total = 0.f;                               // log2 decay of the segment (a channel per thread)

  for (int t0 = 0, buf = 0; t0 < n_tok; t0 += kTmC, buf ^= 1) {
    const int n = min(kTmC, n_tok - t0);
    const bool more = t0 + kTmC < n_tok;
    const __nv_bfloat16* R = RK2 + buf * 2 * kTmC * ns;
    const __nv_bfloat16* K = R + kTmC * ns;
    const __nv_bfloat16* V = V2 + buf * kTmC * kTmVS;
    const __nv_bfloat16* A = A2 + buf * 2 * kTmC * kTmAS;
    float* L = L2 + buf * kTmC * ls;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                               // this chunk has landed; everybody is done with the last one
    if (more) fetch(t0 + kTmC, buf ^ 1);
    total += decay_sums(L, ls, w0, part, np, n);
    __syncthreads();
    // ---- decayed vectors
    for (int i = threadIdx.x; i < kTmC * (np >> 1); i += kTmThreads) {
      const int r = i / (np >> 1), c = (i % (np >> 1)) * 2, o = r * ns + c;
      const float2 li = *reinterpret_cast<const float2*>(L + r * ls + c), ln = *reinterpret_cast<const float2*>(L + (kTmC - 1) * ls + c);
      const float2 k = wm_pair(K + o);
      wm_store_split2(Kh + o, Kl + o, k.x * wm_ex2(ln.x - li.x), k.y * wm_ex2(ln.y - li.y));
      if (!have_state) continue;
      const float2 lp = r ? *reinterpret_cast<const float2*>(L + (r - 1) * ls + c) : make_float2(0.f, 0.f);
      const float2 q = wm_pair(R + o);
      wm_store_split2(Rh + o, Rl + o, q.x * wm_ex2(lp.x), q.y * wm_ex2(lp.y));
    }
    __syncthreads();
    if (!state_only) {
      const int r0 = (warp & 1) * 16, c0 = (warp >> 1) * 16;   // this warp's tile of the output
      float o[2][4];
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) o[nt][0] = o[nt][1] = o[nt][2] = o[nt][3] = 0.f;
      if (have_state) {
#pragma unroll 4
        for (int ks = 0; ks < n16; ++ks) {
          uint32_t ah[4], al[4], sh[4], sl[4];
          const int ao = (r0 + rowin + (mat & 1) * 8) * ns + ks * 16 + (mat >> 1) * 8;
          const int so = (ks * 16 + rowin + 8 * (mat & 1)) * kTmVS + c0 + (mat >> 1) * 8;
          wm_ldsm4(Rh + ao, ah);
          wm_ldsm4(Rl + ao, al);
          wm_ldsm4_t(Sh + so, sh);
          wm_ldsm4_t(Sl + so, sl);
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            wm_mma(o[nt], al, sh[2 * nt], sh[2 * nt + 1]);
            wm_mma(o[nt], ah, sl[2 * nt], sl[2 * nt + 1]);
            wm_mma(o[nt], ah, sh[2 * nt], sh[2 * nt + 1]);
          }
        }
      }
      for (int ks = 0; ks < (r0 + 16) / 16; ++ks) {
        uint32_t ah[4], al[4], v[4];
        const int ao = (r0 + rowin + (mat & 1) * 8) * kTmAS + ks * 16 + (mat >> 1) * 8;
        wm_ldsm4(A + ao, ah);
        wm_ldsm4(A + kTmC * kTmAS + ao, al);
        wm_ldsm4_t(V + (ks * 16 + rowin + 8 * (mat & 1)) * kTmVS + c0 + (mat >> 1) * 8, v);
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
          float* dst = p.y + (start + t0 + i) * p.H * E + static_cast<long long>(h) * E + e0;
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            const int c = c0 + nt * 8 + quad_col;
            if (c < be) *reinterpret_cast<float2*>(dst + c) = make_float2(o[nt][2 * hh], o[nt][2 * hh + 1]);
          }
        }
      }
      if (more) __syncthreads();                   // everybody has read the state operand
    }
    // ---- S = diag(e^(L_n)) S + K^T V
    if (warp < n16) {
      const float* ln = L + (kTmC - 1) * ls + warp * 16 + quad_row;
      st.scale(wm_ex2(ln[0]), wm_ex2(ln[8]));
#pragma unroll
      for (int ks = 0; ks < kTmC / 16; ++ks) {
        uint32_t kh4[4], kl4[4];
        const int ko = (ks * 16 + rowin + (mat >> 1) * 8) * ns + warp * 16 + (mat & 1) * 8;
        wm_ldsm4_t(Kh + ko, kh4);
        wm_ldsm4_t(Kl + ko, kl4);
#pragma unroll
        for (int n2 = 0; n2 < 4; ++n2) {
          uint32_t v[4];
          wm_ldsm4_t(V + (ks * 16 + rowin + 8 * (mat & 1)) * kTmVS + n2 * 16 + (mat >> 1) * 8, v);
#pragma unroll
          for (int q = 0; q < 2; ++q) {
            wm_mma(st.s[2 * n2 + q], kl4, v[2 * q], v[2 * q + 1]);
            wm_mma(st.s[2 * n2 + q], kh4, v[2 * q], v[2 * q + 1]);
          }
        }
      }
      if (!state_only && more) st.split_to(Sh, Sl, kTmVS);
    }
    have_state = !state_only;
  }
  // ---- the state after the segment
  float* s_out = state_only ? sg.carry + (static_cast<long long>(carry_out) * p.H + h) * D * E
                            : (is_last ? p.state + (static_cast<long long>(slot) * p.H + h) * D * E : nullptr);
  if (s_out && warp < n16) st.store(s_out + e0, E, D, be);
  if (state_only && e0 == 0 && threadIdx.x < D) ts.decay[(static_cast<long long>(blockIdx.x) * p.H + h) * D + threadIdx.x] = total;
}

// Chains the contributions of an entry's segments: scratch[base] becomes the state before the entry, scratch[base + i] the state
// before its i-th segment.  chains [n][4]: entry, base, segments, index of its first segment.
__global__ void __launch_bounds__(256)
time_mix_carry_kernel(const RecurrentParams p, const TimeMixScan ts, const int* __restrict__ chains) {
  pdl_entry();
  const int* c = chains + blockIdx.x * 4;
  const int en = c[0], base = c[1], n_seg = c[2], first = c[3], h = blockIdx.y;
  const int size = p.D * p.E, i = blockIdx.z * 256 + threadIdx.x;
  if (i >= size) return;
  const long long stride = static_cast<long long>(p.H) * size;
  float* x = ts.sg.carry + static_cast<long long>(base) * stride + static_cast<long long>(h) * size + i;
  float s = p.e.pos0[en] > 0 ? p.state[static_cast<long long>(p.e.slot[en]) * stride + static_cast<long long>(h) * size + i] : 0.f;
  x[0] = s;
  for (int k = 0; k + 1 < n_seg; ++k) {
    s = s * wm_ex2(ts.decay[(static_cast<long long>(first + k) * p.H + h) * p.D + i / p.E]) + x[(k + 1) * stride];
    x[(k + 1) * stride] = s;
  }
}

}  // namespace apb

extern "C" {
using namespace apb;

// bf16; D a multiple of 8 up to 128, E a multiple of 8, 16-byte aligned columns; z rows of 16-byte aligned columns.  tiles [n_tiles, 2]:
// the chunks of 32 rows of the entries longer than one token, in order; seg_tile [n_seg]: first chunk of every segment; square: scratch
// [n_tiles, H, 2, 32, 32].  Writes y for the segments' rows and the entries' states.  n_chains > 0: some entries have several segments
// (carry, decay [n_seg, H, D]: scratch).
int apb_time_mix_mma(const RecurrentParams* params, const int* tiles, int n_tiles, const int* seg, const int* seg_tile, int n_seg,
                     void* square, float* carry, float* decay, const int* chains, int n_chains, cudaStream_t s) {
  if (n_seg <= 0 || n_tiles <= 0) return 0;
  const RecurrentParams& a = *params;
  if (!recurrent_params_ok(kRuleTimeMix, a) || (a.D % 8) || (a.E % 8) || a.D > kTmMaxD || !a.y || !seg || !tiles || !seg_tile || !square ||
      ((a.ld | a.q_off | a.k_off | a.v_off) & 7) || (a.ldz & 3) || ((reinterpret_cast<uintptr_t>(a.p) | reinterpret_cast<uintptr_t>(a.z)) & 15) ||
      (n_chains > 0 && (!carry || !decay || !chains)))
    return kBadArgument;
  const TimeMixScan ts{ScanSegments{seg, carry}, decay, tiles, seg_tile, static_cast<__nv_bfloat16*>(square)};
  auto start = [&](auto fn, dim3 grid, int smem, auto... args) -> cudaError_t {
    const cudaError_t r = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    return r != cudaSuccess ? r : launch_kernel(fn, grid, dim3(kTmThreads), smem, s, a, ts, args...);
  };
  cudaError_t r = start(time_mix_chunk_kernel, dim3(n_tiles, a.H), time_mix_chunk_smem(a.D));
  if (r != cudaSuccess) return static_cast<int>(r);
  const int smem = time_mix_smem_bytes(a.D), np = (a.D + 15) / 16 * 16;
  const dim3 grid(n_seg, a.H, (a.E + kTmBE - 1) / kTmBE);
  auto run = [&](auto fn) -> cudaError_t {
    if (n_chains > 0) {
      cudaError_t r = start(fn, grid, smem, 1);
      if (r != cudaSuccess) return r;
      r = launch_kernel(time_mix_carry_kernel, dim3(n_chains, a.H, (a.D * a.E + 255) / 256), dim3(256), 0, s, a, ts, chains);
      if (r != cudaSuccess) return r;
    }
    return start(fn, grid, smem, 0);
  };
  return static_cast<int>(np == 128 ? run(time_mix_mma_kernel<128>) : np == 64 ? run(time_mix_mma_kernel<64>) : run(time_mix_mma_kernel<0>));
}
}
