// Matrix memory (see recurrent.cuh) over long entries on tensor cores, with fp32-class products.
//
// Chunks of 32 tokens.  With F_i the running sum of the log forget gates inside the chunk, G_j = i_j - F_j, and S, n, m before the
// chunk, the running maximum is m_i = F_i + M_i with M_i = max(m, max_{j <= i} G_j), and
//     a_ij = D^-1/2 (q_i . k_j) exp(G_j - M_i)  (j <= i),    c_i = D^-1/2 exp(m - M_i)
//     o_i  = (sum_j a_ij v_j + c_i S^T q_i) / (max(|sum_j a_ij + c_i (n . q_i)|, exp(-m_i)) + 1e-6)
//     S <- exp(m - M_n) S + sum_j k_j (exp(G_j - M_n) v_j)^T,  n alike,  m <- F_n + M_n
// so every exponential is at most 1.  q, k and v are bf16 to begin with; fp32 operands (scores, weighted values, the state) are split
// into two bf16 parts, hi + lo, and take part as two m16n8k16 MMAs.  The state itself stays in fp32 registers, n in shared memory.
//
// One CTA = (segment of an entry, head, 64 columns of E), two per SM.  As in ssm_mma.cu, few long entries are cut into segments
// that a first launch reduces to their contributions, chained before the second.
#include "common.cuh"
#include "host_utils.cuh"
#include "recurrent.cuh"
#include "warp_mma.cuh"

namespace apb {

constexpr int kMmThreads = 256;
constexpr int kMmC = 32;                  // tokens per chunk
constexpr int kMmBE = 64;                 // E columns per CTA
constexpr int kMmVS = kMmBE + 8;          // row strides (elements): odd multiples of 16 bytes
constexpr int kMmAS = kMmC + 8;
constexpr int kMmMaxD = 128;
constexpr float kLog2e = 1.4426950408889634f, kLn2 = 0.6931471805599453f;

struct MemoryScan {
  ScanSegments sg;
  const float2* gates;    // [rows, H] log2 of the forget and input gates
  float* aux0;            // [entries][H][D + 1] n, m before the step (a slot's aux is replaced while other columns still start)
  float* carry_aux;       // [scratch states][H][D + 1] n, m (log2)
  float2* totals;         // [n][H] of a segment's contribution: F over the segment, m (log2)
};

__global__ void __launch_bounds__(256)
memory_gates_kernel(const RecurrentParams p, float2* __restrict__ gates, long long n, float* __restrict__ aux0, int n_entries) {
  pdl_entry();
  const long long i = blockIdx.x * 256LL + threadIdx.x;
  if (i >= n) {
    const long long j = i - n, per = static_cast<long long>(p.H) * (p.D + 1);
    if (j < n_entries * per && p.e.pos0[j / per] > 0) aux0[j] = p.aux[p.e.slot[j / per] * per + j % per];
    return;
  }
  const unsigned j = static_cast<unsigned>(i), H = p.H;
  const float2 g = memory_gates<__nv_bfloat16>(p, j / H, static_cast<int>(j % H));
  gates[i] = make_float2(g.x * kLog2e, g.y * kLog2e);
}

__host__ __device__ inline int memory_smem_bytes(int D) {
  const int np = (D + 15) / 16 * 16, ns = np + 8;
  return 2 * (3 * kMmC * ns + 4 * kMmC * kMmVS + 2 * kMmC * kMmAS + 2 * np * kMmVS);
}

// NP: D rounded up to 16 when known at compile time, else 0.
template <int NP>
__global__ void __launch_bounds__(kMmThreads, 2)
memory_mma_kernel(const RecurrentParams p, const MemoryScan ms, int state_only) {
  pdl_entry();
  extern __shared__ __align__(128) uint8_t mm_smem[];
  __shared__ float s_g[2][kMmC], s_m[2][kMmC], s_floor[2][kMmC], s_m0[2];    // G, M, exp(-m) and the maximum before, of two chunks
  __shared__ float s_n[kMmMaxD], s_w[kMmC], s_qn[kMmC], s_rows[4][kMmC];
  const ScanSegments& sg = ms.sg;
  const int* w = sg.seg + blockIdx.x * 6;
  const int en = w[0], t_begin = w[1], n_tok = w[2], carry_in = w[3], carry_out = w[4], is_last = w[5];
  if (state_only && carry_out < 0) return;
  const int h = blockIdx.y, e0 = blockIdx.z * kMmBE, kh = h / (p.H / p.KH);
  const int D = p.D, E = p.E, np = NP ? NP : (D + 15) & ~15, ns = np + 8, n16 = np >> 4;
  const int be = min(kMmBE, E - e0);
  const long long start = p.e.start[en] + t_begin;
  const int pos0 = p.e.pos0[en] + t_begin, slot = p.e.slot[en];
  __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(mm_smem);
  __nv_bfloat16* K2 = Qs + kMmC * ns;            // two buffers [32][ns]
  __nv_bfloat16* V2 = K2 + 2 * kMmC * ns;        // two buffers [32][72]
  __nv_bfloat16* Wh = V2 + 2 * kMmC * kMmVS;     // values times their weight in the state after the chunk, hi / lo
  __nv_bfloat16* Wl = Wh + kMmC * kMmVS;
  __nv_bfloat16* Ah = Wl + kMmC * kMmVS;         // [32][40] scores
  __nv_bfloat16* Al = Ah + kMmC * kMmAS;
  __nv_bfloat16* Sh = Al + kMmC * kMmAS;         // [np][72] state before the chunk
  __nv_bfloat16* Sl = Sh + np * kMmVS;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int quad_row = lane >> 2, quad_col = (lane & 3) * 2;
  const int mat = lane >> 3, rowin = lane & 7;
  const __nv_bfloat16* pb = static_cast<const __nv_bfloat16*>(p.p);
  const float q_scale = 1.f / sqrtf(static_cast<float>(D));

  // rows beyond the segment and columns beyond D are filled with zeros
  const int pc = np >> 3;                        // 16-byte pieces of a row
  auto fetch_rows = [&](int t0, long long off, __nv_bfloat16* dst) {
#pragma unroll
    for (int i = threadIdx.x; i < kMmC * pc; i += kMmThreads) {
      const int r = i / pc, c = i % pc, ok = t0 + r < n_tok && c * 8 < D;
      wm_cp_async16(smem_u32(dst + r * ns + c * 8), pb + (start + (ok ? t0 + r : 0)) * p.ld + off + (ok ? c * 8 : 0), ok ? 16 : 0);
    }
  };
  auto fetch_kv = [&](int t0, int buf) {
    fetch_rows(t0, p.k_off + static_cast<long long>(kh) * D, K2 + buf * kMmC * ns);
    const int r = threadIdx.x >> 3, c = threadIdx.x & 7, ok = t0 + r < n_tok && c * 8 < be;
    wm_cp_async16(smem_u32(V2 + buf * kMmC * kMmVS + r * kMmVS + c * 8),
                  pb + (start + (ok ? t0 + r : 0)) * p.ld + p.v_off + static_cast<long long>(h) * E + e0 + (ok ? c * 8 : 0), ok ? 16 : 0);
  };
  static_assert(kMmThreads == kMmC * kMmBE / 8 && kMmC == 32, "one 16-byte piece of v per thread, one token per lane");

  // the state before the segment
  const float* s_in = nullptr;
  const float* a_in = nullptr;
  float to_log2 = 1.f;
  if (!state_only) {
    if (carry_in >= 0) {
      s_in = sg.carry + (static_cast<long long>(carry_in) * p.H + h) * D * E;
      a_in = ms.carry_aux + (static_cast<long long>(carry_in) * p.H + h) * (D + 1);
    } else if (pos0 > 0) {
      s_in = p.state + (static_cast<long long>(slot) * p.H + h) * D * E;
      a_in = ms.aux0 + (static_cast<long long>(en) * p.H + h) * (D + 1);
      to_log2 = kLog2e;
    }
  }
  float m_run = state_only ? -INFINITY : a_in ? a_in[D] * to_log2 : 0.f, f_run = 0.f;      // warp 7
  auto gates_of = [&](int t0, int buf) {         // warp 7, one token per lane
    const float2 g = t0 + lane < n_tok ? ms.gates[(start + t0 + lane) * p.H + h] : make_float2(0.f, -INFINITY);
    float F = g.x;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, F, o);
      if (lane >= o) F += v;
    }
    const float G = g.y - F;
    float M = G;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, M, o);
      if (lane >= o) M = fmaxf(M, v);
    }
    M = fmaxf(M, m_run);
    s_g[buf][lane] = G;
    s_m[buf][lane] = M;
    s_floor[buf][lane] = wm_ex2(-(F + M));
    if (lane == 0) s_m0[buf] = m_run;
    f_run += __shfl_sync(0xffffffffu, F, 31);
    m_run = __shfl_sync(0xffffffffu, F + M, 31);
  };
  if (!state_only) fetch_rows(0, p.q_off + static_cast<long long>(kh) * D, Qs);
  fetch_kv(0, 0);
  asm volatile("cp.async.commit_group;" ::: "memory");
  if (warp == 7) gates_of(0, 0);
  StateTile st;
  st.load(s_in ? s_in + e0 : nullptr, E, D, be);
  bool have_state = s_in != nullptr;
  if (have_state && warp < n16) st.split_to(Sh, Sl, kMmVS);
  if (threadIdx.x < np) s_n[threadIdx.x] = a_in && threadIdx.x < D ? a_in[threadIdx.x] : 0.f;

  for (int t0 = 0, buf = 0; t0 < n_tok; t0 += kMmC, buf ^= 1) {
    const int n = min(kMmC, n_tok - t0);
    const bool more = t0 + kMmC < n_tok;
    const __nv_bfloat16* K = K2 + buf * kMmC * ns;
    const __nv_bfloat16* V = V2 + buf * kMmC * kMmVS;
    const float *G = s_g[buf], *M = s_m[buf];
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                               // this chunk has landed; everybody is done with the last one
    const float m0 = s_m0[buf], m_end = M[kMmC - 1];
    if (more) {
      fetch_kv(t0 + kMmC, buf ^ 1);
      if (warp == 7) gates_of(t0 + kMmC, buf ^ 1);
    }
    if (threadIdx.x < kMmC) s_w[threadIdx.x] = wm_ex2(G[threadIdx.x] - m_end);
    for (int i = threadIdx.x; i < kMmC * (kMmBE / 2); i += kMmThreads) {
      const int r = i / (kMmBE / 2), o = r * kMmVS + (i % (kMmBE / 2)) * 2;
      const float2 f = wm_pair(V + o);
      const float wt = wm_ex2(G[r] - m_end);
      wm_store_split2(Wh + o, Wl + o, f.x * wt, f.y * wt);
    }
    const int r0 = (warp & 1) * 16, c0 = (warp >> 1) * 16;     // this warp's tile of the output
    float o[2][4];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) o[nt][0] = o[nt][1] = o[nt][2] = o[nt][3] = 0.f;
    if (!state_only) {
      // ---- scores: 16 queries x 8 keys per warp; the state's share of the outputs
      const int k0 = (warp >> 1) * 8;
      float a[4] = {0.f, 0.f, 0.f, 0.f};
      const bool live = k0 <= r0 + 15;
#pragma unroll 4
      for (int ks = 0; ks < n16; ++ks) {
        uint32_t q[4];
        wm_ldsm4(Qs + (r0 + rowin + (mat & 1) * 8) * ns + ks * 16 + (mat >> 1) * 8, q);
        if (live) {
          uint32_t k[2];
          wm_ldsm2(K + (k0 + rowin) * ns + ks * 16 + (mat & 1) * 8, k);
          wm_mma(a, q, k[0], k[1]);
        }
        if (have_state) {
          uint32_t sh[4], sl[4];
          const int so = (ks * 16 + rowin + 8 * (mat & 1)) * kMmVS + c0 + (mat >> 1) * 8;
          wm_ldsm4_t(Sh + so, sh);
          wm_ldsm4_t(Sl + so, sl);
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            wm_mma(o[nt], q, sl[2 * nt], sl[2 * nt + 1]);
            wm_mma(o[nt], q, sh[2 * nt], sh[2 * nt + 1]);
          }
        }
      }
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        const int i = r0 + quad_row + 8 * hh, j = k0 + quad_col;
        const float mi = M[i];
        const float x = j <= i ? a[2 * hh] * q_scale * wm_ex2(G[j] - mi) : 0.f;
        const float y = j + 1 <= i ? a[2 * hh + 1] * q_scale * wm_ex2(G[j + 1] - mi) : 0.f;
        wm_store_split2(Ah + i * kMmAS + j, Al + i * kMmAS + j, x, y);
        float sum = x + y;
        sum += __shfl_xor_sync(0xffffffffu, sum, 1);
        sum += __shfl_xor_sync(0xffffffffu, sum, 2);
        if ((lane & 3) == 0) s_rows[warp >> 1][i] = sum;
        const float f = q_scale * wm_ex2(m0 - mi);
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          o[nt][2 * hh] *= f;
          o[nt][2 * hh + 1] *= f;
        }
      }
      // ---- n . q, four rows per warp
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const int r = warp * 4 + k;
        float sum = 0.f;
        if (have_state)
          for (int d = lane * 2; d < np; d += 64) {
            const float2 q = wm_pair(Qs + r * ns + d);
            sum += q.x * s_n[d] + q.y * s_n[d + 1];
          }
        sum = warp_sum(sum);
        if (lane == 0) s_qn[r] = sum;
      }
    }
    __syncthreads();                               // scores and weights visible; nobody reads q, n or the state operand any more
    if (more && !state_only) fetch_rows(t0 + kMmC, p.q_off + static_cast<long long>(kh) * D, Qs);
    asm volatile("cp.async.commit_group;" ::: "memory");
    const float dn = wm_ex2(m0 - m_end);
    if (!state_only) {
      for (int ks = 0; ks < (r0 + 16) / 16; ++ks) {
        uint32_t ah[4], al[4], v[4];
        const int ao = (r0 + rowin + (mat & 1) * 8) * kMmAS + ks * 16 + (mat >> 1) * 8;
        wm_ldsm4(Ah + ao, ah);
        wm_ldsm4(Al + ao, al);
        wm_ldsm4_t(V + (ks * 16 + rowin + 8 * (mat & 1)) * kMmVS + c0 + (mat >> 1) * 8, v);
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
          const float den = s_rows[0][i] + s_rows[1][i] + s_rows[2][i] + s_rows[3][i] + q_scale * wm_ex2(m0 - M[i]) * s_qn[i];
          const float f = 1.f / (fmaxf(fabsf(den), s_floor[buf][i]) + 1e-6f);
          float* dst = p.y + (start + t0 + i) * p.H * E + static_cast<long long>(h) * E + e0;
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            const int c = c0 + nt * 8 + quad_col;
            if (c < be) *reinterpret_cast<float2*>(dst + c) = make_float2(o[nt][2 * hh] * f, o[nt][2 * hh + 1] * f);
          }
        }
      }
    }
    // ---- state and normaliser
    if (threadIdx.x < np) {
      float x = s_n[threadIdx.x] * dn;
#pragma unroll 8
      for (int j = 0; j < kMmC; ++j) x += s_w[j] * __bfloat162float(K[j * ns + threadIdx.x]);
      s_n[threadIdx.x] = x;
    }
    if (warp < n16) {
      st.scale(dn, dn);
#pragma unroll
      for (int ks = 0; ks < kMmC / 16; ++ks) {
        uint32_t k[4];
        wm_ldsm4_t(K + (ks * 16 + rowin + (mat >> 1) * 8) * ns + warp * 16 + (mat & 1) * 8, k);
#pragma unroll
        for (int n2 = 0; n2 < 4; ++n2) {
          uint32_t wh[4], wl[4];
          const int bo = (ks * 16 + rowin + 8 * (mat & 1)) * kMmVS + n2 * 16 + (mat >> 1) * 8;
          wm_ldsm4_t(Wh + bo, wh);
          wm_ldsm4_t(Wl + bo, wl);
#pragma unroll
          for (int q = 0; q < 2; ++q) {
            wm_mma(st.s[2 * n2 + q], k, wl[2 * q], wl[2 * q + 1]);
            wm_mma(st.s[2 * n2 + q], k, wh[2 * q], wh[2 * q + 1]);
          }
        }
      }
      if (!state_only && more) st.split_to(Sh, Sl, kMmVS);
    }
    have_state = true;
  }
  // ---- the state after the segment (s_n: every thread wrote its own element)
  float* s_out = nullptr;
  float* a_out = nullptr;
  if (state_only) {
    s_out = sg.carry + (static_cast<long long>(carry_out) * p.H + h) * D * E;
    a_out = ms.carry_aux + (static_cast<long long>(carry_out) * p.H + h) * (D + 1);
  } else if (is_last) {
    s_out = p.state + (static_cast<long long>(slot) * p.H + h) * D * E;
    a_out = p.aux + (static_cast<long long>(slot) * p.H + h) * (D + 1);
  }
  if (s_out && warp < n16) st.store(s_out + e0, E, D, be);
  if (a_out && e0 == 0) {
    if (threadIdx.x < D) a_out[threadIdx.x] = s_n[threadIdx.x];
    if (warp == 7 && lane == 0) {
      if (state_only)
        ms.totals[static_cast<long long>(blockIdx.x) * p.H + h] = make_float2(f_run, m_run);
      else
        a_out[D] = m_run * kLn2;
    }
  }
}

// Chains the contributions of an entry's segments: scratch[base] becomes the state before the entry, scratch[base + i] the state
// before its i-th segment.  chains [n][4]: entry, base, segments, index of its first segment.  Elements: S, then n.
__global__ void __launch_bounds__(256)
memory_carry_kernel(const RecurrentParams p, const MemoryScan ms, const int* __restrict__ chains) {
  pdl_entry();
  const int* c = chains + blockIdx.x * 4;
  const int en = c[0], base = c[1], n_seg = c[2], first = c[3], h = blockIdx.y;
  const int size = p.D * p.E, i = blockIdx.z * 256 + threadIdx.x;
  if (i > size + p.D) return;
  const bool seen = p.e.pos0[en] > 0;
  const long long own = static_cast<long long>(p.e.slot[en]) * p.H + h;
  float m = seen ? p.aux[own * (p.D + 1) + p.D] * kLog2e : 0.f;
  const bool is_s = i < size;
  const long long stride = static_cast<long long>(p.H) * (is_s ? size : p.D + 1);
  float* x = (is_s ? ms.sg.carry + static_cast<long long>(h) * size + i : ms.carry_aux + static_cast<long long>(h) * (p.D + 1) + (i - size)) +
             static_cast<long long>(base) * stride;
  const bool is_m = i == size + p.D;
  float s = is_m ? m : !seen ? 0.f : is_s ? p.state[own * size + i] : p.aux[own * (p.D + 1) + (i - size)];
  x[0] = s;
  for (int k = 0; k + 1 < n_seg; ++k) {
    const float2 t = ms.totals[static_cast<long long>(first + k) * p.H + h];
    const float top = fmaxf(t.x + m, t.y);
    s = is_m ? top : s * wm_ex2(t.x + m - top) + x[(k + 1) * stride] * wm_ex2(t.y - top);
    x[(k + 1) * stride] = s;
    m = top;
  }
}

}  // namespace apb

extern "C" {
using namespace apb;

// bf16; D a multiple of 8 up to 128, E a multiple of 8, 16-byte aligned columns.  Writes y for the segments' rows, the entries'
// states and aux.  gates, aux0: scratch [rows, H] float2 and [n_entries, H, D + 1].  n_chains > 0: some entries have several segments (carry, carry_aux, totals:
// scratch).
int apb_memory_mma(const RecurrentParams* params, int rows, int n_entries, void* gates, float* aux0, const int* seg, int n_seg, float* carry, float* carry_aux,
                   void* totals, const int* chains, int n_chains, cudaStream_t s) {
  if (n_seg <= 0) return 0;
  const RecurrentParams& a = *params;
  if (!recurrent_params_ok(kRuleMemory, a) || (a.D % 8) || (a.E % 8) || a.D > kMmMaxD || static_cast<long long>(rows) * a.H > 0x7fffffffLL || !a.y || !gates || !aux0 || !seg ||
      ((a.ld | a.q_off | a.k_off | a.v_off) & 7) || (reinterpret_cast<uintptr_t>(a.p) & 15) ||
      (n_chains > 0 && (!carry || !carry_aux || !totals || !chains)))
    return kBadArgument;
  const MemoryScan ms{ScanSegments{seg, carry}, static_cast<const float2*>(gates), aux0, carry_aux, static_cast<float2*>(totals)};
  const long long n = static_cast<long long>(rows) * a.H, all = n + static_cast<long long>(n_entries) * a.H * (a.D + 1);
  cudaError_t r = launch_kernel(memory_gates_kernel, dim3(static_cast<unsigned>((all + 255) / 256)), dim3(256), 0, s, a, static_cast<float2*>(gates), n,
                                aux0, n_entries);
  if (r != cudaSuccess) return static_cast<int>(r);
  const int smem = memory_smem_bytes(a.D), np = (a.D + 15) / 16 * 16;
  const dim3 grid(n_seg, a.H, (a.E + kMmBE - 1) / kMmBE);
  auto run = [&](auto fn) -> cudaError_t {
    cudaError_t r = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (r != cudaSuccess) return r;
    if (n_chains > 0) {
      r = launch_kernel(fn, grid, dim3(kMmThreads), smem, s, a, ms, 1);
      if (r != cudaSuccess) return r;
      r = launch_kernel(memory_carry_kernel, dim3(n_chains, a.H, (a.D * a.E + a.D + 256) / 256), dim3(256), 0, s, a, ms, chains);
      if (r != cudaSuccess) return r;
    }
    return launch_kernel(fn, grid, dim3(kMmThreads), smem, s, a, ms, 0);
  };
  return static_cast<int>(np == 128 ? run(memory_mma_kernel<128>) : np == 64 ? run(memory_mma_kernel<64>) : run(memory_mma_kernel<0>));
}
}
