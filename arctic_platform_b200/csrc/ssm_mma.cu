// State-space recurrence of long entries on tensor cores, with fp32-class products (see ssm.cuh for the recurrence).
//
// Chunks of 32 tokens.  With L_i the running sum of the log decays inside the chunk and S the state before it,
//     y_i = exp(L_i) S^T C_i + sum_{j <= i} (C_i . B_j) exp(L_i - L_j) dt_j x_j + D x_i
//     S  <- exp(L_n) S + sum_j B_j (exp(L_n - L_j) dt_j x_j)^T
// B, C and x are bf16 to begin with; every fp32 operand (decayed scores, weighted values, the carried state) is split into
// two bf16 numbers, hi + lo, and takes part as two m16n8k16 MMAs with fp32 accumulation, which keeps 16 bits of it.  The
// state itself stays in fp32 registers (the accumulator fragments of the update product), its hi / lo copy in shared memory
// is only the operand of the next chunk's C S product.
//
// One CTA = (segment of an entry, head, 64-column slice of E), two CTAs per SM.  An entry is one segment when there are
// enough entries to fill the GPU.  Otherwise it is cut into several: a first launch (state_only) computes what each
// segment adds to the state, ssm_carry_kernel chains them into the state before each segment, and the second launch runs
// all segments at once.
#include "common.cuh"
#include "host_utils.cuh"
#include "ssm.cuh"
#include "warp_mma.cuh"

namespace apb {

constexpr int kSmThreads = 256;
constexpr int kSmC = 32;                  // tokens per chunk
constexpr int kSmBE = 64;                 // E columns per CTA
constexpr int kSmVS = kSmBE + 8;          // row strides (elements): odd multiples of 16 bytes
constexpr int kSmAS = kSmC + 8;
constexpr int kSmMaxN = 128;

struct SsmSegments {
  const int* seg;         // [n][6]: entry, first token, tokens, scratch index of the state before it (-1: the slot's
                          // state or zero), scratch index for its own contribution (-1: none), 1 = last of its entry
  float* carry;           // [scratch states][H][N][E]
  float* decay;           // [n][H] log2 decay over the whole segment
};

__host__ __device__ inline int ssm_smem_bytes(int N) {
  const int np = (N + 15) / 16 * 16, ns = np + 8;
  return 2 * (3 * kSmC * ns + 4 * kSmC * kSmVS + 2 * kSmC * kSmAS + 2 * np * kSmVS);
}

// NP: N rounded up to 16 when known at compile time, else 0.
template <int NP>
__global__ void __launch_bounds__(kSmThreads, 2)
ssm_mma_kernel(const SsmParams p, const SsmSegments sg, int state_only) {
  pdl_entry();
  extern __shared__ __align__(128) uint8_t sm_smem[];
  __shared__ float s_l[2][kSmC], s_dt[2][kSmC];            // running log2 decays and step sizes of two chunks
  const int* w = sg.seg + blockIdx.x * 6;
  const int en = w[0], t_begin = w[1], n_tok = w[2], carry_in = w[3], carry_out = w[4], is_last = w[5];
  if (state_only && carry_out < 0) return;
  const int h = blockIdx.y, e0 = blockIdx.z * kSmBE, g = h / (p.H / p.G);
  const int N = p.N, E = p.E, np = NP ? NP : (N + 15) & ~15, ns = np + 8, n16 = np >> 4;
  const int be = min(kSmBE, E - e0);
  const long long start = p.e.start[en] + t_begin;
  const int pos0 = p.e.pos0[en] + t_begin, slot = p.e.slot[en];
  __nv_bfloat16* Cs = reinterpret_cast<__nv_bfloat16*>(sm_smem);
  __nv_bfloat16* B2 = Cs + kSmC * ns;            // two buffers [32][ns]
  __nv_bfloat16* V2 = B2 + 2 * kSmC * ns;        // two buffers of x [32][72]
  __nv_bfloat16* Wh = V2 + 2 * kSmC * kSmVS;     // x times its weight in the state after the chunk, hi / lo
  __nv_bfloat16* Wl = Wh + kSmC * kSmVS;
  __nv_bfloat16* Ah = Wl + kSmC * kSmVS;         // [32][40] decayed scores
  __nv_bfloat16* Al = Ah + kSmC * kSmAS;
  __nv_bfloat16* Sh = Al + kSmC * kSmAS;         // [np][72] carried state
  __nv_bfloat16* Sl = Sh + np * kSmVS;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int quad_row = lane >> 2, quad_col = (lane & 3) * 2;
  const int mat = lane >> 3, rowin = lane & 7;
  const __nv_bfloat16* xb = static_cast<const __nv_bfloat16*>(p.xbc);
  const int b_col = p.H * E + g * N, c_col = b_col + p.G * N, x_col = h * E + e0;
  const float skip = __bfloat162float(static_cast<const __nv_bfloat16*>(p.d_skip)[h]);

  // rows beyond the segment and columns beyond N are filled with zeros
  const int pc = np >> 3;                        // 16-byte pieces of a row
  auto fetch_rows = [&](int t0, int col, __nv_bfloat16* dst) {
#pragma unroll
    for (int i = threadIdx.x; i < kSmC * pc; i += kSmThreads) {
      const int r = i / pc, c = i % pc, ok = t0 + r < n_tok && c * 8 < N;
      wm_cp_async16(smem_u32(dst + r * ns + c * 8), xb + (start + (ok ? t0 + r : 0)) * p.ldx + col + (ok ? c * 8 : 0), ok ? 16 : 0);
    }
  };
  auto fetch_bx = [&](int t0, int buf) {
    fetch_rows(t0, b_col, B2 + buf * kSmC * ns);
    const int r = threadIdx.x >> 3, c = threadIdx.x & 7, ok = t0 + r < n_tok && c * 8 < be;
    wm_cp_async16(smem_u32(V2 + buf * kSmC * kSmVS + r * kSmVS + c * 8),
                   xb + (start + (ok ? t0 + r : 0)) * p.ldx + x_col + (ok ? c * 8 : 0), ok ? 16 : 0);
  };
  static_assert(kSmThreads == kSmC * kSmBE / 8 && kSmC == 32, "one 16-byte piece of x per thread, one token per lane");
  auto steps_of = [&](int t0, int buf) {         // one warp
    const float2 st = t0 + lane < n_tok ? p.steps[(start + t0 + lane) * p.H + h] : make_float2(0.f, 0.f);
    float l = st.y;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, l, o);
      if (lane >= o) l += v;
    }
    s_l[buf][lane] = l;
    s_dt[buf][lane] = st.x;
  };
  if (!state_only) fetch_rows(0, c_col, Cs);
  fetch_bx(0, 0);
  asm volatile("cp.async.commit_group;" ::: "memory");
  if (warp == 7) steps_of(0, 0);

  // the warp's 16 state rows, fp32: accumulator fragments over eight 8-column tiles
  float s[8][4];
  const float* s_in = nullptr;
  if (!state_only) {
    if (carry_in >= 0)
      s_in = sg.carry + (static_cast<long long>(carry_in) * p.H + h) * N * E;
    else if (pos0 > 0)
      s_in = p.state + (static_cast<long long>(slot) * p.H + h) * N * E;
  }
  const int sr = warp * 16 + quad_row;
  auto store_state_operand = [&]() {
    if (warp < n16) {
#pragma unroll
      for (int nt = 0; nt < 8; ++nt)
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
          uint32_t hi, lo;
          wm_split2(s[nt][2 * hh], s[nt][2 * hh + 1], hi, lo);
          const int o = (sr + 8 * hh) * kSmVS + nt * 8 + quad_col;
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
      if (s_in && d < N && c < be) v = *reinterpret_cast<const float2*>(s_in + static_cast<long long>(d) * E + e0 + c);
      s[nt][2 * hh] = v.x;
      s[nt][2 * hh + 1] = v.y;
    }
  bool have_state = s_in != nullptr;
  if (have_state) store_state_operand();
  float total = 0.f;                             // log2 decay of the segment

  for (int t0 = 0, buf = 0; t0 < n_tok; t0 += kSmC, buf ^= 1) {
    const int n = min(kSmC, n_tok - t0);
    const bool more = t0 + kSmC < n_tok;
    const __nv_bfloat16* B = B2 + buf * kSmC * ns;
    const __nv_bfloat16* V = V2 + buf * kSmC * kSmVS;
    const float* L = s_l[buf];
    const float* dt = s_dt[buf];
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                               // this chunk has landed; everybody is done with the last one
    if (more) {
      fetch_bx(t0 + kSmC, buf ^ 1);
      if (warp == 7) steps_of(t0 + kSmC, buf ^ 1);
    }
    const float l_end = L[kSmC - 1];
    total += l_end;
    for (int i = threadIdx.x; i < kSmC * (kSmBE / 2); i += kSmThreads) {
      const int r = i / (kSmBE / 2), o = r * kSmVS + (i % (kSmBE / 2)) * 2;
      const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(V + o));
      const float wt = exp2f(l_end - L[r]) * dt[r];
      uint32_t wh, wl;
      wm_split2(f.x * wt, f.y * wt, wh, wl);
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
      for (int ks = 0; ks < n16; ++ks) {
        uint32_t q[4];
        wm_ldsm4(Cs + (r0 + rowin + (mat & 1) * 8) * ns + ks * 16 + (mat >> 1) * 8, q);
        if (live) {
          uint32_t k[2];
          wm_ldsm2(B + (k0 + rowin) * ns + ks * 16 + (mat & 1) * 8, k);
          wm_mma(a, q, k[0], k[1]);
        }
        if (have_state) {                          // C S of the carried state
          uint32_t sh[4], sl[4];
          const int so = (ks * 16 + rowin + 8 * (mat & 1)) * kSmVS + c0 + (mat >> 1) * 8;
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
        const float li = L[i];
        uint32_t hi, lo;
        wm_split2(j <= i ? a[2 * hh] * exp2f(li - L[j]) * dt[j] : 0.f,
                   j + 1 <= i ? a[2 * hh + 1] * exp2f(li - L[j + 1]) * dt[j + 1] : 0.f, hi, lo);
        *reinterpret_cast<uint32_t*>(Ah + i * kSmAS + j) = hi;
        *reinterpret_cast<uint32_t*>(Al + i * kSmAS + j) = lo;
        const float f = exp2f(li);
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          o[nt][2 * hh] *= f;
          o[nt][2 * hh + 1] *= f;
        }
      }
    }
    __syncthreads();                               // scores and W visible; nobody reads C or the state operand any more
    if (more && !state_only) fetch_rows(t0 + kSmC, c_col, Cs);
    asm volatile("cp.async.commit_group;" ::: "memory");
    if (!state_only) {
      for (int ks = 0; ks < (r0 + 16) / 16; ++ks) {
        uint32_t ah[4], al[4], v[4];
        const int ao = (r0 + rowin + (mat & 1) * 8) * kSmAS + ks * 16 + (mat >> 1) * 8;
        wm_ldsm4(Ah + ao, ah);
        wm_ldsm4(Al + ao, al);
        wm_ldsm4_t(V + (ks * 16 + rowin + 8 * (mat & 1)) * kSmVS + c0 + (mat >> 1) * 8, v);
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
          float* dst = p.y + (start + t0 + i) * p.H * E + x_col;
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            const int c = c0 + nt * 8 + quad_col;
            if (c < be) {
              const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(V + i * kSmVS + c));
              *reinterpret_cast<float2*>(dst + c) = make_float2(o[nt][2 * hh] + skip * x.x, o[nt][2 * hh + 1] + skip * x.y);
            }
          }
        }
      }
    }
    // ---- S = exp(L_n) S + sum_j B_j W_j^T
    if (warp < n16) {
      const float dn = exp2f(l_end);
#pragma unroll
      for (int nt = 0; nt < 8; ++nt)
#pragma unroll
        for (int i = 0; i < 4; ++i) s[nt][i] *= dn;
#pragma unroll
      for (int ks = 0; ks < kSmC / 16; ++ks) {
        uint32_t k[4];
        wm_ldsm4_t(B + (ks * 16 + rowin + (mat >> 1) * 8) * ns + warp * 16 + (mat & 1) * 8, k);
#pragma unroll
        for (int n2 = 0; n2 < 4; ++n2) {
          uint32_t wh[4], wl[4];
          const int bo = (ks * 16 + rowin + 8 * (mat & 1)) * kSmVS + n2 * 16 + (mat >> 1) * 8;
          wm_ldsm4_t(Wh + bo, wh);
          wm_ldsm4_t(Wl + bo, wl);
#pragma unroll
          for (int q = 0; q < 2; ++q) {
            wm_mma(s[2 * n2 + q], k, wl[2 * q], wl[2 * q + 1]);
            wm_mma(s[2 * n2 + q], k, wh[2 * q], wh[2 * q + 1]);
          }
        }
      }
    }
    if (!state_only && more) store_state_operand();
    have_state = true;
  }
  // ---- the state after the segment
  float* s_out = state_only ? sg.carry + (static_cast<long long>(carry_out) * p.H + h) * N * E
                            : (is_last ? p.state + (static_cast<long long>(slot) * p.H + h) * N * E : nullptr);
  if (s_out && warp < n16) {
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        const int d = sr + 8 * hh, c = nt * 8 + quad_col;
        if (d < N && c < be)
          *reinterpret_cast<float2*>(s_out + static_cast<long long>(d) * E + e0 + c) = make_float2(s[nt][2 * hh], s[nt][2 * hh + 1]);
      }
  }
  if (state_only && e0 == 0 && threadIdx.x == 0) sg.decay[static_cast<long long>(blockIdx.x) * p.H + h] = total;
}

// Chains the contributions of an entry's segments: scratch[base] becomes the state before the entry, scratch[base + i]
// the state before its i-th segment.  chains [n][4]: entry, base, segments, index of its first segment.
__global__ void __launch_bounds__(256)
ssm_carry_kernel(const SsmParams p, const SsmSegments sg, const int* __restrict__ chains) {
  pdl_entry();
  const int* c = chains + blockIdx.x * 4;
  const int en = c[0], base = c[1], n_seg = c[2], first = c[3], h = blockIdx.y;
  const int size = p.N * p.E;
  const int i = blockIdx.z * 256 + threadIdx.x;
  if (i >= size) return;
  const long long stride = static_cast<long long>(p.H) * size;
  float* x = sg.carry + static_cast<long long>(base) * stride + static_cast<long long>(h) * size + i;
  float s = p.e.pos0[en] > 0 ? p.state[static_cast<long long>(p.e.slot[en]) * stride + static_cast<long long>(h) * size + i] : 0.f;
  x[0] = s;
  for (int k = 0; k + 1 < n_seg; ++k) {
    s = s * exp2f(sg.decay[static_cast<long long>(first + k) * p.H + h]) + x[(k + 1) * stride];
    x[(k + 1) * stride] = s;
  }
}

}  // namespace apb

extern "C" {
using namespace apb;

// bf16; N a multiple of 8 up to 128, E a multiple of 8; xbc [rows, ldx] and steps [rows, H] as apb_ssm leaves them, ldx a
// multiple of 8.  Writes y [rows, H * E] for the segments' rows and the entries' states.  n_chains > 0: some entries have
// several segments (carry is scratch for their states, decay [n_seg, H] for their decays).
int apb_ssm_mma(const void* xbc, long long ldx, const void* steps, const void* d_skip, float* state, float* y,
                const int* e_start, const int* e_len, const int* e_slot, const int* e_pos0, const int* seg, int n_seg,
                float* carry, float* decay, const int* chains, int n_chains, int H, int E, int G, int N, cudaStream_t s) {
  if (n_seg <= 0) return 0;
  if (H <= 0 || E <= 0 || G <= 0 || N <= 0 || H % G || (N % 8) || (E % 8) || N > kSmMaxN || (ldx % 8) ||
      (reinterpret_cast<uintptr_t>(xbc) & 15) || !seg || !y || !state || !steps || (n_chains > 0 && (!carry || !chains || !decay)))
    return kBadArgument;
  SsmParams a{};
  a.e = ServeEntries{e_start, e_len, e_slot, e_pos0};
  a.xbc = const_cast<void*>(xbc);
  a.ldx = ldx;
  a.steps = static_cast<float2*>(const_cast<void*>(steps));
  a.d_skip = d_skip;
  a.state = state;
  a.y = y;
  a.H = H;
  a.E = E;
  a.G = G;
  a.N = N;
  const SsmSegments sg{seg, carry, decay};
  const int smem = ssm_smem_bytes(N), np = (N + 15) / 16 * 16;
  const dim3 grid(n_seg, H, (E + kSmBE - 1) / kSmBE);
  auto run = [&](auto fn) -> cudaError_t {
    cudaError_t r = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (r != cudaSuccess) return r;
    if (n_chains > 0) {
      r = launch_kernel(fn, grid, dim3(kSmThreads), smem, s, a, sg, 1);
      if (r != cudaSuccess) return r;
      r = launch_kernel(ssm_carry_kernel, dim3(n_chains, H, (N * E + 255) / 256), dim3(256), 0, s, a, sg, chains);
      if (r != cudaSuccess) return r;
    }
    return launch_kernel(fn, grid, dim3(kSmThreads), smem, s, a, sg, 0);
  };
  return static_cast<int>(np == 128 ? run(ssm_mma_kernel<128>) : np == 64 ? run(ssm_mma_kernel<64>) : run(ssm_mma_kernel<0>));
}
}
