// Paged causal softmax attention for ragged serving batches: optional score cap, optional chunks (a query sees its own
// chunk of positions only) and sliding windows, sinks, output gates, one or two maps per head (differential attention).  See
// SoftmaxSpec.
//
// Keys and values live in pages of 16 tokens (kcache [pages, G, 16, maps * D], vcache [pages, G, 16, E]; the first kernel also
// takes no vcache: the values are then the first E columns of the key rows); the step's own keys are already there when these
// kernels run, so prompts, portions of prompts and decoded tokens read the same memory.
//
//  * softmax_attn_kernel      any D up to 1024, E up to 512, bf16 or fp32, fp32 arithmetic throughout (the fp32 engine, odd sizes);
//  * softmax_attn_mma_kernel  bf16, D and E multiples of 8, maps * D and E up to 256: m16n8k16 tensor-core tiles whose 16
//                             rows are (query, head of one KV head, map) triples -- decoded tokens and short portions.  A
//                             row's query is zero in the columns of the other map, so one product with the whole cache row
//                             serves both maps.  The key range can be split over CTAs (softmax_merge_kernel).
//
// Long portions run on tcgen05 (serve_softmax_tc.cu).
#include "common.cuh"
#include "host_utils.cuh"
#include "serve_softmax_mma.cuh"

namespace apb {

constexpr int kSoftThreads = 128;

// One CTA per (row, query head); its four warps take every fourth run of 32 keys.
template <typename T, int NV, int MAPS>
__global__ void __launch_bounds__(kSoftThreads)
softmax_attn_kernel(const T* __restrict__ q, long long ldq, const int* __restrict__ row_entry, const ServeEntries e,
                    const int* __restrict__ page_table, int max_pages, const T* __restrict__ kcache,
                    const T* __restrict__ vcache, int v_row, T* __restrict__ out, long long ldo, int H, int G, int D, int E,
                    const SoftmaxSpec sp) {
  pdl_entry();
  extern __shared__ float sx_smem[];
  float* qs = sx_smem;                      // [MAPS * D]
  float* red = sx_smem + MAPS * D;          // [4][MAPS][E]
  __shared__ float ml[4][MAPS][2], part[4];
  const int row = blockIdx.x, h = blockIdx.y, g = h / (H / G);
  const int en = row_entry ? row_entry[row] : row;
  const int r = row - e.start[en];
  if (r < 0 || r >= e.len[en]) return;
  const int pos = e.pos0[en] + r;
  const int* pages = page_table + static_cast<long long>(en) * max_pages;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int i = threadIdx.x; i < MAPS * D; i += kSoftThreads)
    qs[i] = to_f32(q[static_cast<long long>(row) * ldq + static_cast<long long>(h) * MAPS * D + i]);
  __syncthreads();
  float acc[MAPS][NV], m[MAPS], l[MAPS];
#pragma unroll
  for (int a = 0; a < MAPS; ++a) {
    m[a] = -INFINITY;
    l[a] = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) acc[a][i] = 0.f;
  }
  for (int k0 = visible_begin(pos, sp) + warp * 32; k0 <= pos; k0 += 128) {
    const int key = k0 + lane;
    float p[MAPS];
    long long tok = 0;                      // (page, kv head, offset) row of the key
    if (key <= pos) tok = (static_cast<long long>(pages[key / kServePage]) * G + g) * kServePage + key % kServePage;
#pragma unroll
    for (int a = 0; a < MAPS; ++a) {
      float s = -INFINITY;
      if (key <= pos) {
        const T* kp = kcache + (tok * MAPS + a) * D;
        s = 0.f;
        for (int d = 0; d < D; ++d) s += qs[a * D + d] * to_f32(kp[d]);
        s *= sp.scale;
        if (sp.cap > 0.f) s = sp.cap * tanhf(s / sp.cap);
      }
      const float mn = fmaxf(m[a], warp_max(s));          // lane 0's key is visible: finite
      const float f = expf(m[a] - mn);
      p[a] = expf(s - mn);
      l[a] = l[a] * f + warp_sum(p[a]);
      m[a] = mn;
#pragma unroll
      for (int i = 0; i < NV; ++i) acc[a][i] *= f;
    }
    const int n = min(32, pos + 1 - k0);
    for (int j = 0; j < n; ++j) {
      const T* vp = vcache + __shfl_sync(0xffffffffu, tok, j) * v_row;
      float pj[MAPS];
#pragma unroll
      for (int a = 0; a < MAPS; ++a) pj[a] = __shfl_sync(0xffffffffu, p[a], j);
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (i * 32 + lane < E) {
          const float v = to_f32(vp[i * 32 + lane]);
#pragma unroll
          for (int a = 0; a < MAPS; ++a) acc[a][i] += pj[a] * v;
        }
    }
  }
#pragma unroll
  for (int a = 0; a < MAPS; ++a) {
    if (lane == 0) {
      ml[warp][a][0] = m[a];
      ml[warp][a][1] = l[a];
    }
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (i * 32 + lane < E) red[(warp * MAPS + a) * E + i * 32 + lane] = acc[a][i];
  }
  __syncthreads();
  float f[4][MAPS];                         // weight of every warp's part
#pragma unroll
  for (int a = 0; a < MAPS; ++a) {
    float mx = -INFINITY, sum = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) mx = fmaxf(mx, ml[w][a][0]);
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      f[w][a] = ml[w][a][1] > 0.f ? expf(ml[w][a][0] - mx) : 0.f;
      sum += f[w][a] * ml[w][a][1];
    }
    const float inv = inverse_sum(sp, h, mx * 1.4426950408889634f, sum);
#pragma unroll
    for (int w = 0; w < 4; ++w) f[w][a] *= inv;
  }
  const float lam = MAPS == 2 ? *sp.lambda : 0.f;
  float ss = 0.f;
  for (int i = threadIdx.x; i < E; i += kSoftThreads) {
    float o[MAPS];
#pragma unroll
    for (int a = 0; a < MAPS; ++a) {
      o[a] = 0.f;
#pragma unroll
      for (int w = 0; w < 4; ++w)
        if (f[w][a] > 0.f) o[a] += f[w][a] * red[(w * MAPS + a) * E + i];
    }
    if (MAPS == 2) o[0] -= lam * o[MAPS - 1];
    red[i] = o[0];                          // element i of every part was read by this thread only
    ss += o[0] * o[0];
  }
  T* dst = out + static_cast<long long>(row) * ldo + static_cast<long long>(h) * E;
  float post = 1.f;
  if (MAPS == 2) {
    ss = warp_sum(ss);
    if (lane == 0) part[warp] = ss;
    __syncthreads();
    post = sp.post_scale / sqrtf((part[0] + part[1] + part[2] + part[3]) / E + sp.eps);
  }
  for (int i = threadIdx.x; i < E; i += kSoftThreads) dst[i] = from_f32<T>(red[i] * post * output_gate<T>(sp, row, h, i));
}

// ---------------------------------------------------------------------------- tensor-core tiles for few queries
// One CTA = (entry, KV head, key split, pass group); a pass is 16 consecutive rows f of the entry: row f is map f % M of
// head (f / M) % R of query f / (M R), with R query heads per KV head.  Each of the four warps owns every fourth page of
// the split's range, copies K and V pages with cp.async into its own 3-deep ring and runs S = Q K^T, O += exp(S) V as
// m16n8k16 MMAs; the warps' sums are combined at the end.  Ring rows are an odd multiple of 16 bytes apart, so the 8 rows of
// an ldmatrix tile fall into different banks.
constexpr int kSxStages = 3;

// NK, NE: upper bounds of maps * D / 16 and E / 16; FULL: both are equal to them (constant index arithmetic).
// RUNNING: keep a running maximum (no score cap, or a large one); otherwise the scores' reference is fixed.
template <int NK, int NE, bool FULL, bool RUNNING>
__global__ void __launch_bounds__(kSoftThreads)
softmax_attn_mma_kernel(const SoftmaxMmaParams p) {
  pdl_entry();
  extern __shared__ __align__(128) uint8_t sx_ring[];
  const int en = blockIdx.x / p.G, g = blockIdx.x % p.G;
  const int len = p.e.len[en];
  if (len < p.min_len || len > p.max_len) return;
  const int M = p.sp.maps;
  const int DK = FULL ? NK * 16 : p.D * M, E = FULL ? NE * 16 : p.E, R = p.H / p.G, D = p.D;
  const int d16 = (DK + 15) >> 4, e16 = (E + 15) >> 4;
  const int k_row = d16 * 32 + 16, v_row = e16 * 32 + 16;            // ring row bytes
  const int stage_bytes = kServePage * (k_row + v_row);
  const int split = blockIdx.y, splits = gridDim.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int start = p.e.start[en], pos0 = p.e.pos0[en];
  const int* pages = p.page_table + static_cast<long long>(en) * p.max_pages;
  uint8_t* my_ring = sx_ring + warp * (kSxStages * stage_bytes);
  const uint32_t ring = smem_u32(my_ring);
  const int quad_row = lane >> 2, quad_col = (lane & 3) * 2;
  const int mat = lane >> 3, rowin = lane & 7;
  const int kc = DK >> 3, vc = E >> 3;                               // 16-byte chunks of a cache row
  const int n_rows = len * R * M;
  constexpr float kLog2e = 1.4426950408889634f;
  const float cap = p.sp.cap, inv_cap = cap > 0.f ? p.sp.scale / cap : 0.f;
  const float gain = (cap > 0.f ? cap : p.sp.scale) * kLog2e, ref = score_reference(cap) * kLog2e;
  __shared__ float s_ml[4][16][2];

  for (int f0 = blockIdx.z * 16; f0 < n_rows; f0 += gridDim.z * 16) {
    const int q_first = f0 / (R * M), q_last = (min(f0 + 16, n_rows) - 1) / (R * M);
    const int page_lo = visible_begin(pos0 + q_first, p.sp) / kServePage;
    const int n_pages = (pos0 + q_last + kServePage) / kServePage;   // pages up to the last query of the pass
    const int per = (n_pages - page_lo + splits - 1) / splits;
    const int p0 = page_lo + split * per, p1 = min(n_pages, p0 + per);
    const int n_my = p1 > p0 + warp ? (p1 - p0 - warp + 3) / 4 : 0;
    // the half chunk that pads the row to a multiple of 16 takes part in the products: zero it (copies never touch it)
    if (DK & 8)
      for (int i = lane; i < kSxStages * kServePage; i += 32)
        *reinterpret_cast<uint4*>(my_ring + (i / kServePage) * stage_bytes + (i % kServePage) * k_row + DK * 2) = make_uint4(0, 0, 0, 0);
    uint32_t qa[NK][4];
    int hi[2], lo[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int f = f0 + quad_row + 8 * h;
      const bool ok = f < n_rows;
      const int map = ok ? f % M : 0, qi = ok ? f / (R * M) : 0, head = g * R + (ok ? f / M % R : 0);
      hi[h] = ok ? pos0 + qi : -1;
      lo[h] = visible_begin(pos0 + qi, p.sp);
      const __nv_bfloat16* qp = p.q + static_cast<long long>(start + qi) * p.ldq + static_cast<long long>(head) * DK;
      const int d_lo = map * D, d_hi = d_lo + D;
#pragma unroll
      for (int ks = 0; ks < NK; ++ks) {
        const int c0 = ks * 16 + quad_col;
        qa[ks][h] = (ok && c0 >= d_lo && c0 < d_hi) ? *reinterpret_cast<const uint32_t*>(qp + c0) : 0u;
        qa[ks][2 + h] = (ok && c0 + 8 >= d_lo && c0 + 8 < d_hi) ? *reinterpret_cast<const uint32_t*>(qp + c0 + 8) : 0u;
      }
    }
    float o[2 * NE][4], m[2], l[2];
#pragma unroll
    for (int i = 0; i < 2 * NE; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    l[0] = l[1] = 0.f;
    m[0] = m[1] = RUNNING ? -INFINITY : ref;

    auto issue = [&](int j) {
      if (j < n_my) {
        const long long base = (static_cast<long long>(pages[p0 + warp + 4 * j]) * p.G + g) * kServePage;
        const uint32_t dst = ring + (j % kSxStages) * stage_bytes;
        const __nv_bfloat16* kp = p.kcache + base * DK;
#pragma unroll
        for (int i = lane; i < kServePage * kc; i += 32) sx_cp_async16(dst + (i / kc) * k_row + (i % kc) * 16, kp + i * 8);
        const __nv_bfloat16* vp = p.vcache + base * E;
#pragma unroll
        for (int i = lane; i < kServePage * vc; i += 32)
          sx_cp_async16(dst + kServePage * k_row + (i / vc) * v_row + (i % vc) * 16, vp + i * 8);
      }
      asm volatile("cp.async.commit_group;" ::: "memory");
    };
#pragma unroll
    for (int j = 0; j < kSxStages - 1; ++j) issue(j);
#pragma unroll 1
    for (int j = 0; j < n_my; ++j) {
      issue(j + kSxStages - 1);
      asm volatile("cp.async.wait_group %0;" ::"n"(kSxStages - 1) : "memory");
      __syncwarp();
      const uint32_t ks_addr = ring + (j % kSxStages) * stage_bytes;
      const uint32_t vs_addr = ks_addr + kServePage * k_row;
      float sc[2][4];
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) sc[nt][0] = sc[nt][1] = sc[nt][2] = sc[nt][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < NK; ++ks)
        if (ks < d16) {
          uint32_t r[4];
          sx_ldsm_x4(ks_addr + (rowin + 8 * (mat >> 1)) * k_row + (ks * 2 + (mat & 1)) * 16, r);
          sx_mma(sc[0], qa[ks], r[0], r[1]);
          sx_mma(sc[1], qa[ks], r[2], r[3]);
        }
      const int key = (p0 + warp + 4 * j) * kServePage + quad_col;
      uint32_t pa[4];
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        float w[4];                                      // scores in units of log 2
        bool seen[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float s = sc[i >> 1][2 * h + (i & 1)];
          const int k = key + (i >> 1) * 8 + (i & 1);
          seen[i] = k <= hi[h] && k >= lo[h];
          w[i] = (cap > 0.f ? tanh_any(s * inv_cap) : s) * gain;
        }
        if (RUNNING) {
          float mx = m[h];
#pragma unroll
          for (int i = 0; i < 4; ++i) mx = seen[i] ? fmaxf(mx, w[i]) : mx;
          mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
          mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
          if (mx > m[h]) {
            const float f = exp2f(m[h] - mx);            // 0 on the first visible key
            l[h] *= f;
#pragma unroll
            for (int i = 0; i < 2 * NE; ++i) {
              o[i][2 * h] *= f;
              o[i][2 * h + 1] *= f;
            }
            m[h] = mx;
          }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          w[i] = seen[i] ? exp2f(w[i] - m[h]) : 0.f;
          l[h] += w[i];
        }
        pa[h] = pack_bf16x2(w[0], w[1]);
        pa[2 + h] = pack_bf16x2(w[2], w[3]);
      }
#pragma unroll
      for (int dp = 0; dp < NE; ++dp)
        if (dp < e16) {
          uint32_t r[4];
          sx_ldsm_x4_t(vs_addr + (rowin + 8 * (mat & 1)) * v_row + (dp * 2 + (mat >> 1)) * 16, r);
          sx_mma(o[2 * dp], pa, r[0], r[1]);
          sx_mma(o[2 * dp + 1], pa, r[2], r[3]);
        }
      __syncwarp();
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
      l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
    }
    __syncthreads();                                   // every warp is done with its ring: reuse it for the sums
    float* red = reinterpret_cast<float*>(sx_ring);    // [4][16][e16 * 16]
    const int ew = e16 * 16;
#pragma unroll
    for (int i = 0; i < 2 * NE; ++i)
      if (i < 2 * e16) {
#pragma unroll
        for (int h = 0; h < 2; ++h)
          *reinterpret_cast<float2*>(&red[(warp * 16 + quad_row + 8 * h) * ew + i * 8 + quad_col]) =
              make_float2(o[i][2 * h], o[i][2 * h + 1]);
      }
    if ((lane & 3) == 0) {
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        s_ml[warp][quad_row + 8 * h][0] = m[h];
        s_ml[warp][quad_row + 8 * h][1] = l[h];
      }
    }
    __syncthreads();
    const int rows_valid = min(16, n_rows - f0);
    for (int rr = warp * M; rr < rows_valid; rr += 4 * M) {            // one warp per (query, head); maps are neighbours
      float f[2][4], mx[2], sum[2];
#pragma unroll
      for (int a = 0; a < 2; ++a) {
        mx[a] = -INFINITY;
        sum[a] = 0.f;
        if (a < M) {
#pragma unroll
          for (int w = 0; w < 4; ++w)
            if (s_ml[w][rr + a][1] > 0.f) mx[a] = fmaxf(mx[a], s_ml[w][rr + a][0]);
#pragma unroll
          for (int w = 0; w < 4; ++w) {
            f[a][w] = s_ml[w][rr + a][1] > 0.f ? exp2f(s_ml[w][rr + a][0] - mx[a]) : 0.f;
            sum[a] += f[a][w] * s_ml[w][rr + a][1];
          }
        }
      }
      auto total = [&](int a, int c) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) v += (a ? f[1][w] : f[0][w]) * red[(w * 16 + rr + a) * ew + c];
        return v;
      };
      const int qi = (f0 + rr) / (R * M), head = g * R + (f0 + rr) / M % R;
      if (splits > 1) {
        for (int a = 0; a < M; ++a) {
          float* dst = p.part + ((((static_cast<long long>(en) * p.max_len + qi) * p.H + head) * M + a) * splits + split) * (E + 2);
          for (int c = lane; c < E; c += 32) dst[c] = total(a, c);
          if (lane == 0) {
            dst[E] = a ? mx[1] : mx[0];
            dst[E + 1] = a ? sum[1] : sum[0];
          }
        }
      } else {
        const float i0 = inverse_sum(p.sp, head, mx[0], sum[0]), i1 = M == 2 ? 1.f / sum[1] : 0.f;
        softmax_finish(p.sp, E, start + qi, head, p.out + static_cast<long long>(start + qi) * p.ldo + static_cast<long long>(head) * E, lane,
                       [&](int a, int c) { return total(a, c) * (a ? i1 : i0); });
      }
    }
    __syncthreads();                                   // the ring is written again by the next pass
  }
}

// Combines the key splits of the rows handled by the kernel above.  One warp per (entry, query, head).
__global__ void __launch_bounds__(256)
softmax_merge_kernel(const SoftmaxMmaParams p, int n_entries, int splits) {
  pdl_entry();
  const int lane = threadIdx.x & 31;
  const long long gw = (blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x) >> 5;
  if (gw >= static_cast<long long>(n_entries) * p.max_len * p.H) return;
  const int head = static_cast<int>(gw % p.H), qi = static_cast<int>(gw / p.H % p.max_len);
  const int en = static_cast<int>(gw / p.H / p.max_len), len = p.e.len[en];
  if (len < p.min_len || len > p.max_len || qi >= len) return;
  const int M = p.sp.maps, E = p.E;
  const float* src = p.part + gw * M * splits * (E + 2);
  float mx[2] = {-INFINITY, -INFINITY}, inv[2] = {0.f, 0.f};
#pragma unroll
  for (int a = 0; a < 2; ++a) {
    if (a >= M) break;
    const float* s = src + a * splits * (E + 2);
    for (int i = 0; i < splits; ++i)
      if (s[i * (E + 2) + E + 1] > 0.f) mx[a] = fmaxf(mx[a], s[i * (E + 2) + E]);
    float sum = 0.f;
    for (int i = 0; i < splits; ++i)
      if (s[i * (E + 2) + E + 1] > 0.f) sum += exp2f(s[i * (E + 2) + E] - mx[a]) * s[i * (E + 2) + E + 1];
    inv[a] = inverse_sum(p.sp, head, mx[a], sum);
  }
  softmax_finish(p.sp, E, p.e.start[en] + qi, head, p.out + static_cast<long long>(p.e.start[en] + qi) * p.ldo + static_cast<long long>(head) * E, lane,
                 [&](int a, int c) {
                   const float* s = src + a * splits * (E + 2);
                   const float top = a ? mx[1] : mx[0];
                   float v = 0.f;
                   for (int i = 0; i < splits; ++i)
                     if (s[i * (E + 2) + E + 1] > 0.f) v += exp2f(s[i * (E + 2) + E] - top) * s[i * (E + 2) + c];
                   return v * (a ? inv[1] : inv[0]);
                 });
}

int launch_softmax_merge(const SoftmaxMmaParams& p, int n_entries, int splits, cudaStream_t s) {
  const long long warps = static_cast<long long>(n_entries) * p.max_len * p.H;
  return static_cast<int>(launch_kernel(softmax_merge_kernel, dim3(static_cast<unsigned>((warps + 7) / 8)), dim3(256), 0, s, p,
                                        n_entries, splits));
}

}  // namespace apb

extern "C" {
using namespace apb;

// q [rows, H * maps * D] (row stride ldq, already rotated), out [rows, H * E] (row stride ldo).
// page_table [entries, max_pages]; row_entry [rows] or null (row i belongs to entry i).
int apb_softmax_attn(const void* q, long long ldq, const int* row_entry, const int* e_start, const int* e_len,
                     const int* e_slot, const int* e_pos0, const int* page_table, int max_pages, const void* kcache,
                     const void* vcache, void* out, long long ldo, int rows, int H, int G, int D, int E, float scale,
                     float cap, int chunk, int maps, const float* lambda, float post_scale, float eps, int window,
                     const float* sink, const void* gate, long long ldg, int gate_cols, int dtype, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || D <= 0 || E <= 0 || D > 1024 || E > 512 || maps < 1 || maps > 2 || (maps == 2 && !lambda) ||
      chunk < 0 || window < 0 || (maps == 2 && (sink || gate)) || (!vcache && E > maps * D) ||
      (gate && gate_cols != 1 && gate_cols != E))
    return kBadArgument;
  const int v_row = vcache ? E : maps * D;
  if (!vcache) vcache = kcache;
  const ServeEntries e{e_start, e_len, e_slot, e_pos0};
  const SoftmaxSpec sp{scale, cap, chunk, maps, lambda, post_scale, eps, window, sink, gate, ldg, gate_cols};
  const size_t smem = maps * (D + 4 * E) * sizeof(float);              // at most 24 KB
#define APB_SX(NVV, MM)                                                                                              \
  return static_cast<int>(launch_kernel(softmax_attn_kernel<T, NVV, MM>, dim3(rows, H), dim3(kSoftThreads), smem, s, \
                                        static_cast<const T*>(q), ldq, row_entry, e, page_table, max_pages,          \
                                        static_cast<const T*>(kcache), static_cast<const T*>(vcache), v_row,         \
                                        static_cast<T*>(out), ldo, H, G, D, E, sp))
  APB_SERVE_DTYPE(dtype, if (maps == 2 && E <= 128) APB_SX(4, 2); if (maps == 2) APB_SX(16, 2);
                  if (E <= 128) APB_SX(4, 1); APB_SX(16, 1));
#undef APB_SX
}

// bf16, D and E multiples of 8, maps * D and E up to 256; entries of min_len .. max_len rows (max_len: also the bound of the
// grid).  part: fp32 scratch [entries, max_len, H, maps, splits, E + 2] when splits > 1.
int apb_softmax_attn_mma(const void* q, long long ldq, const int* e_start, const int* e_len, const int* e_slot,
                         const int* e_pos0, int n_entries, const int* page_table, int max_pages, const void* kcache,
                         const void* vcache, void* out, long long ldo, float* part, int H, int G, int D, int E, int min_len,
                         int max_len, int splits, float scale, float cap, int chunk, int maps, const float* lambda,
                         float post_scale, float eps, int window, const float* sink, const void* gate, long long ldg,
                         int gate_cols, cudaStream_t s) {
  if (n_entries <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || D <= 0 || E <= 0 || (D % 8) || (E % 8) || maps < 1 || maps > 2 || maps * D > 256 || E > 256 ||
      (ldq % 8) || (reinterpret_cast<uintptr_t>(q) & 15) || min_len < 1 || max_len < min_len || splits < 1 ||
      (splits > 1 && !part) || (maps == 2 && !lambda) || chunk < 0 || window < 0 || (maps == 2 && (sink || gate)) ||
      !vcache || (gate && gate_cols != 1 && gate_cols != E))
    return kBadArgument;
  SoftmaxMmaParams p{static_cast<const __nv_bfloat16*>(q), ldq, ServeEntries{e_start, e_len, e_slot, e_pos0}, page_table,
                     max_pages, static_cast<const __nv_bfloat16*>(kcache), static_cast<const __nv_bfloat16*>(vcache),
                     static_cast<__nv_bfloat16*>(out), ldo, part, H, G, D, E, min_len, max_len,
                     SoftmaxSpec{scale, cap, chunk, maps, lambda, post_scale, eps, window, sink, gate, ldg, gate_cols}};
  const int DK = maps * D, d16 = (DK + 15) / 16, e16 = (E + 15) / 16;
  const int ring = 4 * kSxStages * kServePage * (d16 * 32 + e16 * 32 + 32), sums = 4 * 16 * e16 * 16 * 4;
  const int smem = ring > sums ? ring : sums;
  const int passes = static_cast<int>((static_cast<long long>(max_len) * (H / G) * maps + 15) / 16);
  const dim3 grid(n_entries * G, splits, passes < 256 ? passes : 256);
  auto run = [&](auto fn) -> int {
    if (smem > 46 * 1024) {                  // the default limit counts the static arrays too
      const cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
      if (e != cudaSuccess) return static_cast<int>(e);
    }
    return static_cast<int>(launch_kernel(fn, grid, dim3(kSoftThreads), smem, s, p));
  };
  const bool same = DK == E, fixed = fixed_reference(cap);
  const int n16 = d16 > e16 ? d16 : e16;
  int rc;
  if (fixed && same && E == 128)
    rc = run(softmax_attn_mma_kernel<8, 8, true, false>);
  else if (fixed && same && E == 64)
    rc = run(softmax_attn_mma_kernel<4, 4, true, false>);
  else if (fixed)
    rc = n16 <= 4 ? run(softmax_attn_mma_kernel<4, 4, false, false>)
         : n16 <= 8 ? run(softmax_attn_mma_kernel<8, 8, false, false>) : run(softmax_attn_mma_kernel<16, 16, false, false>);
  else
    rc = n16 <= 4 ? run(softmax_attn_mma_kernel<4, 4, false, true>)
         : n16 <= 8 ? run(softmax_attn_mma_kernel<8, 8, false, true>) : run(softmax_attn_mma_kernel<16, 16, false, true>);
  if (rc || splits == 1) return rc;
  return launch_softmax_merge(p, n_entries, splits, s);
}
}
