// Routing of a mixture of experts in a serving step, without a host round trip.
//
//   scores = softmax(logits), or sigmoid(logits), over N experts, the last of which may be identity experts (their output is the
//   input);
//   the `top` experts with the largest scores + correction are chosen, their weights are the scores without it.
//
// moe_serve_route_kernel: one warp per row chooses, blocks count the rows of every expert, and the last block to finish turns
// the counts into first rows and into the tile tables of the two grouped products.  moe_serve_gather_kernel copies every row
// to the rows of its experts, the scaled form multiplied by its weight (experts that weigh their input).  Where a row lands inside its expert does not matter: rows of a product do not mix.
#include "common.cuh"
#include "host_utils.cuh"
#include "serve_common.cuh"

namespace apb {

constexpr int kMoeThreads = 256;
constexpr int kMoeWarps = kMoeThreads / 32;
constexpr int kMoePerLane = 16;                      // up to 512 experts
constexpr int kMoeMax = 32 * kMoePerLane;

struct MoeRouteParams {
  const float* logits;     // [rows, ld]
  long long ld;
  const void* correction;  // [N] activation type or null
  const int* live;         // [rows] or null: rows with a negative entry take no expert
  int sigmoid;             // scores are sigmoids of the logits (0: their softmax)
  int rows, N, E, top;     // E routed experts in front of N - E identity experts
  int* expert;             // [rows, top] routed expert, -1: none
  int* rank;               // [rows, top] row inside the expert
  float* weight;           // [rows, top]
  float* ident;            // [rows] sum of the identity experts' weights
  int* counters;           // [E + 1] zero between launches
  int* first;              // [E] first row of every expert
  int4* tiles1;            // {first row, end row, first row of the expert's weights, column tile}
  int4* tiles2;
  int* n_tiles;            // [2]
  int n_out1, n_out2, tile;
};

template <typename T>
__global__ void __launch_bounds__(kMoeThreads)
moe_serve_route_kernel(const MoeRouteParams p) {
  pdl_entry();
  __shared__ int hist[kMoeMax], base[kMoeMax];
  __shared__ int is_last;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int e = threadIdx.x; e < p.E; e += kMoeThreads) hist[e] = 0;
  __syncthreads();
  const int row = blockIdx.x * kMoeWarps + warp;
  const bool live = row < p.rows && (!p.live || p.live[row] >= 0);
  int mine = -1, my_rank = 0;                        // lane r: choice r
  float my_weight = 0.f, ident = 0.f;
  if (live) {
    const float* z = p.logits + static_cast<long long>(row) * p.ld;
    float sc[kMoePerLane], pick[kMoePerLane], mx = -INFINITY;
#pragma unroll
    for (int j = 0; j < kMoePerLane; ++j) {
      const int e = lane + 32 * j;
      sc[j] = e < p.N ? z[e] : -INFINITY;
      mx = fmaxf(mx, sc[j]);
    }
    if (p.sigmoid) {
#pragma unroll
      for (int j = 0; j < kMoePerLane; ++j) {
        pick[j] = sc[j];                             // without a correction the logits order the scores, also where those round to 1
        sc[j] = 1.f / (1.f + expf(-sc[j]));
      }
    } else {
      mx = warp_max(mx);
      float sum = 0.f;
#pragma unroll
      for (int j = 0; j < kMoePerLane; ++j) {
        sc[j] = lane + 32 * j < p.N ? expf(sc[j] - mx) : 0.f;
        sum += sc[j];
      }
      sum = warp_sum(sum);
#pragma unroll
      for (int j = 0; j < kMoePerLane; ++j) sc[j] /= sum;
    }
#pragma unroll
    for (int j = 0; j < kMoePerLane; ++j) {
      const int e = lane + 32 * j;
      if (e >= p.N)
        pick[j] = -INFINITY;
      else if (p.correction || !p.sigmoid)
        pick[j] = sc[j] + (p.correction ? to_f32(static_cast<const T*>(p.correction)[e]) : 0.f);
    }
    for (int r = 0; r < p.top; ++r) {
      float best = -INFINITY, w = 0.f;
      int be = kMoeMax;
#pragma unroll
      for (int j = 0; j < kMoePerLane; ++j)
        if (pick[j] > best) {                        // ascending: the first of equals
          best = pick[j];
          be = lane + 32 * j;
          w = sc[j];
        }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ob = __shfl_xor_sync(0xffffffffu, best, o), ow = __shfl_xor_sync(0xffffffffu, w, o);
        const int oe = __shfl_xor_sync(0xffffffffu, be, o);
        if (ob > best || (ob == best && oe < be)) {
          best = ob;
          be = oe;
          w = ow;
        }
      }
      if (be >= p.N) break;                          // not a number: no expert
#pragma unroll
      for (int j = 0; j < kMoePerLane; ++j)
        if (lane + 32 * j == be) pick[j] = -INFINITY;
      if (be >= p.E) {
        ident += w;
      } else if (lane == r) {
        mine = be;
        my_weight = w;
      }
    }
    if (mine >= 0) my_rank = atomicAdd(&hist[mine], 1);
  }
  __syncthreads();
  for (int e = threadIdx.x; e < p.E; e += kMoeThreads) base[e] = hist[e] ? atomicAdd(p.counters + e, hist[e]) : 0;
  __syncthreads();
  if (row < p.rows) {
    if (lane < p.top) {
      const long long o = static_cast<long long>(row) * p.top + lane;
      p.expert[o] = mine;
      p.rank[o] = mine >= 0 ? base[mine] + my_rank : 0;
      p.weight[o] = my_weight;
    }
    if (lane == 0) p.ident[row] = ident;
  }
  // ---------------------------------------------------------------- the last block: first rows and tile tables
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) is_last = atomicAdd(p.counters + p.E, 1) == static_cast<int>(gridDim.x) - 1;
  __syncthreads();
  if (!is_last) return;
  __threadfence();
  __shared__ int blk[kMoeMax];
  for (int e = threadIdx.x; e < p.E; e += kMoeThreads) {
    const int n = __ldcg(p.counters + e);
    hist[e] = n;                                     // rows, then first row
    blk[e] = (n + p.tile - 1) / p.tile;              // row blocks, then first row block
    p.counters[e] = 0;
  }
  if (threadIdx.x == 0) p.counters[p.E] = 0;
  __syncthreads();
  if (warp == 0) {                                   // exclusive sums, 32 experts at a time
    int at = 0, bat = 0;
    for (int e0 = 0; e0 < p.E; e0 += 32) {
      const int e = e0 + lane;
      const int n = e < p.E ? hist[e] : 0, m = e < p.E ? blk[e] : 0;
      int a = n, b = m;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int ua = __shfl_up_sync(0xffffffffu, a, o), ub = __shfl_up_sync(0xffffffffu, b, o);
        if (lane >= o) a += ua, b += ub;
      }
      if (e < p.E) {
        base[e] = n;
        hist[e] = at + a - n;
        blk[e] = bat + b - m;
        p.first[e] = at + a - n;
      }
      at += __shfl_sync(0xffffffffu, a, 31);
      bat += __shfl_sync(0xffffffffu, b, 31);
    }
    if (lane < 2) p.n_tiles[lane] = bat * (((lane ? p.n_out2 : p.n_out1) + p.tile - 1) / p.tile);
  }
  __syncthreads();
  for (int e = warp; e < p.E; e += kMoeWarps) {
    const int n = base[e], r0 = hist[e], blocks = (n + p.tile - 1) / p.tile;
    for (int which = 0; which < 2; ++which) {
      const int n_out = which ? p.n_out2 : p.n_out1, nt = (n_out + p.tile - 1) / p.tile;
      int4* dst = (which ? p.tiles2 : p.tiles1) + static_cast<long long>(blk[e]) * nt;
      for (int i = lane; i < blocks * nt; i += 32) {
        const int b = i % blocks, t = i / blocks;    // row blocks of one column tile run side by side and share its weights
        dst[i] = make_int4(r0 + b * p.tile, r0 + n, e * n_out, t);
      }
    }
  }
}

// xs[slot of (row, choice)] = h[row]; also writes the slots.  One block per row.
template <typename V>
__global__ void __launch_bounds__(128)
moe_serve_gather_kernel(const V* __restrict__ h, int n, const int* __restrict__ expert, const int* __restrict__ rank,
                        const int* __restrict__ first, int top, int* __restrict__ slots, V* __restrict__ xs) {
  pdl_entry();
  __shared__ int s[32];
  const long long row = blockIdx.x;
  if (threadIdx.x < top) {
    const int e = expert[row * top + threadIdx.x];
    const int v = e >= 0 ? first[e] + rank[row * top + threadIdx.x] : -1;
    s[threadIdx.x] = v;
    slots[row * top + threadIdx.x] = v;
  }
  __syncthreads();
  for (int c = threadIdx.x; c < n; c += 128) {
    const V v = h[row * n + c];
    for (int k = 0; k < top; ++k)
      if (s[k] >= 0) xs[static_cast<long long>(s[k]) * n + c] = v;
  }
}

// The same, every row multiplied by its weight.
template <typename T, int V>
__global__ void __launch_bounds__(128)
moe_serve_gather_scaled_kernel(const T* __restrict__ h, int n, const int* __restrict__ expert, const int* __restrict__ rank,
                               const int* __restrict__ first, const float* __restrict__ weight, int top, int* __restrict__ slots,
                               T* __restrict__ xs) {
  pdl_entry();
  __shared__ int s[32];
  __shared__ float w[32];
  const long long row = blockIdx.x;
  if (threadIdx.x < top) {
    const int e = expert[row * top + threadIdx.x];
    const int v = e >= 0 ? first[e] + rank[row * top + threadIdx.x] : -1;
    s[threadIdx.x] = v;
    w[threadIdx.x] = weight[row * top + threadIdx.x];
    slots[row * top + threadIdx.x] = v;
  }
  __syncthreads();
  for (int c = threadIdx.x * V; c < n; c += 128 * V) {
    float v[V];
    if constexpr (V == 8) {
      const uint4 raw = *reinterpret_cast<const uint4*>(h + row * n + c);
      const uint32_t u[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u[i]));
        v[2 * i] = f.x;
        v[2 * i + 1] = f.y;
      }
    } else {
      v[0] = to_f32(h[row * n + c]);
    }
    for (int k = 0; k < top; ++k) {
      if (s[k] < 0) continue;
      T* dst = xs + static_cast<long long>(s[k]) * n + c;
      const float f = w[k];
      if constexpr (V == 8)
        *reinterpret_cast<uint4*>(dst) = make_uint4(pack_bf16x2(v[0] * f, v[1] * f), pack_bf16x2(v[2] * f, v[3] * f),
                                                    pack_bf16x2(v[4] * f, v[5] * f), pack_bf16x2(v[6] * f, v[7] * f));
      else
        *dst = from_f32<T>(v[0] * f);
    }
  }
}

}  // namespace apb

extern "C" {
using namespace apb;

int apb_moe_serve_route(const float* logits, long long ld, const void* correction, const int* live, int rows, int N, int E,
                        int top, int* expert, int* rank, float* weight, float* ident, int* counters, int* first, void* tiles1,
                        void* tiles2, int* n_tiles, int n_out1, int n_out2, int tile, int sigmoid, int dtype, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (E <= 0 || N < E || N > kMoeMax || top < 1 || top > 32 || top > N || ld < N || tile < 1 || !counters) return kBadArgument;
  const MoeRouteParams p{logits, ld, correction, live, sigmoid, rows, N, E, top, expert, rank, weight, ident, counters, first,
                         static_cast<int4*>(tiles1), static_cast<int4*>(tiles2), n_tiles, n_out1, n_out2, tile};
  const dim3 grid((rows + kMoeWarps - 1) / kMoeWarps);
  APB_SERVE_DTYPE(dtype, return static_cast<int>(launch_kernel(moe_serve_route_kernel<T>, grid, dim3(kMoeThreads), 0, s, p)));
}

// h [rows, row_bytes], xs [slots, row_bytes]
int apb_moe_serve_gather(const void* h, int rows, long long row_bytes, const int* expert, const int* rank, const int* first,
                         int top, int* slots, void* xs, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (top < 1 || top > 32 || row_bytes <= 0) return kBadArgument;
  const uintptr_t a = reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(xs) | static_cast<uintptr_t>(row_bytes);
#define APB_GATHER(V)                                                                                                       \
  return static_cast<int>(launch_kernel(moe_serve_gather_kernel<V>, dim3(rows), dim3(128), 0, s, static_cast<const V*>(h),  \
                                        static_cast<int>(row_bytes / sizeof(V)), expert, rank, first, top, slots,          \
                                        static_cast<V*>(xs)))
  if ((a & 15) == 0) APB_GATHER(uint4);
  if ((a & 3) == 0) APB_GATHER(uint32_t);
  APB_GATHER(uint16_t);
#undef APB_GATHER
}

// The same with every row times its weight; h and xs [rows, n] of the activation type.
int apb_moe_serve_gather_scaled(const void* h, int rows, int n, const int* expert, const int* rank, const int* first,
                                const float* weight, int top, int* slots, void* xs, int dtype, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (top < 1 || top > 32 || n <= 0 || !weight) return kBadArgument;
  const bool vec = dtype == 0 && !(n & 7) && !((reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(xs)) & 15);
#define APB_GATHER(TT, VV)                                                                                                   \
  return static_cast<int>(launch_kernel(moe_serve_gather_scaled_kernel<TT, VV>, dim3(rows), dim3(128), 0, s,                 \
                                        static_cast<const TT*>(h), n, expert, rank, first, weight, top, slots, static_cast<TT*>(xs)))
  if (vec) APB_GATHER(__nv_bfloat16, 8);
  APB_SERVE_DTYPE(dtype, APB_GATHER(T, 1));
#undef APB_GATHER
}
}
