// Recurrent mixers (see recurrent.cuh) on a ragged serving batch, fp32 arithmetic.
//
//  * recurrent_decode_kernel  entries of one token: gates, convolution, state update, norm and output gate of a (sequence, head)
//                             fused; streams its state once (read, update, write) -- bound by the bytes of the state;
//  * recurrent_scan_kernel    longer entries, token by token (the fp32 engine, odd sizes): one CTA per (entry, head, 32 columns of
//                             the state), that part of the state in shared memory;
//  * head_norm_gate_kernel    norm and output gate of the longer entries' rows;
//  * token_shift_kernel       the inputs of time mixing: h + (previous token's h - h) mu for several mu.
//
// All three rules are one update.  A token turns into qa, ka, a, kd [D], v [E] and scalars such that with the old state S
//     u = beta (v - S^T ka)  (delta rule; else v),   o = (S^T qa + c u) * fin,   S' = diag(a) S + kd u^T.
//
// bf16 engines run the longer entries on tensor cores (memory_mma.cu, delta_mma.cu, time_mix_mma.cu).
#include "common.cuh"
#include "host_utils.cuh"
#include "recurrent.cuh"

namespace apb {

constexpr int kRecThreads = 256;

struct TokenParts {         // shared memory
  float *qa, *ka, *a, *kd;  // [D]
  float* v;                 // [E]
  float* n;                 // [D] memory only: the normaliser, updated
  float (*red)[8];          // [3][8]
};
struct TokenScalars {
  float c, beta, fin;
};

// Sums of three values over the block.
__device__ __forceinline__ float3 rec_block_sum(float x, float y, float z, float (*red)[8]) {
  x = warp_sum(x);
  y = warp_sum(y);
  z = warp_sum(z);
  __syncthreads();                       // the last sums have been read
  if ((threadIdx.x & 31) == 0) {
    red[0][threadIdx.x >> 5] = x;
    red[1][threadIdx.x >> 5] = y;
    red[2][threadIdx.x >> 5] = z;
  }
  __syncthreads();
  float3 r = make_float3(0.f, 0.f, 0.f);
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    r.x += red[0][i];
    r.y += red[1][i];
    r.z += red[2][i];
  }
  return r;
}

// The parts of one token.  CONV: the delta rule's convolution is computed here (one-token entries), from the history in `old_h`,
// which moves on into `new_h`; otherwise its results are read.  m: the memory's running maximum.
template <int RULE, typename T, bool CONV>
__device__ __forceinline__ TokenScalars recurrent_token(const RecurrentParams& p, long long row, int h, int pos, const float* old_h,
                                                        float* new_h, float& m, const TokenParts& s) {
  const int D = p.D, E = p.E, kh = h / (p.H / p.KH);
  const T* pr = static_cast<const T*>(p.p) + row * p.ld;
  const float scale = 1.f / sqrtf(static_cast<float>(D));
  if constexpr (RULE == kRuleMemory) {
    const float2 g = memory_gates<T>(p, row, h);
    const float top = fmaxf(g.x + m, g.y), a = expf(g.x + m - top), b = expf(g.y - top);
    m = top;
    float c = 0.f, den = 0.f;
    for (int d = threadIdx.x; d < D; d += kRecThreads) {
      const float q = to_f32(pr[p.q_off + kh * D + d]) * scale, k = to_f32(pr[p.k_off + kh * D + d]) * b;
      const float n = a * s.n[d] + k;
      s.n[d] = n;
      s.qa[d] = a * q;
      s.a[d] = a;
      s.kd[d] = k;
      c += q * k;
      den += n * q;
    }
    for (int i = threadIdx.x; i < E; i += kRecThreads) s.v[i] = to_f32(pr[p.v_off + h * E + i]);
    const float3 r = rec_block_sum(c, den, 0.f, s.red);
    return TokenScalars{r.x, 1.f, 1.f / (fmaxf(fabsf(r.y), expf(-top)) + 1e-6f)};
  } else if constexpr (RULE == kRuleDelta) {
    const float2 g = delta_gates<T>(p, row, h);
    const float dec = expf(g.x);
    const int nk = p.KH * D, channels = 2 * nk + p.H * E, hist = p.taps - 1;
    const bool owner = h % (p.H / p.KH) == 0;            // writes the history of its q and k
    auto value = [&](int c, bool keep) -> float {
      if constexpr (!CONV) return to_f32(static_cast<const T*>(p.xc)[row * p.ldx + c]);
      const T* w = static_cast<const T*>(p.conv_w) + c;
      const float cur = to_f32(pr[p.q_off + c]);
      float v = to_f32(w[static_cast<long long>(hist) * channels]) * cur;
      for (int j = 0; j < hist; ++j) {
        const float x = pos - hist + j >= 0 ? old_h[static_cast<long long>(j) * channels + c] : 0.f;
        v += to_f32(w[static_cast<long long>(j) * channels]) * x;
        if (j > 0 && keep) new_h[static_cast<long long>(j - 1) * channels + c] = x;
      }
      if (hist > 0 && keep) new_h[static_cast<long long>(hist - 1) * channels + c] = cur;
      return to_f32(from_f32<T>(v / (1.f + expf(-v))));   // q, k and v are activations
    };
    float qq = 0.f, kk = 0.f, qk = 0.f;
    for (int i = threadIdx.x; i < E; i += kRecThreads) s.v[i] = value(2 * nk + h * E + i, true);
    for (int d = threadIdx.x; d < D; d += kRecThreads) {
      const float q = value(kh * D + d, owner), k = value(nk + kh * D + d, owner);
      s.qa[d] = q;
      s.kd[d] = k;
      qq += q * q;
      kk += k * k;
      qk += q * k;
    }
    const float3 r = rec_block_sum(qq, kk, qk, s.red);
    const float fq = scale / sqrtf(r.x + 1e-6f), fk = 1.f / sqrtf(r.y + 1e-6f);
    for (int d = threadIdx.x; d < D; d += kRecThreads) {
      s.qa[d] *= fq * dec;
      const float k = s.kd[d] * fk;
      s.kd[d] = k;
      s.ka[d] = k * dec;
      s.a[d] = dec;
    }
    return TokenScalars{fq * fk * r.z, g.y, 1.f};
  } else {
    float c = 0.f;
    const T* u = static_cast<const T*>(p.w1) + h * D;
    const T* w0 = static_cast<const T*>(p.w0) + h * D;
    for (int d = threadIdx.x; d < D; d += kRecThreads) {
      const float r = to_f32(pr[p.q_off + kh * D + d]), k = to_f32(pr[p.k_off + kh * D + d]);
      s.qa[d] = r;
      s.kd[d] = k;
      s.a[d] = expf(-expf(p.z[row * p.ldz + h * D + d] + to_f32(w0[d])));
      c += r * k * to_f32(u[d]);
    }
    for (int i = threadIdx.x; i < E; i += kRecThreads) s.v[i] = to_f32(pr[p.v_off + h * E + i]);
    return TokenScalars{rec_block_sum(c, 0.f, 0.f, s.red).x, 1.f, 1.f};
  }
}

// ---------------------------------------------------------------------------- one token
template <int V>
__device__ __forceinline__ float4 rec_load(const float* p) {
  if constexpr (V == 4) return __ldcs(reinterpret_cast<const float4*>(p));
  return make_float4(*p, 0.f, 0.f, 0.f);
}
template <int V>
__device__ __forceinline__ void rec_store(float* p, const float4& v) {
  if constexpr (V == 4)
    __stcs(reinterpret_cast<float4*>(p), v);
  else
    *p = v.x;
}

// AHEAD: state rows per thread that are on their way while the token's parts are computed (and stay in registers).
template <int RULE, typename T, int VEC, int AHEAD>
__global__ void __launch_bounds__(kRecThreads, AHEAD > 8 ? 2 : AHEAD > 4 ? 3 : 4)
recurrent_decode_kernel(const RecurrentParams p) {
  pdl_entry();
  extern __shared__ __align__(16) float rec_smem[];
  __shared__ float red[3][8];
  const int en = blockIdx.x, h = blockIdx.y;
  if (p.e.len[en] != 1) return;
  const int D = p.D, E = p.E;
  const int nx = min(E / VEC, kRecThreads), ny = kRecThreads / nx;
  TokenParts s;
  s.v = rec_smem;                              // [E]
  float* us = s.v + E;                         // [E]
  float* rq = us + E;                          // [ny][E]
  float* rk = rq + ny * E;                     // [ny][E] (delta)
  s.qa = rk + (RULE == kRuleDelta ? ny * E : 0);
  s.ka = s.qa + D;
  s.a = s.ka + D;
  s.kd = s.a + D;
  s.n = s.kd + D;
  s.red = red;
  const long long row = p.e.start[en];
  const int slot = p.e.slot[en], pos = p.e.pos0[en];
  float* S = p.state + (static_cast<long long>(slot) * p.H + h) * D * E;
  const int tx = threadIdx.x % nx, ty = threadIdx.x / nx;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 ahead[AHEAD];
#pragma unroll
  for (int k = 0; k < AHEAD; ++k) {
    const int d = ty + k * ny;
    ahead[k] = pos > 0 && ty < ny && d < D ? rec_load<VEC>(S + static_cast<long long>(d) * E + tx * VEC) : zero;   // position 0: the slot may hold anything
  }
  float m = 0.f;
  float* aux = nullptr;
  if constexpr (RULE == kRuleMemory) {
    aux = p.aux + (static_cast<long long>(slot) * p.H + h) * (D + 1);
    if (pos > 0) m = aux[D];
    for (int d = threadIdx.x; d < D; d += kRecThreads) s.n[d] = pos > 0 ? aux[d] : 0.f;
  }
  const float* old_h = nullptr;
  float* new_h = nullptr;
  if (RULE == kRuleDelta && p.taps > 1) {
    const int par = p.parity[slot] & 1;
    const long long size = static_cast<long long>(p.taps - 1) * (2 * p.KH * D + p.H * E);
    old_h = p.hist + (static_cast<long long>(slot) * 2 + par) * size;
    new_h = p.hist + (static_cast<long long>(slot) * 2 + (par ^ 1)) * size;
  }
  const TokenScalars t = recurrent_token<RULE, T, true>(p, row, h, pos, old_h, new_h, m, s);
  if constexpr (RULE == kRuleMemory) {
    for (int d = threadIdx.x; d < D; d += kRecThreads) aux[d] = s.n[d];
    if (threadIdx.x == 0) aux[D] = m;          // everybody has read it: the sums above met at a barrier
  }
  __syncthreads();
  auto rows_of = [&](int cx, auto f) {         // f(d, old state) over this thread's rows of column run cx
    int d = ty;
    if (cx == tx) {
#pragma unroll
      for (int k = 0; k < AHEAD; ++k, d += ny)
        if (d < D) f(d, ahead[k]);
    }
#pragma unroll 4
    for (; d < D; d += ny) f(d, pos > 0 ? rec_load<VEC>(S + static_cast<long long>(d) * E + cx * VEC) : zero);
  };
  auto update = [&](int d, int cx, const float4& o, const float4& u) {
    const float a = s.a[d], k = s.kd[d];
    rec_store<VEC>(S + static_cast<long long>(d) * E + cx * VEC,
                   make_float4(o.x * a + k * u.x, o.y * a + k * u.y, o.z * a + k * u.z, o.w * a + k * u.w));
  };
  auto run_of = [&](const float* x, int cx) {
    return VEC == 4 ? *reinterpret_cast<const float4*>(x + cx * 4) : make_float4(x[cx], 0.f, 0.f, 0.f);
  };
  if (ty < ny) {
    for (int cx = tx; cx < E / VEC; cx += nx) {
      float4 aq = zero, ak = zero;
      const float4 u = run_of(s.v, cx);
      rows_of(cx, [&](int d, const float4& o) {
        const float q = s.qa[d];
        aq = make_float4(aq.x + q * o.x, aq.y + q * o.y, aq.z + q * o.z, aq.w + q * o.w);
        if constexpr (RULE == kRuleDelta) {
          const float k = s.ka[d];
          ak = make_float4(ak.x + k * o.x, ak.y + k * o.y, ak.z + k * o.z, ak.w + k * o.w);
        } else {
          update(d, cx, o, u);
        }
      });
      const float vq[4] = {aq.x, aq.y, aq.z, aq.w}, vk[4] = {ak.x, ak.y, ak.z, ak.w};
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        rq[ty * E + cx * VEC + i] = vq[i];
        if (RULE == kRuleDelta) rk[ty * E + cx * VEC + i] = vk[i];
      }
    }
  }
  __syncthreads();
  float ss = 0.f;
  for (int i = threadIdx.x; i < E; i += kRecThreads) {
    float o = 0.f, u = s.v[i];
    for (int y = 0; y < ny; ++y) o += rq[y * E + i];
    if constexpr (RULE == kRuleDelta) {
      float k = 0.f;
      for (int y = 0; y < ny; ++y) k += rk[y * E + i];
      u = t.beta * (u - k);
      us[i] = u;
    }
    o = (o + t.c * u) * t.fin;
    rq[i] = o;                                 // column i of every part was read by this thread only
    ss += o * o;
  }
  const float r = 1.f / sqrtf(rec_block_sum(ss, 0.f, 0.f, red).x / E + p.eps);
  if constexpr (RULE == kRuleDelta) {
    if (ty < ny)
      for (int cx = tx; cx < E / VEC; cx += nx) {
        const float4 u = run_of(us, cx);
        rows_of(cx, [&](int d, const float4& o) { update(d, cx, o, u); });
      }
  }
  const T* gain = static_cast<const T*>(p.gain) + static_cast<long long>(h) * p.gain_step;
  const T* z = static_cast<const T*>(p.p) + row * p.ld + p.g_off + h * E;
  T* out = static_cast<T*>(p.out) + row * p.ldo + h * E;
  for (int i = threadIdx.x; i < E; i += kRecThreads) out[i] = from_f32<T>(rq[i] * r * to_f32(gain[i]) * rec_gate(to_f32(z[i]), p.silu));
}

// ---------------------------------------------------------------------------- longer entries, token by token
constexpr int kRecCols = 32;

template <int RULE, typename T>
__global__ void __launch_bounds__(kRecThreads)
recurrent_scan_kernel(const RecurrentParams p) {
  pdl_entry();
  extern __shared__ __align__(16) float rec_smem[];
  __shared__ float red[3][8], rq[8][kRecCols], rk[8][kRecCols];
  const int en = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * kRecCols;
  const int len = p.e.len[en];
  if (len <= 1) return;
  const int D = p.D, E = p.E, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  TokenParts s;
  float* S = rec_smem;                         // [D][32]
  s.qa = S + D * kRecCols;
  s.ka = s.qa + D;
  s.a = s.ka + D;
  s.kd = s.a + D;
  s.n = s.kd + D;
  s.v = s.n + D;
  s.red = red;
  const long long start = p.e.start[en];
  const int slot = p.e.slot[en], pos0 = p.e.pos0[en], col = e0 + lane;
  const bool ok = col < E;
  float* Sg = p.state + (static_cast<long long>(slot) * p.H + h) * D * E;
  for (int d = warp; d < D; d += 8) S[d * kRecCols + lane] = pos0 > 0 && ok ? Sg[static_cast<long long>(d) * E + col] : 0.f;
  float m = 0.f;
  const float* aux_in = nullptr;
  if constexpr (RULE == kRuleMemory) {
    aux_in = p.aux + (static_cast<long long>(slot) * p.H + h) * (D + 1);
    if (pos0 > 0) m = aux_in[D];
    for (int d = threadIdx.x; d < D; d += kRecThreads) s.n[d] = pos0 > 0 ? aux_in[d] : 0.f;
  }
  for (int t = 0; t < len; ++t) {
    const TokenScalars k = recurrent_token<RULE, T, false>(p, start + t, h, pos0 + t, nullptr, nullptr, m, s);
    __syncthreads();
    const float v = ok ? s.v[col] : 0.f;
    float aq = 0.f, ak = 0.f;
    for (int d = warp; d < D; d += 8) {
      const float o = S[d * kRecCols + lane];
      aq += s.qa[d] * o;
      if (RULE == kRuleDelta)
        ak += s.ka[d] * o;
      else
        S[d * kRecCols + lane] = s.a[d] * o + s.kd[d] * v;
    }
    rq[warp][lane] = aq;
    if (RULE == kRuleDelta) rk[warp][lane] = ak;
    __syncthreads();
    float u = v;
    if constexpr (RULE == kRuleDelta) {
      float x = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) x += rk[w][lane];
      u = k.beta * (v - x);
      for (int d = warp; d < D; d += 8) S[d * kRecCols + lane] = s.a[d] * S[d * kRecCols + lane] + s.kd[d] * u;
    }
    if (warp == 0 && ok) {
      float o = k.c * u;
#pragma unroll
      for (int w = 0; w < 8; ++w) o += rq[w][lane];
      p.y[(start + t) * p.H * E + static_cast<long long>(h) * E + col] = o * k.fin;
    }
    __syncthreads();                           // the parts are written again
  }
  for (int d = warp; d < D; d += 8)
    if (ok) Sg[static_cast<long long>(d) * E + col] = S[d * kRecCols + lane];
}

// The memory's normaliser and running maximum after the longer entries: their states before them are read by all column slices
// of the kernel above, so they are advanced afterwards.  One CTA per (entry, head).
template <typename T>
__global__ void __launch_bounds__(kRecThreads)
memory_aux_kernel(const RecurrentParams p) {
  pdl_entry();
  const int en = blockIdx.x, h = blockIdx.y, len = p.e.len[en];
  if (len <= 1) return;
  const int D = p.D, kh = h / (p.H / p.KH), pos0 = p.e.pos0[en];
  const long long start = p.e.start[en];
  float* aux = p.aux + (static_cast<long long>(p.e.slot[en]) * p.H + h) * (D + 1);
  const float m0 = pos0 > 0 ? aux[D] : 0.f;
  __syncthreads();
  float m = m0;
  for (int d0 = 0; d0 < D; d0 += kRecThreads) {
    const int d = d0 + threadIdx.x;
    float n = pos0 > 0 && d < D ? aux[d] : 0.f;
    m = m0;
    for (int t = 0; t < len; ++t) {
      const float2 g = memory_gates<T>(p, start + t, h);
      const float top = fmaxf(g.x + m, g.y);
      const float k = d < D ? to_f32(static_cast<const T*>(p.p)[(start + t) * p.ld + p.k_off + kh * D + d]) : 0.f;
      n = expf(g.x + m - top) * n + expf(g.y - top) * k;
      m = top;
    }
    if (d < D) aux[d] = n;
  }
  if (threadIdx.x == 0) aux[D] = m;
}

// ---------------------------------------------------------------------------- norm and output gate
// One warp per (row, head) of the entries longer than one token.
template <typename T, int V>
__global__ void __launch_bounds__(256)
head_norm_gate_kernel(const RecurrentParams p, const int* __restrict__ row_entry, int rows) {
  pdl_entry();
  const unsigned gw = blockIdx.x * 8u + (threadIdx.x >> 5), H = p.H;       // rows * heads fits: the entry point checks
  if (gw >= rows * H) return;
  const int lane = threadIdx.x & 31, h = static_cast<int>(gw % H), E = p.E;
  const long long row = gw / H;
  if (row_entry && p.e.len[row_entry[row]] <= 1) return;
  const float* y = p.y + static_cast<long long>(gw) * E;
  const T* z = static_cast<const T*>(p.p) + row * p.ld + p.g_off + h * E;
  const T* gain = static_cast<const T*>(p.gain) + static_cast<long long>(h) * p.gain_step;
  T* out = static_cast<T*>(p.out) + row * p.ldo + h * E;
  float ss = 0.f;
  if constexpr (V == 4) {
    float4 keep = make_float4(0.f, 0.f, 0.f, 0.f);             // the first 128 columns stay in registers
    for (int c = lane * 4; c < E; c += 128) {
      const float4 v = *reinterpret_cast<const float4*>(y + c);
      if (c < 128) keep = v;
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    const float r = 1.f / sqrtf(warp_sum(ss) / E + p.eps);
    auto two = [](uint32_t w) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w)); };
    auto gate = [&](float x) { return __fdividef(p.silu ? x : 1.f, 1.f + __expf(-x)); };
    for (int c = lane * 4; c < E; c += 128) {
      const float4 v = c < 128 ? keep : *reinterpret_cast<const float4*>(y + c);
      const uint2 zr = *reinterpret_cast<const uint2*>(z + c), gr = *reinterpret_cast<const uint2*>(gain + c);
      const float2 z0 = two(zr.x), z1 = two(zr.y), g0 = two(gr.x), g1 = two(gr.y);
      *reinterpret_cast<uint2*>(out + c) = make_uint2(pack_bf16x2(v.x * r * g0.x * gate(z0.x), v.y * r * g0.y * gate(z0.y)),
                                                      pack_bf16x2(v.z * r * g1.x * gate(z1.x), v.w * r * g1.y * gate(z1.y)));
    }
  } else {
    for (int c = lane; c < E; c += 32) ss += y[c] * y[c];
    const float r = 1.f / sqrtf(warp_sum(ss) / E + p.eps);
    for (int c = lane; c < E; c += 32) out[c] = from_f32<T>(y[c] * r * to_f32(gain[c]) * rec_gate(to_f32(z[c]), p.silu));
  }
}

// ---------------------------------------------------------------------------- inputs of time mixing
// out[s] = h + (h of the token before - h) * mu[s] for s < n_mix; the token before an entry's first row is in `hist` [slots, 2, W]
// (double buffered: the last row leaves its h in the other half), and zero ahead of a sequence.  Block 0 also writes the tile table
// of the grouped product over out [n_mix * rows, W]: group s uses the weight rows from s * w_step on and cols[s] of its columns.
constexpr int kShiftMax = 8;
struct ShiftParams {
  ServeEntries e;
  const int* row_entry;
  const void* h;
  const void* mu;           // [n_mix, W]
  float* hist;
  const int* parity;
  void* out;                // [n_mix, rows, W]
  int rows, W, n_mix;
  int4* tiles;              // or null
  int* n_tiles;
  int tile, w_step;
  int cols[kShiftMax];
};

template <typename T, int V, int R>            // R rows per block
__global__ void __launch_bounds__(128)
token_shift_kernel(const ShiftParams p) {
  pdl_entry();
  if (blockIdx.x == 0 && p.tiles) {
    const int blocks = (p.rows + p.tile - 1) / p.tile;
    int at = 0;
    for (int s = 0; s < p.n_mix; ++s) {
      const int nt = (p.cols[s] + p.tile - 1) / p.tile;
      for (int i = threadIdx.x; i < blocks * nt; i += 128)
        p.tiles[at + i] = make_int4(s * p.rows + (i % blocks) * p.tile, (s + 1) * p.rows, s * p.w_step, i / blocks);
      at += blocks * nt;
    }
    if (threadIdx.x == 0) *p.n_tiles = at;
  }
  const int row0 = blockIdx.x * R;
  for (int c = threadIdx.x * V; c < p.W; c += 128 * V) {
    float mu[kShiftMax][V], h[V], before[V];
    auto load = [&](const T* src, float(&v)[V]) {
      if constexpr (V == 4) {
        const uint2 raw = *reinterpret_cast<const uint2*>(src);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        v[0] = a.x;
        v[1] = a.y;
        v[2] = b.x;
        v[3] = b.y;
      } else {
        v[0] = to_f32(*src);
      }
    };
#pragma unroll
    for (int s = 0; s < kShiftMax; ++s)
      if (s < p.n_mix) load(static_cast<const T*>(p.mu) + static_cast<long long>(s) * p.W + c, mu[s]);
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int row = row0 + i;
      if (row >= p.rows) break;
      const int en = p.row_entry ? p.row_entry[row] : row;
      const int at = row - p.e.start[en], len = p.e.len[en], slot = p.e.slot[en];
      if (at < 0 || at >= len) continue;
      const int par = p.parity[slot] & 1;
      const T* src = static_cast<const T*>(p.h) + static_cast<long long>(row) * p.W + c;
      if (at == 0) {
        const float* old = p.hist + (static_cast<long long>(slot) * 2 + par) * p.W + c;
#pragma unroll
        for (int j = 0; j < V; ++j) before[j] = p.e.pos0[en] > 0 ? old[j] : 0.f;
      } else if (i == 0) {
        load(src - p.W, before);
      } else {
#pragma unroll
        for (int j = 0; j < V; ++j) before[j] = h[j];
      }
      load(src, h);
      if (at == len - 1) {
        float* next = p.hist + (static_cast<long long>(slot) * 2 + (par ^ 1)) * p.W + c;
#pragma unroll
        for (int j = 0; j < V; ++j) next[j] = h[j];
      }
#pragma unroll
      for (int s = 0; s < kShiftMax; ++s)
        if (s < p.n_mix) {
          T* dst = static_cast<T*>(p.out) + (static_cast<long long>(s) * p.rows + row) * p.W + c;
          float v[V];
#pragma unroll
          for (int j = 0; j < V; ++j) v[j] = h[j] + (before[j] - h[j]) * mu[s][j];
          if constexpr (V == 4)
            *reinterpret_cast<uint2*>(dst) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
          else
            *dst = from_f32<T>(v[0]);
        }
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
tanh_rows_kernel(T* __restrict__ x, long long ld, int rows, int n) {
  pdl_entry();
  const unsigned i = blockIdx.x * 256u + threadIdx.x, w = n;
  if (i >= rows * w) return;
  T* v = x + static_cast<long long>(i / w) * ld + i % w;
  *v = from_f32<T>(tanhf(to_f32(*v)));
}

template <typename F>
static int rec_smem_limit(F fn, size_t bytes) {
  if (bytes > 220 * 1024) return kBadArgument;
  return bytes <= 40 * 1024 ? 0 : static_cast<int>(cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes)));
}

template <int RULE, typename T>
static int recurrent_run(const RecurrentParams& a, const int* row_entry, int n_entries, int rows, int decode, int scan, int finish,
                         cudaStream_t s) {
  if (decode) {
    const bool v4 = !(a.E & 3) && !(reinterpret_cast<uintptr_t>(a.state) & 15);
    const int cols = v4 ? a.E / 4 : a.E, nx = cols < kRecThreads ? cols : kRecThreads, ny = kRecThreads / nx;
    const size_t smem = (2 * a.E + static_cast<size_t>(RULE == kRuleDelta ? 2 : 1) * ny * a.E + 5 * a.D) * sizeof(float);
    auto run = [&](auto fn) -> int {
      const int rc = rec_smem_limit(fn, smem);
      return rc ? rc : static_cast<int>(launch_kernel(fn, dim3(n_entries, a.H), dim3(kRecThreads), smem, s, a));
    };
    const int each = (a.D + ny - 1) / ny;      // state rows per thread
    const int rc = !v4 ? run(recurrent_decode_kernel<RULE, T, 1, 8>) : each <= 4 ? run(recurrent_decode_kernel<RULE, T, 4, 4>)
                   : each <= 8 || RULE != kRuleDelta ? run(recurrent_decode_kernel<RULE, T, 4, 8>) : run(recurrent_decode_kernel<RULE, T, 4, 16>);
    if (rc) return rc;
  }
  if (scan) {
    const size_t smem = (static_cast<size_t>(a.D) * (kRecCols + 5) + a.E) * sizeof(float);
    auto fn = recurrent_scan_kernel<RULE, T>;
    int rc = rec_smem_limit(fn, smem);
    if (!rc)
      rc = static_cast<int>(launch_kernel(fn, dim3(n_entries, a.H, (a.E + kRecCols - 1) / kRecCols), dim3(kRecThreads), smem, s, a));
    if (!rc && RULE == kRuleMemory)
      rc = static_cast<int>(launch_kernel(memory_aux_kernel<T>, dim3(n_entries, a.H), dim3(kRecThreads), 0, s, a));
    if (rc) return rc;
  }
  if (finish) {
    const dim3 grid(static_cast<unsigned>((static_cast<long long>(rows) * a.H + 7) / 8));
    const bool v4 = sizeof(T) == 2 && !(a.E & 3) && !((a.ld | a.g_off | a.ldo | a.gain_step) & 3) &&
                    !((reinterpret_cast<uintptr_t>(a.p) | reinterpret_cast<uintptr_t>(a.gain) | reinterpret_cast<uintptr_t>(a.out)) & 7);
    if constexpr (sizeof(T) == 2) {
      if (v4) return static_cast<int>(launch_kernel(head_norm_gate_kernel<T, 4>, grid, dim3(256), 0, s, a, row_entry, rows));
    }
    return static_cast<int>(launch_kernel(head_norm_gate_kernel<T, 1>, grid, dim3(256), 0, s, a, row_entry, rows));
  }
  return 0;
}

}  // namespace apb

extern "C" {
using namespace apb;

// Runs the one-token entries (decode), the longer ones token by token (scan; y is written) and / or the norm and gate of the
// longer entries' rows (finish; y is read).  rule: 0 matrix memory, 1 delta rule, 2 time mixing.
int apb_recurrent(int rule, const RecurrentParams* params, const int* row_entry, int n_entries, int rows, int decode, int scan,
                  int finish, int dtype, cudaStream_t s) {
  if (n_entries <= 0 || rows <= 0) return 0;
  const RecurrentParams& a = *params;
  if (!recurrent_params_ok(rule, a) || ((scan || finish) && !a.y) || static_cast<long long>(rows) * a.H > 0x7fffffffLL || (rule == kRuleDelta && scan && !a.xc)) return kBadArgument;
  APB_SERVE_DTYPE(dtype, if (rule == kRuleMemory) return recurrent_run<kRuleMemory, T>(a, row_entry, n_entries, rows, decode, scan, finish, s);
                  if (rule == kRuleDelta) return recurrent_run<kRuleDelta, T>(a, row_entry, n_entries, rows, decode, scan, finish, s);
                  if (rule == kRuleTimeMix) return recurrent_run<kRuleTimeMix, T>(a, row_entry, n_entries, rows, decode, scan, finish, s));
}

// h [rows, W], mu [n_mix, W], out [n_mix, rows, W]; hist [slots, 2, W] fp32.  tiles (or null): room for the table of the grouped
// product, see the kernel; cols [n_mix] on the host.
int apb_token_shift(const void* h, const void* mu, float* hist, const int* parity, void* out, const int* row_entry,
                    const int* e_start, const int* e_len, const int* e_slot, const int* e_pos0, int rows, int W, int n_mix,
                    void* tiles, int* n_tiles, int tile, int w_step, const int* cols, int dtype, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (!h || !mu || !hist || !parity || !out || W <= 0 || n_mix < 1 || n_mix > kShiftMax || (tiles && (!n_tiles || !cols || tile < 1)))
    return kBadArgument;
  ShiftParams p{ServeEntries{e_start, e_len, e_slot, e_pos0}, row_entry, h, mu, hist, parity, out, rows, W, n_mix,
                static_cast<int4*>(tiles), n_tiles, tile, w_step, {}};
  for (int i = 0; i < n_mix && tiles; ++i) p.cols[i] = cols[i];
  const bool vec = dtype == 0 && !(W & 3) && !((reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(mu) | reinterpret_cast<uintptr_t>(out)) & 7);
  const int per = rows >= 1024 ? 4 : 1;
  const dim3 grid((rows + per - 1) / per);
  if (vec)
    return static_cast<int>(per == 4 ? launch_kernel(token_shift_kernel<__nv_bfloat16, 4, 4>, grid, dim3(128), 0, s, p)
                                     : launch_kernel(token_shift_kernel<__nv_bfloat16, 4, 1>, grid, dim3(128), 0, s, p));
  APB_SERVE_DTYPE(dtype, return static_cast<int>(per == 4 ? launch_kernel(token_shift_kernel<T, 1, 4>, grid, dim3(128), 0, s, p)
                                                          : launch_kernel(token_shift_kernel<T, 1, 1>, grid, dim3(128), 0, s, p)));
}

// x [rows, n] columns (row stride ld) <- tanh(x)
int apb_tanh_rows(void* x, long long ld, int rows, int n, int dtype, cudaStream_t s) {
  if (rows <= 0 || n <= 0) return 0;
  if (static_cast<long long>(rows) * n > 0x7fffffffLL) return kBadArgument;
  const dim3 grid(static_cast<unsigned>((static_cast<long long>(rows) * n + 255) / 256));
  APB_SERVE_DTYPE(dtype, return static_cast<int>(launch_kernel(tanh_rows_kernel<T>, grid, dim3(256), 0, s, static_cast<T*>(x), ld, rows, n)));
}
}
