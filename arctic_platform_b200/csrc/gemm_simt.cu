// GEMM on CUDA cores, fp32 accumulation: C[M,N] = A[M,K] * B[N,K]^T for fp32 operands (the fp32 engine: true 32-bit
// products, no TF32) and for bf16 operands whose row lengths are not multiples of 8, which the TMA-fed tensor-core
// kernels cannot address.  Same epilogues as those kernels where a serving step needs them; grouped products (a tile table) and
// products per head (column blocks of A and C, row blocks of B) as there.
#include "common.cuh"
#include "gemm_common.cuh"
#include "host_utils.cuh"
#include "serve_common.cuh"

namespace apb {

constexpr int kSgTile = 64, kSgK = 16;

__device__ __forceinline__ float clamped_glu(float g, float u, float limit) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g / (1.f + expf(-1.702f * g)) * (u + 1.f);
}

struct SimtParams {
  const void* A;
  const void* B;
  void* C;
  long long lda, ldb, ldc;
  int M, N, K, epi;
  const void* bias;
  void* C2;
  long long ldc2;
  float glu_limit;
  const int4* tile_map;      // {first row, end row, first row of B, column tile} per block, *num_tiles of them, or null
  const int* num_tiles;
  long long a_step, c_step;  // columns of A and C per head (blockIdx.z); B has N rows per head
  const void* gate;          // kEpiSigmoidGate: laid out like C
  long long ldg;
};

template <typename T>
__global__ void __launch_bounds__(256)
gemm_simt_kernel(const SimtParams p) {
  pdl_entry();
  __shared__ float as[kSgK][kSgTile + 4], bs[kSgK][kSgTile + 4];
  int m0 = blockIdx.y * kSgTile, n0 = blockIdx.x * kSgTile, M = p.M;
  long long b_row = static_cast<long long>(blockIdx.z) * p.N;
  if (p.tile_map) {
    if (static_cast<int>(blockIdx.x) >= *p.num_tiles) return;
    const int4 t = p.tile_map[blockIdx.x];
    m0 = t.x;
    M = t.y;
    b_row = t.z;
    n0 = t.w * kSgTile;
  }
  const int N = p.N, K = p.K, epi = p.epi;
  const long long lda = p.lda, ldb = p.ldb, ldc = p.ldc, ldc2 = p.ldc2, c_shift = blockIdx.z * p.c_step;
  const T* A = static_cast<const T*>(p.A) + blockIdx.z * p.a_step;
  const T* B = static_cast<const T*>(p.B) + b_row * ldb;
  const T* bias = static_cast<const T*>(p.bias);
  void *C = p.C, *C2 = p.C2;
  const float glu_limit = p.glu_limit;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kSgK) {
    for (int i = threadIdx.x; i < kSgTile * kSgK; i += 256) {
      const int r = i / kSgK, k = i % kSgK;
      as[k][r] = (m0 + r < M && k0 + k < K) ? to_f32(A[(m0 + r) * lda + k0 + k]) : 0.f;
      bs[k][r] = (n0 + r < N && k0 + k < K) ? to_f32(B[(n0 + r) * ldb + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kSgK; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&as[k][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&bs[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] += av[i] * bv[j];
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const long long m = m0 + ty * 4 + i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= N) continue;
      const float v = acc[i][j] + (bias ? to_f32(bias[n]) : 0.f);
      if (epi == kEpiBf16)
        static_cast<T*>(C)[m * ldc + c_shift + n] = from_f32<T>(v);
      else if (epi == kEpiSigmoidGate)
        static_cast<T*>(C)[m * ldc + c_shift + n] =
            from_f32<T>(v / (1.f + expf(-to_f32(static_cast<const T*>(p.gate)[m * p.ldg + c_shift + n]))));
      else if (epi == kEpiF32)
        static_cast<float*>(C)[m * ldc + n] = v;
      else if (epi == kEpiF32Accum || epi == kEpiF32Atomic)
        static_cast<float*>(C)[m * ldc + n] += v;
      else if (is_glu_epilogue(epi) && !(j & 1) && n + 1 < N) {
        const float u = acc[i][j | 1] + (bias ? to_f32(bias[n + 1]) : 0.f);
        const float y = epi == kEpiSwiGLU ? v / (1.f + expf(-v)) * u
                        : epi == kEpiGeGLU ? gelu_tanh_f(v) * u : clamped_glu(v, u, glu_limit);
        static_cast<T*>(C2)[m * ldc2 + (n >> 1)] = from_f32<T>(y);
      }
    }
  }
}

}  // namespace apb

extern "C" {
using namespace apb;

// epi: 0 C in the operand type, 1 C fp32, 2 / 3 C fp32 += (one writer per element); columns interleaved (gate, up): C2[m, n/2] =
// 4 silu(gate) * up, 9 gelu_tanh(gate) * up, 10 the clamped GLU (glu_limit > 0), in the operand type; 11 C = v * sigmoid(gate) in
// the operand type.  bias [N] (operand type) or null.
static int gemm_simt_impl(const SimtParams& p, int heads, int max_tiles, int dtype, cudaStream_t s) {
  if (p.M <= 0 || p.N <= 0 || p.K <= 0) return 0;
  if (is_glu_epilogue(p.epi) ? !p.C2 : !p.C) return kBadArgument;
  if (p.epi == kEpiClampGLU && !(p.glu_limit > 0.f)) return kBadArgument;
  if (p.epi == kEpiSigmoidGate && !p.gate) return kBadArgument;
  if (p.epi != kEpiBf16 && p.epi != kEpiF32 && p.epi != kEpiF32Accum && p.epi != kEpiF32Atomic && p.epi != kEpiSigmoidGate &&
      !is_glu_epilogue(p.epi))
    return kBadArgument;
  const dim3 grid = p.tile_map ? dim3(max_tiles) : dim3((p.N + kSgTile - 1) / kSgTile, (p.M + kSgTile - 1) / kSgTile, heads);
  APB_SERVE_DTYPE(dtype, return static_cast<int>(launch_kernel(gemm_simt_kernel<T>, grid, dim3(256), 0, s, p)));
}

int apb_gemm_simt(const void* A, const void* B, void* C, int M, int N, int K, long long lda, long long ldb,
                  long long ldc, int epi, const void* bias, void* C2, long long ldc2, float glu_limit, int dtype, cudaStream_t s) {
  return gemm_simt_impl(SimtParams{A, B, C, lda, ldb, ldc, M, N, K, epi, bias, C2, ldc2, glu_limit}, 1, 0, dtype, s);
}

// A tile table written by a kernel, 64 x 64 tiles: rows of A and C by group, B stacked.
int apb_gemm_simt_grouped(const void* A, const void* B, void* C, int M, int N, int K, long long lda, long long ldb, long long ldc,
                          int epi, void* C2, long long ldc2, float glu_limit, const void* tile_map, int max_tiles,
                          const int* num_tiles, int dtype, cudaStream_t s) {
  if (!tile_map || !num_tiles || max_tiles <= 0) return kBadArgument;
  return gemm_simt_impl(SimtParams{A, B, C, lda, ldb, ldc, M, N, K, epi, nullptr, C2, ldc2, glu_limit, static_cast<const int4*>(tile_map),
                                   num_tiles}, 1, max_tiles, dtype, s);
}

// C[:, h c_step + n] = A[:, h a_step + k] B[h N + n, k] for every head h; epi 0 or 11 (gate laid out like C).
int apb_gemm_simt_heads(const void* A, const void* B, void* C, int M, int N, int K, int heads, long long lda, long long ldb,
                        long long ldc, long long a_step, long long c_step, int epi, const void* gate, long long ldg, int dtype,
                        cudaStream_t s) {
  if (heads <= 0 || (epi != kEpiBf16 && epi != kEpiSigmoidGate)) return kBadArgument;
  return gemm_simt_impl(SimtParams{A, B, C, lda, ldb, ldc, M, N, K, epi, nullptr, nullptr, 0, 0.f, nullptr, nullptr, a_step, c_step,
                                   gate, ldg}, heads, 0, dtype, s);
}
}
