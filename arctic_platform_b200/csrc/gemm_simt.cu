// GEMM on CUDA cores, fp32 accumulation: C[M,N] = A[M,K] * B[N,K]^T for fp32 operands (the fp32 engine: true 32-bit
// products, no TF32) and for bf16 operands whose row lengths are not multiples of 8, which the TMA-fed tensor-core
// kernels cannot address.  Same epilogues as those kernels where a serving step needs them.
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

template <typename T>
__global__ void __launch_bounds__(256)
gemm_simt_kernel(const T* __restrict__ A, const T* __restrict__ B, void* __restrict__ C, long long lda, long long ldb,
                 long long ldc, int M, int N, int K, int epi, const T* __restrict__ bias, void* __restrict__ C2,
                 long long ldc2, float glu_limit) {
  pdl_entry();
  __shared__ float as[kSgK][kSgTile + 4], bs[kSgK][kSgTile + 4];
  const int m0 = blockIdx.y * kSgTile, n0 = blockIdx.x * kSgTile;
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
        static_cast<T*>(C)[m * ldc + n] = from_f32<T>(v);
      else if (epi == kEpiF32)
        static_cast<float*>(C)[m * ldc + n] = v;
      else if (epi == kEpiF32Accum || epi == kEpiF32Atomic)
        static_cast<float*>(C)[m * ldc + n] += v;
      else if (is_glu_epilogue(epi) && !(j & 1) && n + 1 < N) {
        const float u = acc[i][j | 1] + (bias ? to_f32(bias[n + 1]) : 0.f);
        const float y = epi == kEpiGeGLU ? gelu_tanh_f(v) * u : clamped_glu(v, u, glu_limit);
        static_cast<T*>(C2)[m * ldc2 + (n >> 1)] = from_f32<T>(y);
      }
    }
  }
}

}  // namespace apb

extern "C" {
using namespace apb;

// epi: 0 C in the operand type, 1 C fp32, 2 / 3 C fp32 += (one writer per element), 9 columns interleaved (gate, up):
// C2[m, n/2] = gelu_tanh(gate) * up in the operand type, 10 the same with the clamped GLU (glu_limit > 0).  bias [N] (operand type) or null.
int apb_gemm_simt(const void* A, const void* B, void* C, int M, int N, int K, long long lda, long long ldb,
                  long long ldc, int epi, const void* bias, void* C2, long long ldc2, float glu_limit, int dtype, cudaStream_t s) {
  if (M <= 0 || N <= 0 || K <= 0) return 0;
  if (epi == kEpiGeGLU || epi == kEpiClampGLU ? !C2 : !C) return kBadArgument;
  if (epi == kEpiClampGLU && !(glu_limit > 0.f)) return kBadArgument;
  if (epi != kEpiBf16 && epi != kEpiF32 && epi != kEpiF32Accum && epi != kEpiF32Atomic && epi != kEpiGeGLU && epi != kEpiClampGLU)
    return kBadArgument;
  const dim3 grid((N + kSgTile - 1) / kSgTile, (M + kSgTile - 1) / kSgTile);
  APB_SERVE_DTYPE(dtype, return static_cast<int>(launch_kernel(
                             gemm_simt_kernel<T>, grid, dim3(256), 0, s, static_cast<const T*>(A),
                             static_cast<const T*>(B), C, lda, ldb, ldc, M, N, K, epi, static_cast<const T*>(bias), C2,
                             ldc2, glu_limit)));
}
}
