// fp32 GEMM for the models' 32-bit mode: C[M,N] = A[M,K] * B[N,K]^T, true fp32 products and sums (no TF32).
//
// A 64 x 64 tile per CTA of 256 threads, 4 x 4 outputs per thread, K in steps of 16 through shared memory. Any M, N, K
// and leading dimensions. The sum over K runs in the same order for every element whatever M is, so a row's result does
// not depend on how many other rows share the call.
#include "b200/host.h"
#include "b200/primitives.cuh"

namespace b200 {

constexpr int kFT = 64, kFK = 16;

__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* __restrict__ A, const float* __restrict__ B,
                                                       float* __restrict__ C, int M, int N, int K, int lda, int ldb, int ldc) {
  __shared__ float sa[kFK][kFT + 4], sb[kFK][kFT + 4];
  const int m0 = blockIdx.y * kFT, n0 = blockIdx.x * kFT;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  griddep_launch_dependents();
  griddep_wait();
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kFK) {
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const int r = ty + 16 * u, k = k0 + tx;
      sa[tx][r] = (m0 + r < M && k < K) ? A[static_cast<size_t>(m0 + r) * lda + k] : 0.f;
      sb[tx][r] = (n0 + r < N && k < K) ? B[static_cast<size_t>(n0 + r) * ldb + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kFK; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&sa[k][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&sb[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m < M && n < N) C[static_cast<size_t>(m) * ldc + n] = acc[i][j];
    }
}

}  // namespace b200

using namespace b200;

B200_API int b200_gemm_f32(const float* A, const float* B, float* C, int M, int N, int K, int lda, int ldb, int ldc,
                           void* stream) {
  B200_REQUIRE(M > 0 && N > 0 && K > 0, "empty problem %dx%dx%d", M, N, K);
  B200_REQUIRE(lda >= K && ldb >= K && ldc >= N, "leading dimensions are smaller than the rows");
  const dim3 grid((N + kFT - 1) / kFT, (M + kFT - 1) / kFT);
  B200_REQUIRE(grid.y <= 65535, "M (%d) is too large", M);
  B200_CHECK_CUDA(launch_pdl(gemm_f32_kernel, grid, dim3(256), 0, static_cast<cudaStream_t>(stream), A, B, C, M, N, K, lda, ldb, ldc));
  return kOk;
}
