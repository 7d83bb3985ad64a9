// C = A B^T in true fp32 on the FMA pipe: the matrix product of the fp32 serving mode (exactness before speed; the
// bf16 product is tw_gemm_bf16). A [M, K], B [N, K], C [M, N], rows contiguous, any sizes. 64 x 64 tiles, 4 x 4
// outputs per thread.
#include "tw_host.h"
#include "tw_kernels.h"
#include "tw_common.cuh"

namespace tw {

constexpr int GF_T = 64, GF_K = 16;

__global__ void __launch_bounds__(256)
gemm_f32_kernel(const float* __restrict__ A, long long lda, const float* __restrict__ B, long long ldb,
                float* __restrict__ C, long long ldc, const float* __restrict__ bias, int M, int N, int K) {
  __shared__ float sa[GF_K][GF_T + 4], sb[GF_K][GF_T + 4];
  const int m0 = blockIdx.y * GF_T, n0 = blockIdx.x * GF_T;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += GF_K) {
    for (int i = threadIdx.x; i < GF_T * GF_K; i += 256) {
      const int r = i / GF_K, k = i - r * GF_K;
      const bool kin = k0 + k < K;
      sa[k][r] = (kin && m0 + r < M) ? A[(m0 + r) * lda + k0 + k] : 0.f;
      sb[k][r] = (kin && n0 + r < N) ? B[(n0 + r) * ldb + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < GF_K; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        a[i] = sa[k][ty * 4 + i];
        b[i] = sb[k][tx * 4 + i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n < N) C[m * ldc + n] = acc[i][j] + (bias != nullptr ? bias[n] : 0.f);
    }
  }
}

}  // namespace tw

extern "C" int tw_gemm_f32(const float* A, long long lda, const float* B, long long ldb, float* C, long long ldc,
                           const float* bias, int M, int N, int K, cudaStream_t stream) {
  if (M <= 0 || N <= 0) return 0;
  const dim3 grid((N + tw::GF_T - 1) / tw::GF_T, (M + tw::GF_T - 1) / tw::GF_T);
  if (grid.y > 65535) {
    tw::set_last_error("gemm_f32: %d rows are too many for one launch", M);
    return 1;
  }
  tw::gemm_f32_kernel<<<grid, 256, 0, stream>>>(A, lda, B, ldb, C, ldc, bias, M, N, K);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) {
    tw::set_last_error("gemm_f32 launch failed: %s", cudaGetErrorString(e));
    return 1;
  }
  return 0;
}
