// C = A B^T in true fp32 on the FMA pipe: the matrix product of the fp32 serving mode (exactness before speed; the
// bf16 product is tw_gemm_bf16). A [M, K], B [N, K], C [M, N], rows contiguous, any sizes. 64 x 64 tiles, 4 x 4
// outputs per thread. Grouped form: every tile_rows rows of A belong to one expert, whose N rows of B they take; rows may
// be scaled.
#include "tw_host.h"
#include "tw_kernels.h"
#include "tw_common.cuh"

namespace tw {

constexpr int GF_T = 64, GF_K = 16;

__global__ void __launch_bounds__(256)
gemm_f32_kernel(const float* __restrict__ A, long long lda, const float* __restrict__ B, long long ldb,
                float* __restrict__ C, long long ldc, const float* __restrict__ bias, int M, int N, int K,
                const int* __restrict__ tile_expert, const int* __restrict__ num_tiles, int tile_rows, int n_per_expert,
                const float* __restrict__ row_scale) {
  __shared__ float sa[GF_K][GF_T + 4], sb[GF_K][GF_T + 4];
  const int m0 = blockIdx.y * GF_T, n0 = blockIdx.x * GF_T;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  if (tile_expert != nullptr) {
    const int tile = m0 / tile_rows;
    if (tile >= *num_tiles) return;
    B += static_cast<long long>(tile_expert[tile]) * n_per_expert * ldb;
  }
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
      if (n < N) C[m * ldc + n] = (acc[i][j] + (bias != nullptr ? bias[n] : 0.f)) * (row_scale != nullptr ? row_scale[m] : 1.f);
    }
  }
}

}  // namespace tw

static int gemm_f32(const float* A, long long lda, const float* B, long long ldb, float* C, long long ldc,
                    const float* bias, int M, int N, int K, const int* tile_expert, const int* num_tiles, int tile_rows,
                    int n_per_expert, const float* row_scale, cudaStream_t stream) {
  if (M <= 0 || N <= 0) return 0;
  const dim3 grid((N + tw::GF_T - 1) / tw::GF_T, (M + tw::GF_T - 1) / tw::GF_T);
  if (grid.y > 65535) {
    tw::set_last_error("gemm_f32: %d rows are too many for one launch", M);
    return 1;
  }
  tw::gemm_f32_kernel<<<grid, 256, 0, stream>>>(A, lda, B, ldb, C, ldc, bias, M, N, K, tile_expert, num_tiles, tile_rows,
                                               n_per_expert, row_scale);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) {
    tw::set_last_error("gemm_f32 launch failed: %s", cudaGetErrorString(e));
    return 1;
  }
  return 0;
}

extern "C" int tw_gemm_f32(const float* A, long long lda, const float* B, long long ldb, float* C, long long ldc,
                           const float* bias, int M, int N, int K, cudaStream_t stream) {
  return gemm_f32(A, lda, B, ldb, C, ldc, bias, M, N, K, nullptr, nullptr, 0, 0, nullptr, stream);
}

extern "C" int tw_gemm_f32_grouped(const float* A, long long lda, const float* B, long long ldb, float* C, long long ldc,
                                   int M, int N, int K, const int* tile_expert, const int* num_tiles, int tile_rows,
                                   int n_per_expert, const float* row_scale, cudaStream_t stream) {
  if (tile_expert == nullptr || num_tiles == nullptr || tile_rows <= 0 || tile_rows % tw::GF_T != 0) {
    tw::set_last_error("gemm_f32_grouped: needs the tile -> expert map, tiles of a multiple of %d rows", tw::GF_T);
    return 1;
  }
  return gemm_f32(A, lda, B, ldb, C, ldc, nullptr, M, N, K, tile_expert, num_tiles, tile_rows, n_per_expert, row_scale,
                  stream);
}
