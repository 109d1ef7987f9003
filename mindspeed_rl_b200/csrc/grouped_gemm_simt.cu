// Grouped (per-expert) GEMM on the CUDA cores: C[r, :] = A[r, :] * B_e^T for the rows of expert e.
//
// Serves what the tensor-core kernel (moe_gemm_tcgen05.cu) does not: fp32 operands (true 32-bit products) and
// bf16 operands whose inner size or strides do not fit its tiles.  A [P, K] is grouped by expert in 128-row
// tiles (`tile_expert`), B holds the experts' [N, K] weights one after the other.  64 x 64 output tiles, 16-deep
// slices in shared memory, 4 x 4 results per thread, fp32 accumulation; sub-tiles of pad rows are skipped.
#include "dtype_utils.cuh"

namespace msrl {

constexpr int GS_BM = 64, GS_BN = 64, GS_BK = 16;

template <typename T>
__global__ void __launch_bounds__(256)
grouped_gemm_simt_kernel(const T* A, const T* B, T* C, int N, int K, const int* tile_expert, const int* counts,
                         const int* offsets) {
  __shared__ float sA[GS_BK][GS_BM + 4], sB[GS_BK][GS_BN + 4];
  const int m0 = blockIdx.y * GS_BM, n0 = blockIdx.x * GS_BN;
  const int e = tile_expert[m0 / 128];
  if (e < 0) return;
  const int end = offsets[e] + counts[e];              // first pad row of the segment
  if (m0 >= end) return;
  const T* Be = B + (long long)e * N * K;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += GS_BK) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int idx = threadIdx.x + i * 256;           // 64 rows x 16 columns, columns fastest
      const int r = idx >> 4, c = idx & 15;
      sA[c][r] = (m0 + r < end && k0 + c < K) ? ldf(A + (long long)(m0 + r) * K + k0 + c) : 0.f;
      sB[c][r] = (n0 + r < N && k0 + c < K) ? ldf(Be + (long long)(n0 + r) * K + k0 + c) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < GS_BK; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        a[i] = sA[k][ty * 4 + i];
        b[i] = sB[k][tx * 4 + i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] += a[i] * b[j];
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int r = m0 + ty * 4 + i, c = n0 + tx * 4 + j;
      if (r < end && c < N) stf(C + (long long)r * N + c, acc[i][j]);
    }
}

}  // namespace msrl

using namespace msrl;

MSRL_API int msrl_grouped_gemm_simt(const void* A, const void* B, void* C, int rows, int N, int K,
                                    const int* tile_expert, const int* counts, const int* offsets, int is_f32,
                                    cudaStream_t st) {
  if (rows == 0 || N == 0) return 0;
  if (rows % 128 != 0) return (int)cudaErrorInvalidValue;
  const dim3 grid((unsigned)((N + GS_BN - 1) / GS_BN), (unsigned)(rows / GS_BM));
  if (grid.y > 65535u) return (int)cudaErrorInvalidValue;
  if (is_f32)
    grouped_gemm_simt_kernel<float><<<grid, 256, 0, st>>>((const float*)A, (const float*)B, (float*)C, N, K,
                                                          tile_expert, counts, offsets);
  else
    grouped_gemm_simt_kernel<__nv_bfloat16><<<grid, 256, 0, st>>>((const __nv_bfloat16*)A, (const __nv_bfloat16*)B,
                                                                  (__nv_bfloat16*)C, N, K, tile_expert, counts, offsets);
  return (int)cudaGetLastError();
}
