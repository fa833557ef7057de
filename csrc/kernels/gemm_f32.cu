// True 32-bit matrix product  out[b][m][n] = sum_k A[b][m][k] * B[b][n][k]  (fp32 FMA, no tensor cores): the projections of
// 32-bit passes.  A holds activation rows, B weight rows, both with k contiguous.
#include "ds41_stack.cuh"

namespace ds41 {

constexpr int kF32Tile = 64;
constexpr int kF32K = 16;

__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* A, const float* B, float* out, int M, int N, int K,
                                                       long long lda, long long ldb, long long ldo, long long sa,
                                                       long long sb, long long so, const int* batch_map,
                                                       const int* n_active) {
  __shared__ float as[kF32K][kF32Tile + 4];
  __shared__ float bs[kF32K][kF32Tile + 4];
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int n0 = blockIdx.x * kF32Tile, m0 = blockIdx.y * kF32Tile;
  pdl_launch_dependents();
  pdl_wait();
  if (n_active != nullptr && static_cast<int>(blockIdx.z) >= *n_active) return;
  A += blockIdx.z * sa;
  B += (batch_map != nullptr ? batch_map[blockIdx.z] : static_cast<int>(blockIdx.z)) * sb;
  out += blockIdx.z * so;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kF32K) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int row = ty + 16 * j, k = k0 + tx;
      as[tx][row] = m0 + row < M && k < K ? A[(m0 + row) * lda + k] : 0.f;
      bs[tx][row] = n0 + row < N && k < K ? B[(n0 + row) * ldb + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kF32K; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        a[j] = as[k][ty * 4 + j];
        b[j] = bs[k][tx * 4 + j];
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
      if (n < N) out[m * ldo + n] = acc[i][j];
    }
  }
}

}  // namespace ds41

using namespace ds41;

extern "C" int ds41_gemm_f32(const float* A, const float* B, float* out, int M, int N, int K, long long lda, long long ldb,
                             long long ldo, int batch, long long a_batch_stride, long long b_batch_stride,
                             long long out_batch_stride, const int* batch_map, const int* n_active, void* stream) {
  if (A == nullptr || B == nullptr || out == nullptr || M <= 0 || N <= 0 || K <= 0 || batch <= 0 || batch > 65535 ||
      lda < K || ldb < K || ldo < N || (M + kF32Tile - 1) / kF32Tile > 65535)
    return cudaErrorInvalidValue;
  const dim3 grid((N + kF32Tile - 1) / kF32Tile, (M + kF32Tile - 1) / kF32Tile, batch);
  return launch_pdl(gemm_f32_kernel, grid, dim3(256), 0, static_cast<cudaStream_t>(stream), A, B, out, M, N, K, lda, ldb,
                    ldo, a_batch_stride, b_batch_stride, out_batch_stride, batch_map, n_active);
}
