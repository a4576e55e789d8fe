// True fp32 GEMM (no TF32): C[M, N] = A[M, K] * B[N, K]^T, every product and sum an fp32 FMA. It serves the fp32 mode
// of the layer-stack models, whose purpose is exactness; the 16-bit path is the tensor-core GEMM of gemm.cu / gemm2.cu.
// 64 x 64 tile, 256 threads, 4 x 4 outputs each; the k order is the same for every M, so a row does not depend on the
// batch it is in.
#include "common.cuh"

namespace {
constexpr int TM = 64, TN = 64, TK = 16;

__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* __restrict__ A, const float* __restrict__ B, float* __restrict__ C,
                                                       int M, int N, int K, long long lda, long long ldb, long long ldc) {
  __shared__ float sA[TK][TM + 4], sB[TK][TN + 4];
  const int m0 = blockIdx.y * TM, n0 = blockIdx.x * TN;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lk = threadIdx.x & 15, lr = threadIdx.x >> 4;      // loader: column k, rows lr + 16 i
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += TK) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = lr + 16 * i, k = k0 + lk;
      sA[lk][r] = (m0 + r < M && k < K) ? A[(long long)(m0 + r) * lda + k] : 0.f;
      sB[lk][r] = (n0 + r < N && k < K) ? B[(long long)(n0 + r) * ldb + k] : 0.f;
    }
    __syncthreads();
    float part[4][4] = {};                 // 16 products at a time: two short sums lose less than one long one
#pragma unroll
    for (int k = 0; k < TK; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = sA[k][ty * 4 + i]; b[i] = sB[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) part[i][j] = fmaf(a[i], b[j], part[i][j]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] += part[i][j];
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) break;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n < N) C[(long long)m * ldc + n] = acc[i][j];
    }
  }
}
}  // namespace

DLTI_API int dlti_gemm_f32(const float* A, const float* B, float* C, int M, int N, int K, long long lda, long long ldb, long long ldc,
                           cudaStream_t st) {
  if (M <= 0 || N <= 0) return 0;
  if (K <= 0 || (M + TM - 1) / TM > 65535) return DLTI_ERR_BAD_ARG;
  gemm_f32_kernel<<<dim3((N + TN - 1) / TN, (M + TM - 1) / TM), 256, 0, st>>>(A, B, C, M, N, K, lda, ldb, ldc);
  dlti_count_launch();
  return (int)cudaGetLastError();
}
