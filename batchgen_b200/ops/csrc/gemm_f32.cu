// fp32 GEMM on the CUDA cores (no reduced-precision mode), dense, ragged grouped, and per head over columns of one matrix:
// D[m, n] = A[m, :] . B[n, :].
//
// The 32-bit form of a model on a GPU: it serves as the exact run that the 16-bit form is measured against, so it is
// written for exactness and any shape (tails in M, N and K are guarded), not for throughput.  64 x 64 tiles, 256 threads
// with 4 x 4 outputs each, K in steps of 16 through shared memory.
#include "common.cuh"

namespace bg {
namespace f32gemm {

constexpr int TM = 64, TN = 64, TK = 16;

// grouped: blockIdx.z is the group; its rows are offsets[g] .. offsets[g] + counts[g].  Per head (head_a, head_d: columns between the
// heads of A and D): blockIdx.z is the head.
__global__ void __launch_bounds__(256)
gemm_kernel(const float* __restrict__ A, int lda, const float* __restrict__ B, int ldb, float* __restrict__ D, int ldd,
            const int* __restrict__ offsets, const int* __restrict__ counts, int M, int N, int K, int head_a, int head_d) {
  __shared__ float As[TK][TM + 4], Bs[TK][TN + 4];
  const int g = blockIdx.z;
  int m_lo = 0, m_hi = M;
  if (offsets != nullptr) {
    m_lo = offsets[g];
    m_hi = min(M, m_lo + (counts != nullptr ? counts[g] : offsets[g + 1] - m_lo));
    B += (size_t)g * N * ldb;
  } else if (head_d > 0) {
    A += (size_t)g * head_a;
    B += (size_t)g * N * ldb;
    D += (size_t)g * head_d;
  }
  const int m0 = m_lo + blockIdx.y * TM, n0 = blockIdx.x * TN;
  if (m0 >= m_hi) return;
  const int tid = threadIdx.x, tx = tid % 16, ty = tid / 16;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += TK) {
#pragma unroll
    for (int i = 0; i < TM * TK / 256; ++i) {
      const int e = tid + i * 256, k = e % TK, m = e / TK;
      As[k][m] = (m0 + m < m_hi && k0 + k < K) ? A[(size_t)(m0 + m) * lda + k0 + k] : 0.f;
      Bs[k][m] = (n0 + m < N && k0 + k < K) ? B[(size_t)(n0 + m) * ldb + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < TK; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = As[k][ty * 4 + i]; b[i] = Bs[k][tx * 4 + i]; }
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
    if (m >= m_hi) break;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n < N) D[(size_t)m * ldd + n] = acc[i][j];
    }
  }
}

}  // namespace f32gemm
}  // namespace bg

extern "C" int bg_gemm_f32(const float* A, int lda, const float* B, int ldb, float* D, int ldd, const int* offsets,
                           const int* counts, int groups, int M, int max_rows, int N, int K, cudaStream_t stream) {
  using namespace bg::f32gemm;
  if (M <= 0 || N <= 0) return 0;
  if (K <= 0 || lda < K || ldb < K || ldd < N || (offsets != nullptr && groups <= 0)) return -1;
  const int rows = offsets != nullptr ? max_rows : M;
  dim3 grid((N + TN - 1) / TN, (rows + TM - 1) / TM, offsets != nullptr ? groups : 1);
  if (grid.y > 65535 || grid.z > 65535) return -1;
  gemm_kernel<<<grid, 256, 0, stream>>>(A, lda, B, ldb, D, ldd, offsets, counts, M, N, K, 0, 0);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

// D[t, h, n] = A[t, h, :K] . W[h, n, :K]: element (t, h, k) of A at t * lda + h * head_a + k, of D at t * ldd + h * head_d + n
extern "C" int bg_head_gemm_f32(const float* A, int lda, int head_a, const float* W, int ldw, float* D, int ldd, int head_d, int T, int H, int N,
                                int K, cudaStream_t stream) {
  using namespace bg::f32gemm;
  if (T <= 0 || N <= 0 || H <= 0) return 0;
  if (K <= 0 || ldw < K || head_a < K || head_d < N) return -1;
  dim3 grid((N + TN - 1) / TN, (T + TM - 1) / TM, H);
  if (grid.y > 65535 || grid.z > 65535) return -1;
  gemm_kernel<<<grid, 256, 0, stream>>>(A, lda, W, ldw, D, ldd, nullptr, nullptr, T, N, K, head_a, head_d);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}
