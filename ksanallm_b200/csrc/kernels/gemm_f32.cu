// True 32-bit GEMM on the CUDA cores, for models served entirely in fp32 (no reduced-precision tensor-core mode):
// D[M,N] = A[M,K] W[N,K]^T (+ bias[N]) (+ residual[M,N]). 64 x 64 tiles, 4 x 4 outputs per thread, K walked in steps of
// 16 in ascending order for every shape, so that a row's result does not depend on the other rows of the call.
#include "pdl.cuh"
#include <cuda_runtime.h>

namespace ksana {

constexpr int kSgTile = 64, kSgK = 16, kSgThreads = 256;

__global__ void __launch_bounds__(kSgThreads)
gemm_f32_kernel(const float* __restrict__ A, int lda, const float* __restrict__ W, int ldw, float* __restrict__ D, int ldd,
                const float* __restrict__ bias, const float* __restrict__ residual, int ldr, int M, int N, int K,
                long long a_batch, long long w_batch, long long d_batch, const float* __restrict__ gate, int ldg, long long g_batch,
                const int* __restrict__ tile_expert, int num_experts) {
  pdl_trigger();
  pdl_wait();
  if (tile_expert) {                    // rows of one expert per 128-row tile; W stacks the experts' N rows
    const int e = tile_expert[blockIdx.y * kSgTile / 128];
    if (e < 0 || e >= num_experts) return;
    W += static_cast<size_t>(e) * N * ldw;
  }
  A += blockIdx.z * a_batch;
  W += blockIdx.z * w_batch;
  D += blockIdx.z * d_batch;
  if (gate) gate += blockIdx.z * g_batch;
  __shared__ float as[kSgK][kSgTile + 4], ws[kSgK][kSgTile + 4];
  const int m0 = blockIdx.y * kSgTile, n0 = blockIdx.x * kSgTile;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;          // staging: one row, four consecutive k per thread
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kSgK) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int k = k0 + lk + e;
      as[lk + e][lr] = (m0 + lr < M && k < K) ? A[static_cast<size_t>(m0 + lr) * lda + k] : 0.f;
      ws[lk + e][lr] = (n0 + lr < N && k < K) ? W[static_cast<size_t>(n0 + lr) * ldw + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kSgK; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) { a[e] = as[k][ty * 4 + e]; b[e] = ws[k][tx * 4 + e]; }
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
      if (n >= N) continue;
      float v = acc[i][j];
      if (bias) v += bias[n];
      if (residual) v += residual[static_cast<size_t>(m) * ldr + n];
      if (gate) v /= 1.f + __expf(-gate[static_cast<size_t>(m) * ldg + n]);
      D[static_cast<size_t>(m) * ldd + n] = v;
    }
  }
}

}  // namespace ksana

using namespace ksana;

extern "C" int ksana_gemm_f32(const float* A, int lda, const float* W, int ldw, float* D, int ldd, const float* bias,
                              const float* residual, int ldr, int M, int N, int K, cudaStream_t st) {
  if (M <= 0 || N <= 0 || K <= 0) return 0;
  const dim3 grid((N + kSgTile - 1) / kSgTile, (M + kSgTile - 1) / kSgTile);
  if (grid.y > 65535u) return -10;
  return launch_pdl(gemm_f32_kernel, grid, dim3(kSgThreads), 0, st, A, lda, W, ldw, D, ldd, bias, residual, ldr, M, N, K,
                    0LL, 0LL, 0LL, static_cast<const float*>(nullptr), 0, 0LL, static_cast<const int*>(nullptr), 0) == cudaSuccess ? 0 : -4;
}

// D[b] = A[b] W[b]^T for every b, with a gate times sigmoid(gate[b]) element by element; a_batch / w_batch / d_batch: elements between batch entries.
extern "C" int ksana_gemm_f32_batched(const float* A, int lda, long long a_batch, const float* W, int ldw, long long w_batch,
                                      float* D, int ldd, long long d_batch, int batch, int M, int N, int K, const float* gate,
                                      int ldg, long long g_batch, cudaStream_t st) {
  if (M <= 0 || N <= 0 || K <= 0 || batch <= 0) return 0;
  const dim3 grid((N + kSgTile - 1) / kSgTile, (M + kSgTile - 1) / kSgTile, batch);
  if (grid.y > 65535u || batch > 65535) return -10;
  const float* none = nullptr;
  return launch_pdl(gemm_f32_kernel, grid, dim3(kSgThreads), 0, st, A, lda, W, ldw, D, ldd, none, none, 0, M, N, K, a_batch, w_batch,
                    d_batch, gate, ldg, g_batch, static_cast<const int*>(nullptr), 0) == cudaSuccess ? 0 : -4;
}

// Mixture of experts: 128-row tiles of A, tile i times W[tile_expert[i]] (W [E * N, K]; a negative entry: an unused tile).
extern "C" int ksana_gemm_grouped_f32(const float* A, int lda, const float* W, int ldw, float* D, int ldd, int M_cap, int N, int K,
                                      int E, const int* tile_expert, cudaStream_t st) {
  if (M_cap <= 0 || N <= 0 || K <= 0 || E <= 0) return 0;
  if (M_cap % 128 || !tile_expert || M_cap / kSgTile > 65535) return -10;
  const dim3 grid((N + kSgTile - 1) / kSgTile, M_cap / kSgTile);
  const float* none = nullptr;
  return launch_pdl(gemm_f32_kernel, grid, dim3(kSgThreads), 0, st, A, lda, W, ldw, D, ldd, none, none, 0, M_cap, N, K, 0LL, 0LL, 0LL,
                    none, 0, 0LL, tile_expert, E) == cudaSuccess ? 0 : -4;
}
