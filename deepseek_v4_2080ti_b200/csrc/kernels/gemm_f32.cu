// y[T, N] = x[T, K] W[N, K]^T entirely in fp32 (no reduced-precision matrix mode): the projections of a runtime that is
// asked for 32-bit arithmetic.  64 x 64 tiles, 4 x 4 results per thread, K in steps of 16 through shared memory.
#include "ops.h"
#include <cuda_runtime.h>

namespace {

constexpr int BT = 64, BN = 64, BK = 16;

__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* __restrict__ x, const float* __restrict__ w,
                                                       float* __restrict__ y, int T, int N, int K) {
  __shared__ float sx[BK][BT + 4], sw[BK][BN + 4];
  const int t0 = blockIdx.y * BT, n0 = blockIdx.x * BN;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;   // loader: row of the tile, first of four K columns
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += BK) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int k = k0 + lk + j;
      sx[lk + j][lr] = (t0 + lr < T && k < K) ? x[(size_t)(t0 + lr) * K + k] : 0.f;
      sw[lk + j][lr] = (n0 + lr < N && k < K) ? w[(size_t)(n0 + lr) * K + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < BK; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = sx[k][ty * 4 + i]; b[i] = sw[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int t = t0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (t < T && n < N) y[(size_t)t * N + n] = acc[i][j];
    }
}

}  // namespace

extern "C" int b200_gemm_f32(const float* x, const float* w, float* y, int T, int N, int K, cudaStream_t stream) {
  if (T <= 0 || N <= 0 || K <= 0 || (T + BT - 1) / BT > 65535) return -6;
  gemm_f32_kernel<<<dim3((N + BN - 1) / BN, (T + BT - 1) / BT), 256, 0, stream>>>(x, w, y, T, N, K);
  return (int)cudaGetLastError();
}
