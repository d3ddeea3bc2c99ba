// y[T, N] = x[T, K] W[N, K]^T entirely in fp32 (no reduced-precision matrix mode): the projections of a runtime that is
// asked for 32-bit arithmetic.  64 x 64 tiles, 4 x 4 results per thread, K in steps of 16 through shared memory.  Three forms:
// one product, a product per head of strided operands, and a product per expert over expert-sorted rows.
#include "ops.h"
#include <cuda_runtime.h>

namespace {

constexpr int BT = 64, BN = 64, BK = 16;

// One tile: rows [t0, T) of x and y, features [n0, N) of w.
__device__ __forceinline__ void tile_f32(const float* __restrict__ x, int ldx, const float* __restrict__ w, float* __restrict__ y,
                                         int ldy, int t0, int n0, int T, int N, int K) {
  __shared__ float sx[BK][BT + 4], sw[BK][BN + 4];
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;   // loader: row of the tile, first of four K columns
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += BK) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int k = k0 + lk + j;
      sx[lk + j][lr] = (t0 + lr < T && k < K) ? x[(size_t)(t0 + lr) * ldx + k] : 0.f;
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
      if (t < T && n < N) y[(size_t)t * ldy + n] = acc[i][j];
    }
}

__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* __restrict__ x, int ldx, const float* __restrict__ w,
                                                       float* __restrict__ y, int ldy, int T, int N, int K, long long x_step,
                                                       long long w_step, long long y_step) {
  tile_f32(x + blockIdx.z * x_step, ldx, w + blockIdx.z * w_step, y + blockIdx.z * y_step, ldy, blockIdx.y * BT, blockIdx.x * BN, T,
           N, K);
}

__global__ void __launch_bounds__(256) gemm_f32_grouped_kernel(const float* __restrict__ x, const float* __restrict__ w,
                                                               float* __restrict__ y, const int4* __restrict__ work,
                                                               const int* __restrict__ num_work, int N, int K) {
  for (int i = blockIdx.x; i < *num_work; i += gridDim.x) {
    const int4 k = work[i];                                // group, feature tile, first row, rows
    tile_f32(x + (size_t)k.z * K, K, w + (size_t)k.x * N * K, y + (size_t)k.z * N, N, 0, k.y * BN, k.w, N, K);
  }
}

}  // namespace

extern "C" int b200_gemm_f32(const float* x, const float* w, float* y, int T, int N, int K, cudaStream_t stream) {
  if (T <= 0 || N <= 0 || K <= 0 || (T + BT - 1) / BT > 65535) return -6;
  gemm_f32_kernel<<<dim3((N + BN - 1) / BN, (T + BT - 1) / BT), 256, 0, stream>>>(x, K, w, y, N, T, N, K, 0, 0, 0);
  return (int)cudaGetLastError();
}

// y[t, h, :N] = x[t, h, :K] W[h]^T for H heads: rows `ldx` / `ldy` apart, heads `x_head` / `y_head` apart, W [H, N, K].
extern "C" int b200_head_linear_f32(const float* x, int ldx, int x_head, const float* w, float* y, int ldy, int y_head, int T, int H,
                                    int N, int K, cudaStream_t stream) {
  if (T <= 0 || H <= 0 || H > 65535 || N <= 0 || K <= 0 || (T + BT - 1) / BT > 65535) return -6;
  gemm_f32_kernel<<<dim3((N + BN - 1) / BN, (T + BT - 1) / BT, H), 256, 0, stream>>>(x, ldx, w, y, ldy, T, N, K, x_head,
                                                                                      (long long)N * K, y_head);
  return (int)cudaGetLastError();
}

// Expert-sorted rows x [rows, K], W [groups, N, K], y [rows, N]; the work table is b200_moe_plan's for tiles of 64 rows and
// ceil(N / 64) feature tiles.
extern "C" int b200_gemm_f32_grouped(const float* x, const float* w, float* y, int N, int K, const void* work, const int* num_work,
                                     int max_work, cudaStream_t stream) {
  if (N <= 0 || K <= 0 || max_work <= 0) return -6;
  gemm_f32_grouped_kernel<<<max_work < 1184 ? max_work : 1184, 256, 0, stream>>>(x, w, y, reinterpret_cast<const int4*>(work),
                                                                                 num_work, N, K);
  return (int)cudaGetLastError();
}
