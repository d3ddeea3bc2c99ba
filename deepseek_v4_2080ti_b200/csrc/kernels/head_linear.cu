// A small matrix per head on the rows of a short batch: y[t, h, :N] = x[t, h, :K] W[h]^T in bf16 with fp32 sums (the up
// projections of latent attention around its absorbed form).  The weights are streamed once per 64 rows; operands go from
// global memory straight into tensor-core fragments: the order of the dimensions inside a dot product is free, so a lane takes
// 16 contiguous bytes of a row as its share of two k-steps.  Prompt-sized batches use the big GEMMs instead.
//
// rows_linear_f32: the same for one matrix with few rows of its own and fp32 results (a router): more warps share K, because
// the features alone would occupy a handful of SMs.  rows_token_gate: that with gelu and the token's side embedding as epilogue.
#include <cuda_bf16.h>
#include <stdint.h>
#include "gelu.cuh"
#include "launch.h"
#include "ops.h"

namespace {
using namespace b200;

__device__ __forceinline__ void mma_bf16(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

constexpr int NW = 16;                     // features per block; the warps share K

__device__ __forceinline__ void store2(__nv_bfloat16* p, int n, int N, float a, float b) {        // N is even
  *reinterpret_cast<__nv_bfloat162*>(p + n) = __floats2bfloat162_rn(a, b);
}
__device__ __forceinline__ void store2(float* p, int n, int N, float a, float b) {
  p[n] = a;
  if (n + 1 < N) p[n + 1] = b;
}

// Where a pair of features of a row goes: stored as it is, or behind gelu and times the row's token's embedding.
template <typename Out>
struct Plain {
  Out* y;
  int ldy, y_head;
  __device__ __forceinline__ void put(int t, int h, int n, int N, float a, float b) const { store2(y + (size_t)t * ldy + h * y_head, n, N, a, b); }
};
struct TokenGate {
  __nv_bfloat16* y;
  const __nv_bfloat16* table;      // [vocab, ld_table], this projection's part from column `col` on
  const int* ids;
  int ldy, ld_table, col, vocab;
  __device__ __forceinline__ void put(int t, int, int n, int N, float a, float b) const {
    const int id = ids[t];
    float2 e = make_float2(0.f, 0.f);
    if (id >= 0 && id < vocab) e = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(table + (size_t)id * ld_table + col + n));
    store2(y + (size_t)t * ldy, n, N, gelu_tanh(a) * e.x, gelu_tanh(b) * e.y);
  }
};

// grid (features / 16, heads, rows / (16 MT)); K % 16 == 0 (32-wide chunks, the last may be half).  The warps'
// sums are added up through shared memory.
template <int MT, int WARPS, typename Sink>
__global__ void __launch_bounds__(WARPS * 32)
head_linear_kernel(const __nv_bfloat16* __restrict__ x, int ldx, int x_head, const __nv_bfloat16* __restrict__ w,
                   Sink sink, int T, int N, int K) {
  __shared__ float red[WARPS][MT][2][4][32];
  pdl_grid_trigger();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gr = lane >> 2, kk = lane & 3;
  const int h = blockIdx.y, n0 = blockIdx.x * NW, t0 = blockIdx.z * 16 * MT;
  const uint4 zero = make_uint4(0, 0, 0, 0);
  const __nv_bfloat16* wh = w + (size_t)h * N * K;
  float acc[MT][2][4] = {};
  pdl_grid_wait();
#pragma unroll 4
  for (int k0 = warp * 32; k0 < K; k0 += 32 * WARPS) {
    const int k = k0 + kk * 8;
    uint4 b[2];
#pragma unroll
    for (int nb = 0; nb < 2; ++nb) {
      const int n = n0 + nb * 8 + gr;
      b[nb] = n < N && k < K ? *reinterpret_cast<const uint4*>(wh + (size_t)n * K + k) : zero;
    }
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      const int ta = t0 + mt * 16 + gr, tb = ta + 8;
      const uint4 a0 = ta < T && k < K ? *reinterpret_cast<const uint4*>(x + (size_t)ta * ldx + h * x_head + k) : zero;
      const uint4 a1 = tb < T && k < K ? *reinterpret_cast<const uint4*>(x + (size_t)tb * ldx + h * x_head + k) : zero;
#pragma unroll
      for (int nb = 0; nb < 2; ++nb) {
        mma_bf16(acc[mt][nb], a0.x, a1.x, a0.y, a1.y, b[nb].x, b[nb].y);
        mma_bf16(acc[mt][nb], a0.z, a1.z, a0.w, a1.w, b[nb].z, b[nb].w);
      }
    }
  }
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nb = 0; nb < 2; ++nb)
#pragma unroll
      for (int i = 0; i < 4; ++i) red[warp][mt][nb][i][lane] = acc[mt][nb][i];
  __syncthreads();
  // item: (row tile, feature half, row half), a pair of features per lane
  for (int item = warp; item < MT * 4; item += WARPS) {
    const int mt = item >> 2, nb = (item >> 1) & 1, hf = item & 1;
    float v0 = 0.f, v1 = 0.f;
#pragma unroll
    for (int u = 0; u < WARPS; ++u) {
      v0 += red[u][mt][nb][hf * 2][lane];
      v1 += red[u][mt][nb][hf * 2 + 1][lane];
    }
    const int t = t0 + mt * 16 + gr + hf * 8, n = n0 + nb * 8 + kk * 2;
    if (t < T && n < N) sink.put(t, h, n, N, v0, v1);
  }
}

template <int WARPS, typename Sink>
int run(const void* x, int ldx, int x_head, const void* w, const Sink& sink, int T, int H, int N, int K, cudaStream_t stream) {
  const int mt = T <= 16 ? 1 : T <= 32 ? 2 : 4;
  if ((T + 16 * mt - 1) / (16 * mt) > 65535) return -6;
  const dim3 grid((N + NW - 1) / NW, H, (T + 16 * mt - 1) / (16 * mt)), block(WARPS * 32);
  auto xp = reinterpret_cast<const __nv_bfloat16*>(x);
  auto wp = reinterpret_cast<const __nv_bfloat16*>(w);
  if (mt == 1) return (int)launch_pdl(head_linear_kernel<1, WARPS, Sink>, grid, block, 0, stream, xp, ldx, x_head, wp, sink, T, N, K);
  if (mt == 2) return (int)launch_pdl(head_linear_kernel<2, WARPS, Sink>, grid, block, 0, stream, xp, ldx, x_head, wp, sink, T, N, K);
  if constexpr (WARPS <= 8)
    return (int)launch_pdl(head_linear_kernel<4, WARPS, Sink>, grid, block, 0, stream, xp, ldx, x_head, wp, sink, T, N, K);
  return -6;
}

// One matrix: few blocks, so many warps share K (their sums fit into shared memory for up to 32 rows at a time).
template <typename Sink>
int run_rows(const void* x, int ldx, const void* w, const Sink& sink, int T, int N, int K, cudaStream_t stream) {
  return T <= 32 && K >= 1024 ? run<16>(x, ldx, 0, w, sink, T, 1, N, K, stream) : run<8>(x, ldx, 0, w, sink, T, 1, N, K, stream);
}

}  // namespace

// Rows `ldx` / `ldy` elements apart, heads `x_head` / `y_head` apart (multiples of 8), W [H, N, K]; N even, K % 16 == 0.
extern "C" int b200_head_linear(const void* x, int ldx, int x_head, const void* w, void* y, int ldy, int y_head, int T, int H, int N,
                                int K, cudaStream_t stream) {
  if (T <= 0 || H <= 0 || H > 65535 || N <= 0 || (N & 1) || K <= 0 || (K & 15) || ((ldx | x_head | ldy | y_head) & 7)) return -6;
  return run<4>(x, ldx, x_head, w, Plain<__nv_bfloat16>{reinterpret_cast<__nv_bfloat16*>(y), ldy, y_head}, T, H, N, K, stream);
}

// y [T, ldy] fp32 = x [T, ldx] W [N, K]^T; K % 16 == 0.
extern "C" int b200_rows_linear_f32(const void* x, int ldx, const void* w, float* y, int ldy, int T, int N, int K,
                                    cudaStream_t stream) {
  if (T <= 0 || N <= 0 || K <= 0 || (K & 15) || (ldx & 7) || ldy < N) return -6;
  return run_rows(x, ldx, w, Plain<float>{y, ldy, 0}, T, N, K, stream);
}

// y [T, ldy] bf16 = gelu(x [T, ldx] W [N, K]^T) * table[ids, col:col + N]; K % 16 == 0, N, ld_table and col even.
extern "C" int b200_rows_token_gate(const void* x, int ldx, const void* w, const void* table, int ld_table, int col, int vocab,
                                    const int* ids, void* y, int ldy, int T, int N, int K, cudaStream_t stream) {
  if (T <= 0 || N <= 0 || (N & 1) || K <= 0 || (K & 15) || (ldx & 7) || (ldy & 1) || ldy < N || ((ld_table | col) & 1) || col < 0 ||
      col + N > ld_table || vocab <= 0 || !ids)
    return -6;
  const TokenGate sink = {reinterpret_cast<__nv_bfloat16*>(y), reinterpret_cast<const __nv_bfloat16*>(table), ids, ldy, ld_table, col, vocab};
  return run_rows(x, ldx, w, sink, T, N, K, stream);
}
