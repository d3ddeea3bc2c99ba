// Activations that look at a whole row, or at the row's token.
//
//   poly_norm    y = a N(z) + b N(z^2) + c N(z^3) + e,   N: over the root mean square of the row's `cols` values
//   token_gate   y = gelu_tanh(z) * table[token, part]   a layer's part of the token's side embedding (short batches take it
//                in the epilogue of their projection, head_linear.cu)
//
// bf16 or fp32 data, fp32 arithmetic.  Rows are `ld` wide (a multiple of 8); columns past `cols` are written as zero.
#include "gelu.cuh"
#include "launch.h"
#include "ops.h"
#include "vec8.cuh"

namespace {
using namespace b200;

struct PolyShape {
  float a, b, c, e, eps;
};

// A block per row.  KEEP: rounds of eight columns per thread held in registers; 0: the row is read twice.
template <typename T, int KEEP>
__global__ void __launch_bounds__(512) poly_norm_kernel(const T* __restrict__ z, int ldz, T* __restrict__ y, int ldy, int cols, PolyShape s) {
  __shared__ float red[3][16];
  pdl_grid_trigger();
  pdl_grid_wait();
  const int nvec = ldy >> 3, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nw = blockDim.x >> 5;
  const T* src = z + (size_t)blockIdx.x * ldz;
  T* dst = y + (size_t)blockIdx.x * ldy;
  Raw8<T> keep[KEEP ? KEEP : 1];
  float s1 = 0.f, s2 = 0.f, s3 = 0.f;
  auto add = [&](const Raw8<T>& r, int v) {
    float f[8];
    r.get(f);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const float q = v * 8 + j < cols ? f[j] * f[j] : 0.f;
      s1 += q;
      s2 = fmaf(q, q, s2);
      s3 = fmaf(q * q, q, s3);
    }
  };
  if (KEEP) {
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int v = tid + i * blockDim.x;
      if (v < nvec) keep[i].load(src + v * 8);
      else keep[i].zero();
    }
#pragma unroll
    for (int i = 0; i < KEEP; ++i) add(keep[i], tid + i * blockDim.x);
  } else {
    for (int v = tid; v < nvec; v += blockDim.x) {
      Raw8<T> r;
      r.load(src + v * 8);
      add(r, v);
    }
  }
  s1 = warp_sum_all(s1);
  s2 = warp_sum_all(s2);
  s3 = warp_sum_all(s3);
  if (lane == 0) { red[0][warp] = s1; red[1][warp] = s2; red[2][warp] = s3; }
  __syncthreads();
  s1 = s2 = s3 = 0.f;
  for (int w = 0; w < nw; ++w) { s1 += red[0][w]; s2 += red[1][w]; s3 += red[2][w]; }
  const float inv_n = 1.f / (float)cols;
  const float r1 = s.a / sqrtf(s1 * inv_n + s.eps), r2 = s.b / sqrtf(s2 * inv_n + s.eps), r3 = s.c / sqrtf(s3 * inv_n + s.eps);
  auto finish = [&](const Raw8<T>& r, int v) {
    float f[8];
    r.get(f);
#pragma unroll
    for (int j = 0; j < 8; ++j) f[j] = v * 8 + j < cols ? fmaf(f[j], fmaf(f[j], fmaf(f[j], r3, r2), r1), s.e) : 0.f;
    store8(dst + v * 8, f);
  };
  if (KEEP) {
#pragma unroll
    for (int i = 0; i < KEEP; ++i)
      if (tid + i * blockDim.x < nvec) finish(keep[i], tid + i * blockDim.x);
  } else {
    for (int v = tid; v < nvec; v += blockDim.x) {
      Raw8<T> r;
      r.load(src + v * 8);
      finish(r, v);
    }
  }
}

// table rows `ld_table` apart, the layer's part at column `col`.
template <typename T>
__global__ void token_gate_kernel(const T* __restrict__ z, int ldz, const T* __restrict__ table, int ld_table, int col, int vocab,
                                  const int* __restrict__ ids, T* __restrict__ y, int ldy, int rows) {
  pdl_grid_trigger();
  pdl_grid_wait();
  const int nvec = ldy >> 3;
  const long long total = (long long)rows * nvec;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long row = i / nvec;
    const int c = (int)(i - row * nvec) * 8, id = ids[row];
    float f[8], e[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    load8(z + row * ldz + c, f);
    if (id >= 0 && id < vocab) load8(table + (size_t)id * ld_table + col + c, e);
#pragma unroll
    for (int j = 0; j < 8; ++j) f[j] = gelu_tanh(f[j]) * e[j];
    store8(y + row * ldy + c, f);
  }
}

template <typename T>
int run_poly_norm(const void* z, int ldz, void* y, int ldy, int cols, const PolyShape& s, int rows, cudaStream_t stream) {
  const int nvec = ldy >> 3, want = nvec <= 256 ? 1 : nvec <= 512 ? 2 : 4;          // vectors of a thread
  int threads = ((nvec + want - 1) / want + 31) / 32 * 32;
  if (threads > 512) threads = 512;
  const int vec = (nvec + threads - 1) / threads;
  const T* zp = reinterpret_cast<const T*>(z);
  T* yp = reinterpret_cast<T*>(y);
  if (vec == 1) return (int)launch_pdl(poly_norm_kernel<T, 1>, dim3(rows), dim3(threads), 0, stream, zp, ldz, yp, ldy, cols, s);
  if (vec == 2) return (int)launch_pdl(poly_norm_kernel<T, 2>, dim3(rows), dim3(threads), 0, stream, zp, ldz, yp, ldy, cols, s);
  if (vec <= 4) return (int)launch_pdl(poly_norm_kernel<T, 4>, dim3(rows), dim3(threads), 0, stream, zp, ldz, yp, ldy, cols, s);
  return (int)launch_pdl(poly_norm_kernel<T, 0>, dim3(rows), dim3(512), 0, stream, zp, ldz, yp, ldy, cols, s);
}

}  // namespace

// z rows `ldz` apart with at least ldy columns, y [rows, ldy]; the norm runs over `cols` <= ldy values.
extern "C" int b200_poly_norm(const void* z, int ldz, void* y, int ldy, int rows, int cols, float a, float b, float c, float e, float eps,
                              int f32, cudaStream_t stream) {
  if (rows <= 0 || ldy <= 0 || (ldy & 7) || (ldz & 7) || ldz < ldy || cols <= 0 || cols > ldy) return -6;
  const PolyShape s = {a, b, c, e, eps};
  return f32 ? run_poly_norm<float>(z, ldz, y, ldy, cols, s, rows, stream) : run_poly_norm<__nv_bfloat16>(z, ldz, y, ldy, cols, s, rows, stream);
}

// z rows `ldz` apart, y [rows, ldy]; table [vocab, ld_table] with ldy columns from `col` on (col, ld_table multiples of 8).
extern "C" int b200_token_gate(const void* z, int ldz, const void* table, int ld_table, int col, int vocab, const int* ids, void* y,
                               int ldy, int rows, int f32, cudaStream_t stream) {
  if (rows <= 0 || ldy <= 0 || (ldy & 7) || (ldz & 7) || ldz < ldy || (ld_table & 7) || (col & 7) || col < 0 || col + ldy > ld_table ||
      vocab <= 0 || !ids)
    return -6;
  const long long total = (long long)rows * (ldy >> 3), blocks = (total + 255) / 256;
  const dim3 grid((unsigned)(blocks < 148 * 16 ? blocks : 148 * 16));
  if (f32)
    return (int)launch_pdl(token_gate_kernel<float>, grid, dim3(256), 0, stream, reinterpret_cast<const float*>(z), ldz,
                           reinterpret_cast<const float*>(table), ld_table, col, vocab, ids, reinterpret_cast<float*>(y), ldy, rows);
  return (int)launch_pdl(token_gate_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, reinterpret_cast<const __nv_bfloat16*>(z), ldz,
                         reinterpret_cast<const __nv_bfloat16*>(table), ld_table, col, vocab, ids, reinterpret_cast<__nv_bfloat16*>(y),
                         ldy, rows);
}
