// Residual-stream step of a decoder with a norm before AND after each sublayer, one launch per sublayer boundary:
//
//   x   (+)= norm(delta + bias) * post_w        the sublayer's output enters the fp32 residual through its own norm
//   x    += step                                optional vector added between layers (start of a looped pass)
//   out   = norm(x) * pre_w                     input of the next sublayer, or of the output head
//   out   = x                                   without pre_w: the next sublayer reads the residual itself (rounded)
//
// Every part is optional.  The row may start from a (scaled) embedding table instead of a stored residual (first layer), and
// the launch may be restricted to a list of rows (output head of the wanted positions only).  The norm is a layer norm
// (centred) or an RMS norm, with plain or one-plus weights.  The residual is fp32; delta and out are bf16 or fp32.
// Rows are `ld` wide in memory (a multiple of 8); columns past `cols` are zero on input and written as zero.
#include "launch.h"
#include "ops.h"
#include "vec8.cuh"

namespace {
using namespace b200;

template <typename T>
struct ResidualNormParams {
  float* x;                  // [rows, ld] residual
  const int* ids;            // not null: the row starts as table[ids[row]] instead of x[row]
  const T* table;            // [vocab, ld]
  int vocab;
  const T* delta;            // [rows, ld] or null
  const float* bias;         // [ld] or null, added to delta before its norm
  const float* post_w;       // [ld] or null (null with a delta: delta is added as it is)
  const float* step;         // [ld] or null
  const float* pre_w;        // [ld] or null
  T* out;                    // [rows out, ld] or null
  const int* rows;           // not null: output row i works on stored row rows[i]
  int ld, cols, rms, unit_offset, write_x;
  float eps, table_scale;
};

template <typename T, int VEC>
__global__ void residual_norm_kernel(ResidualNormParams<T> p) {
  __shared__ float red[32];
  pdl_grid_trigger();
  pdl_grid_wait();
  const size_t orow = blockIdx.x;
  const size_t row = p.rows ? (size_t)p.rows[orow] : orow;
  const int nvec = p.ld >> 3;
  const float inv_n = 1.f / (float)p.cols;
  float x[VEC][8], d[VEC][8];

  // y <- norm(y) * w over the real columns (two passes over registers: mean, then mean of squared deviations)
  auto normalise = [&](float (&y)[VEC][8], const float* w) {
    float mean = 0.f;
    if (!p.rms) {
      float s = 0.f;
#pragma unroll
      for (int it = 0; it < VEC; ++it)
#pragma unroll
        for (int j = 0; j < 8; ++j) s += y[it][j];
      mean = block_sum_all(s, red) * inv_n;
    }
    float ss = 0.f;
#pragma unroll
    for (int it = 0; it < VEC; ++it) {
      const int v = threadIdx.x + it * blockDim.x;
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        y[it][j] = v * 8 + j < p.cols ? y[it][j] - mean : 0.f;
        ss += y[it][j] * y[it][j];
      }
    }
    const float inv = 1.f / sqrtf(block_sum_all(ss, red) * inv_n + p.eps);
#pragma unroll
    for (int it = 0; it < VEC; ++it) {
      const int v = threadIdx.x + it * blockDim.x;
      if (v < nvec) {
        float g[8];
        load8(w + v * 8, g);
#pragma unroll
        for (int j = 0; j < 8; ++j) y[it][j] = y[it][j] * inv * (p.unit_offset ? 1.f + g[j] : g[j]);
      }
    }
  };

  const T* src_row = nullptr;
  if (p.ids) {
    const int id = p.ids[row];
    if (id >= 0 && id < p.vocab) src_row = p.table + (size_t)id * p.ld;
  }
#pragma unroll
  for (int it = 0; it < VEC; ++it) {
    const int v = threadIdx.x + it * blockDim.x;
#pragma unroll
    for (int j = 0; j < 8; ++j) x[it][j] = d[it][j] = 0.f;
    if (v < nvec) {
      if (!p.ids) load8(p.x + row * p.ld + v * 8, x[it]);
      else if (src_row) {
        load8(src_row + v * 8, x[it]);
#pragma unroll
        for (int j = 0; j < 8; ++j) x[it][j] *= p.table_scale;
      }
      if (p.delta) {
        load8(p.delta + row * p.ld + v * 8, d[it]);
        if (p.bias) {
          float b[8];
          load8(p.bias + v * 8, b);
#pragma unroll
          for (int j = 0; j < 8; ++j) d[it][j] += b[j];
        }
      }
    }
  }
  if (p.delta) {
    if (p.post_w) normalise(d, p.post_w);
#pragma unroll
    for (int it = 0; it < VEC; ++it)
#pragma unroll
      for (int j = 0; j < 8; ++j) x[it][j] += d[it][j];
  }
#pragma unroll
  for (int it = 0; it < VEC; ++it) {
    const int v = threadIdx.x + it * blockDim.x;
    if (v < nvec) {
      if (p.step) {
        float s[8];
        load8(p.step + v * 8, s);
#pragma unroll
        for (int j = 0; j < 8; ++j) x[it][j] += s[j];
      }
      if (p.write_x) store8(p.x + row * p.ld + v * 8, x[it]);
    }
  }
  if (!p.out) return;
  if (p.pre_w) normalise(x, p.pre_w);
#pragma unroll
  for (int it = 0; it < VEC; ++it) {
    const int v = threadIdx.x + it * blockDim.x;
    if (v < nvec) store8(p.out + orow * p.ld + v * 8, x[it]);
  }
}

template <typename T>
int launch_residual_norm(ResidualNormParams<T> p, int n, cudaStream_t stream) {
  const int nvec = p.ld >> 3;
  int threads = (nvec + 31) / 32 * 32;
  if (threads > 512) threads = 512;
  const int vec = (nvec + threads - 1) / threads;
  const dim3 grid(n), block(threads);
  if (vec == 1) return (int)launch_pdl(residual_norm_kernel<T, 1>, grid, block, 0, stream, p);
  if (vec == 2) return (int)launch_pdl(residual_norm_kernel<T, 2>, grid, block, 0, stream, p);
  if (vec <= 4) return (int)launch_pdl(residual_norm_kernel<T, 4>, grid, block, 0, stream, p);
  return -6;
}

template <typename T>
int run_residual_norm(float* x, const int* ids, const void* table, int vocab, const void* delta, const float* bias,
                      const float* post_w, const float* step, const float* pre_w, void* out, const int* rows, int n, int ld,
                      int cols, float eps, int rms, int unit_offset, int write_x, float table_scale, cudaStream_t stream) {
  ResidualNormParams<T> p;
  p.x = x; p.ids = ids; p.table = reinterpret_cast<const T*>(table); p.vocab = vocab;
  p.delta = reinterpret_cast<const T*>(delta); p.bias = bias; p.post_w = post_w; p.step = step; p.pre_w = pre_w;
  p.out = reinterpret_cast<T*>(out); p.rows = rows; p.ld = ld; p.cols = cols; p.rms = rms; p.unit_offset = unit_offset;
  p.write_x = write_x; p.eps = eps; p.table_scale = table_scale;
  return launch_residual_norm(p, n, stream);
}

}  // namespace

// n rows; f32 != 0: table / delta / out are fp32, otherwise bf16.  ld % 8 == 0, cols <= ld <= 16384.
extern "C" int b200_residual_norm(float* x, const int* ids, const void* table, int vocab, const void* delta,
                                  const float* bias, const float* post_w, const float* step, const float* pre_w, void* out,
                                  const int* rows, int n, int ld, int cols, float eps, int rms, int unit_offset, int write_x,
                                  float table_scale, int f32, cudaStream_t stream) {
  if (n <= 0 || ld <= 0 || (ld & 7) || ld > 16384 || cols <= 0 || cols > ld) return -6;
  if ((pre_w && !out) || (!ids && !x) || (write_x && !x) || (ids && !table)) return -6;
  return f32 ? run_residual_norm<float>(x, ids, table, vocab, delta, bias, post_w, step, pre_w, out, rows, n, ld, cols, eps,
                                        rms, unit_offset, write_x, table_scale, stream)
             : run_residual_norm<__nv_bfloat16>(x, ids, table, vocab, delta, bias, post_w, step, pre_w, out, rows, n, ld,
                                                cols, eps, rms, unit_offset, write_x, table_scale, stream);
}
