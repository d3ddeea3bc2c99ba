// y = xIELU(z + bias) over rows: for z > 0  ap z^2 + z / 2,  otherwise  an (exp(z) - 1 - z) + z / 2, with the two
// positive coefficients given as numbers.  bf16 or fp32 data, fp32 arithmetic; `ld` (a multiple of 8) columns per row,
// columns whose input and bias are zero stay zero.  (bf16 projections take the activation in the GEMM's epilogue instead,
// b200_gemm_bf16_bias_xielu.)
//
// b200_glu: gated units (glu.cuh) over a projection that holds gate and up features interleaved in tiles of `tile` columns
// [gate tile | up tile | gate tile | ...], the layout the fused GEMM (b200_gemm_bf16_glu) wants its weights in.
#include "launch.h"
#include "ops.h"
#include "vec8.cuh"
#include "xielu.cuh"
#include "glu.cuh"

namespace {
using namespace b200;

template <typename T>
__global__ void bias_xielu_kernel(const T* __restrict__ in, const float* __restrict__ bias, T* __restrict__ out,
                                  long long nvec_total, int nvec, float ap, float an) {
  pdl_grid_trigger();
  pdl_grid_wait();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < nvec_total; i += (long long)gridDim.x * blockDim.x) {
    float z[8];
    load8(in + i * 8, z);
    if (bias) {
      float b[8];
      load8(bias + (i % nvec) * 8, b);
#pragma unroll
      for (int j = 0; j < 8; ++j) z[j] += b[j];
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) z[j] = sizeof(T) == 2 ? xielu_bf16(z[j], ap, an) : xielu(z[j], ap, an);
    store8(out + i * 8, z);
  }
}

template <typename T>
__global__ void glu_kernel(const T* __restrict__ in, int ld, T* __restrict__ out, long long nvec_total, int nvec, int tile, GluShape s) {
  pdl_grid_trigger();
  pdl_grid_wait();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < nvec_total; i += (long long)gridDim.x * blockDim.x) {
    const long long row = i / nvec;
    const int c = (int)(i - row * nvec) * 8;
    const T* src = in + row * ld + (c / tile) * 2 * tile + c % tile;
    float g[8], u[8];
    load8(src, g);
    load8(src + tile, u);
#pragma unroll
    for (int j = 0; j < 8; ++j) g[j] = glu<sizeof(T) == 2>(g[j], u[j], s);
    store8(out + i * 8, g);
  }
}

}  // namespace

// in: rows of 2 * inter columns, `ld` apart, out [rows, inter]; inter a multiple of tile, tile and ld multiples of 8.
extern "C" int b200_glu(const void* in, int ld, void* out, long long rows, int inter, int tile, float limit, float slope, int f32,
                        cudaStream_t stream) {
  if (rows <= 0 || inter <= 0 || tile <= 0 || (tile & 7) || inter % tile || (ld & 7) || ld < 2 * inter) return -6;
  const int nvec = inter >> 3;
  const long long total = rows * nvec;
  const long long blocks = (total + 255) / 256;
  const dim3 grid((unsigned)(blocks < 148 * 16 ? blocks : 148 * 16));
  const GluShape s = {limit, slope};
  if (f32)
    return (int)launch_pdl(glu_kernel<float>, grid, dim3(256), 0, stream, reinterpret_cast<const float*>(in), ld,
                           reinterpret_cast<float*>(out), total, nvec, tile, s);
  return (int)launch_pdl(glu_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, reinterpret_cast<const __nv_bfloat16*>(in), ld,
                         reinterpret_cast<__nv_bfloat16*>(out), total, nvec, tile, s);
}

extern "C" int b200_bias_xielu(const void* in, const float* bias, void* out, long long rows, int ld, float ap, float an,
                               int f32, cudaStream_t stream) {
  if (rows <= 0 || ld <= 0 || (ld & 7)) return -6;
  const int nvec = ld >> 3;
  const long long total = rows * nvec;
  const long long blocks = (total + 255) / 256;
  const dim3 grid((unsigned)(blocks < 148 * 16 ? blocks : 148 * 16));
  if (f32)
    return (int)launch_pdl(bias_xielu_kernel<float>, grid, dim3(256), 0, stream, reinterpret_cast<const float*>(in), bias,
                           reinterpret_cast<float*>(out), total, nvec, ap, an);
  return (int)launch_pdl(bias_xielu_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream,
                         reinterpret_cast<const __nv_bfloat16*>(in), bias, reinterpret_cast<__nv_bfloat16*>(out), total, nvec,
                         ap, an);
}
