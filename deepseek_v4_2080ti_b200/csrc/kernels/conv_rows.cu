// Causal depthwise convolution over a batch of rows that belong to several sequences, with optional bias and SiLU.
//
//   y[r, c] = act(bias[c] + sum_j w[j, c] x_{back(j)}[c]),   back(j) = taps - 1 - j rows before r in r's own sequence
//
// Rows of one sequence are neighbours; row_first[r] is the sequence's first row of this batch, row_slot[r] its state slot,
// positions[r] its position.  Inputs from before the batch come from the slot's tail (the last taps - 1 inputs, oldest
// first); inputs from before position 0 are zero, so a slot needs no clearing.  A sequence that brings a single row has its
// tail replaced right here (one thread holds all of it); the tail of a longer portion, which several blocks read, is replaced
// by the kernel that runs the recurrence behind the convolution (selective_scan.cu), or by conv_tails.  One thread: 8
// channels, `strip` rows.
#include "launch.h"
#include "ops.h"
#include "vec8.cuh"

namespace {
using namespace b200;

template <typename T>
struct ConvRowsParams {
  const T* x;              // [rows, ldx]
  const float* w;          // [taps, C]
  const float* bias;       // [C] or null
  T* tail;                 // [slots, taps - 1, C]
  const int *row_first, *row_slot, *positions;
  T* y;                    // [rows, ldy]
  int ldx, ldy, rows, C, taps, silu, strip;
};

template <typename T, int K>
__global__ void __launch_bounds__(128) conv_rows_kernel(ConvRowsParams<T> p) {
  pdl_grid_trigger();
  const int taps = K ? K : p.taps;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  const bool on = c < p.C;
  float w[K ? K : 1][8], b[8] = {};
  if (on) {
    if (p.bias) load8(p.bias + c, b);
    if (K) {
#pragma unroll
      for (int j = 0; j < K; ++j) load8(p.w + (size_t)j * p.C + c, w[j]);
    }
  }
  pdl_grid_wait();
  if (!on) return;
  const int r0 = blockIdx.y * p.strip, r1 = min(p.rows, r0 + p.strip);
  auto finish = [&](int r, float (&acc)[8]) {
    if (p.silu) {
#pragma unroll
      for (int i = 0; i < 8; ++i)
        acc[i] = sizeof(T) == 2 ? __fdividef(acc[i], 1.f + __expf(-acc[i])) : acc[i] / (1.f + expf(-acc[i]));
    }
    store8(p.y + (size_t)r * p.ldy + c, acc);
  };
  if (K > 1 && p.strip > 1) {
    const int first = p.row_first[r0];
    if (r0 - first >= K - 1 && p.row_first[r1 - 1] == first) {
      // a strip inside one sequence's portion: every row is read once and stays in a window of registers
      float win[K ? K : 1][8];
#pragma unroll
      for (int j = 1; j < K; ++j) load8(p.x + (size_t)(r0 - K + j) * p.ldx + c, win[j]);
#pragma unroll 4
      for (int r = r0; r < r1; ++r) {
        float acc[8];
#pragma unroll
        for (int j = 0; j + 1 < K; ++j)
#pragma unroll
          for (int i = 0; i < 8; ++i) win[j][i] = win[j + 1][i];
        load8(p.x + (size_t)r * p.ldx + c, win[K ? K - 1 : 0]);
#pragma unroll
        for (int i = 0; i < 8; ++i) acc[i] = b[i];
#pragma unroll
        for (int j = 0; j < K; ++j)
#pragma unroll
          for (int i = 0; i < 8; ++i) acc[i] = fmaf(w[j][i], win[j][i], acc[i]);
        finish(r, acc);
      }
      return;
    }
  }
  for (int r = r0; r < r1; ++r) {
    const int off = r - p.row_first[r], pos = p.positions[r];
    T* tail = p.tail + ((size_t)p.row_slot[r] * (taps - 1)) * p.C + c;
    const bool solo = off == 0 && (r + 1 == p.rows || p.row_first[r + 1] == r + 1);
    float acc[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i] = b[i];
#pragma unroll
    for (int j = 0; j < taps; ++j) {
      const int back = taps - 1 - j;
      if (back > pos) continue;
      float f[8];
      load8(back <= off ? p.x + (size_t)(r - back) * p.ldx + c : tail + (size_t)(taps - 1 - (back - off)) * p.C, f);
      if (!K) load8(p.w + (size_t)j * p.C + c, w[0]);
#pragma unroll
      for (int i = 0; i < 8; ++i) acc[i] = fmaf(w[K ? j : 0][i], f[i], acc[i]);
    }
    if (solo) {
      // the inputs of the last taps - 1 positions, this row's included (loaded again: exact copies of what lies there)
      if (K) {
        float keep[K ? K : 1][8];
#pragma unroll
        for (int j = 1; j < K; ++j) load8(j + 1 < K ? tail + (size_t)j * p.C : p.x + (size_t)r * p.ldx + c, keep[j]);
#pragma unroll
        for (int j = 1; j < K; ++j) store8(tail + (size_t)(j - 1) * p.C, keep[j]);
      } else {
        for (int j = 1; j < taps; ++j) {
          float f[8];
          load8(j + 1 < taps ? tail + (size_t)j * p.C : p.x + (size_t)r * p.ldx + c, f);
          store8(tail + (size_t)(j - 1) * p.C, f);
        }
      }
    }
    finish(r, acc);
  }
}

template <typename T>
int run_conv_rows(const void* x, int ldx, const float* w, const float* bias, void* tail, const int* row_first,
                  const int* row_slot, const int* positions, void* y, int ldy, int rows, int C, int taps, int silu,
                  cudaStream_t stream) {
  ConvRowsParams<T> p;
  p.x = reinterpret_cast<const T*>(x); p.w = w; p.bias = bias; p.tail = reinterpret_cast<T*>(tail);
  p.row_first = row_first; p.row_slot = row_slot; p.positions = positions; p.y = reinterpret_cast<T*>(y);
  p.ldx = ldx; p.ldy = ldy; p.rows = rows; p.C = C; p.taps = taps; p.silu = silu;
  p.strip = 1;
  while (p.strip < 16 && (long long)rows * C / 8 / p.strip > 148LL * 4096) p.strip *= 2;
  const dim3 grid((C / 8 + 127) / 128, (rows + p.strip - 1) / p.strip);
  if (grid.y > 65535) return -6;
  switch (taps) {
    case 2: return (int)launch_pdl(conv_rows_kernel<T, 2>, grid, dim3(128), 0, stream, p);
    case 3: return (int)launch_pdl(conv_rows_kernel<T, 3>, grid, dim3(128), 0, stream, p);
    case 4: return (int)launch_pdl(conv_rows_kernel<T, 4>, grid, dim3(128), 0, stream, p);
    default: return (int)launch_pdl(conv_rows_kernel<T, 0>, grid, dim3(128), 0, stream, p);
  }
}

// New tails of the portions with more than one row: the inputs of their last taps - 1 positions.  A thread owns eight channels of
// a tail; a portion shorter than the tail moves what stays of the old one.
template <typename T>
__global__ void conv_tails_kernel(const T* __restrict__ x, int ldx, T* __restrict__ tail, const int* __restrict__ first,
                                  const int* __restrict__ length, const int* __restrict__ slot, int C, int keep) {
  pdl_grid_trigger();
  pdl_grid_wait();
  const int e = blockIdx.y, n = length[e], c = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  if (n < 2 || c >= C) return;
  T* dst = tail + (size_t)slot[e] * keep * C + c;
  const T* src = x + (size_t)first[e] * ldx + c;
  for (int j = 0; j < keep; ++j) {
    const int at = n - keep + j;             // row of the portion, or behind its start: an entry of the old tail
    float f[8];
    load8(at >= 0 ? src + (size_t)at * ldx : dst + (size_t)(keep + at) * C, f);
    store8(dst + (size_t)j * C, f);
  }
}

}  // namespace

// x [rows, >= C] the convolution's inputs; tails [slots, taps - 1, C] of the entries with more than one row are replaced.
extern "C" int b200_conv_tails(const void* x, int ldx, void* tail, const int* first, const int* length, const int* slot, int entries,
                               int C, int taps, int f32, cudaStream_t stream) {
  if (entries <= 0 || entries > 65535 || C <= 0 || (C & 7) || (ldx & 7) || ldx < C || taps < 2 || taps > 64) return -6;
  const dim3 grid((C / 8 + 127) / 128, entries);
  if (f32)
    return (int)launch_pdl(conv_tails_kernel<float>, grid, dim3(128), 0, stream, reinterpret_cast<const float*>(x), ldx,
                           reinterpret_cast<float*>(tail), first, length, slot, C, taps - 1);
  return (int)launch_pdl(conv_tails_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, reinterpret_cast<const __nv_bfloat16*>(x), ldx,
                         reinterpret_cast<__nv_bfloat16*>(tail), first, length, slot, C, taps - 1);
}

// x rows of C channels (C, ldx, ldy multiples of 8); f32 != 0: x, tail, y are fp32, otherwise bf16.
extern "C" int b200_conv_rows(const void* x, int ldx, const float* w, const float* bias, void* tail, const int* row_first,
                              const int* row_slot, const int* positions, void* y, int ldy, int rows, int C, int taps, int silu,
                              int f32, cudaStream_t stream) {
  if (rows <= 0 || C <= 0 || (C & 7) || (ldx & 7) || (ldy & 7) || ldx < C || ldy < C || taps < 1 || taps > 64) return -6;
  return f32 ? run_conv_rows<float>(x, ldx, w, bias, tail, row_first, row_slot, positions, y, ldy, rows, C, taps, silu, stream)
             : run_conv_rows<__nv_bfloat16>(x, ldx, w, bias, tail, row_first, row_slot, positions, y, ldy, rows, C, taps, silu,
                                            stream);
}
