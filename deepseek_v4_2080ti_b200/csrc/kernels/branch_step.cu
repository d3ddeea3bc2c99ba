// Step of an fp32 residual that takes several sublayer results at once:
//
//   x' = x + sum_b n_b / rms(n_b) * w_b + d_1 + d_2 + sum_k r_k y_k        normed branches, plain branches, routed experts
//   c  = x'                                                                 rounded to the activations' type
//   h  = x' / rms(x') * weight                                              input of the next sublayers, or of the output head
//   m  = h + conv(h)                                                        causal convolution over the sequence, per channel
//
// Every part is optional.  The first normed branch may be a row of an embedding table instead of a stored row, and without a
// residual x starts from zero.  The convolution reads the rows before h's in its own sequence: for a batch of single rows
// those lie in the slot's tail, which is moved on right here (one block holds the whole row); portions leave m to conv_rows.cu.
// h is rounded to the activations' type before the convolution, so that a stored tail and a neighbour give the same result.
// Rows are `ld` wide in memory (a multiple of 8); columns past `cols` are zero on input and written as zero.
#include "launch.h"
#include "ops.h"
#include "vec8.cuh"

namespace {
using namespace b200;

template <typename T>
struct BranchStepParams {
  const float* x;            // [rows, ld] or null: starts from zero
  float* x_out;              // [rows, ld] or null (may be x)
  const int* ids;            // not null: the first normed branch is table[ids[row]]
  const T* table;            // [vocab, ld]
  int vocab;
  const T* normed[2];        // [rows, ld] or null
  const float* normed_w[2];  // [ld]
  const T* plain[2];         // [rows, ld] or null
  const T* routed;           // [routes, ld_routed] or null
  const int* route_row;      // [rows, top]
  const float* route_w;      // [rows, top]
  int ld_routed, top;
  T* copy_out;               // [rows, ld] or null
  const float* weight;       // [ld]
  T* h_out;                  // [rows, ld] or null
  T* m_out;                  // [rows, ld] or null: single rows only
  const float* conv_w;       // [taps, ld], last row: the row itself (with the 1 of h in it)
  T* tail;                   // [slots, taps - 1, ld], oldest first
  const int *row_slot, *positions;
  int taps;
  const int* rows;           // not null: output row i is stored row rows[i]
  int ld, cols;
  float eps;
};

__device__ __forceinline__ float rounded(float v, __nv_bfloat16) { return __bfloat162float(__float2bfloat16(v)); }
__device__ __forceinline__ float rounded(float v, float) { return v; }

// Two sums over the block at once.
__device__ __forceinline__ float2 block_sum2(float2 v, float2* red) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    v.x += __shfl_xor_sync(0xffffffffu, v.x, o);
    v.y += __shfl_xor_sync(0xffffffffu, v.y, o);
  }
  const int lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (lane == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float2 t = lane < nw ? red[lane] : make_float2(0.f, 0.f);
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    t.x += __shfl_xor_sync(0xffffffffu, t.x, o);
    t.y += __shfl_xor_sync(0xffffffffu, t.y, o);
  }
  __syncthreads();
  return t;
}

constexpr int ROUTES = 4;      // routed rows in flight

// Loads go out first, as they lie in memory: the kernel lives on loads in flight.
template <typename T, int VEC>
__global__ void __launch_bounds__(512, VEC == 1 ? 2 : 1) branch_step_kernel(BranchStepParams<T> p) {
  __shared__ float2 red[32];
  extern __shared__ int s_route[];           // [top] row of the routed output or -1, then [top] weights
  pdl_grid_trigger();
  pdl_grid_wait();
  const int nvec = p.ld >> 3;
  const size_t orow = blockIdx.x, row = p.rows ? (size_t)p.rows[orow] : orow;
  float* s_w = reinterpret_cast<float*>(s_route + p.top);
  if (p.routed) {
    for (int k = threadIdx.x; k < p.top; k += blockDim.x) {
      s_route[k] = p.route_row[row * p.top + k];
      s_w[k] = p.route_w[row * p.top + k];
    }
  }
  const T* src[2] = {p.normed[0] ? p.normed[0] + row * p.ld : nullptr, p.normed[1] ? p.normed[1] + row * p.ld : nullptr};
  if (p.ids) {
    const int id = p.ids[row];
    src[0] = id >= 0 && id < p.vocab ? p.table + (size_t)id * p.ld : nullptr;
  }
  const bool has0 = p.ids || src[0], has1 = src[1] != nullptr;      // uniform in the block
  float x[VEC][8], n0[VEC][8], n1[VEC][8];
  float2 ss = make_float2(0.f, 0.f);
#pragma unroll
  for (int it = 0; it < VEC; ++it) {
    const int v = threadIdx.x + it * blockDim.x;
    const bool in = v < nvec;
    const size_t at = row * p.ld + v * 8;
    Raw8<float> xr;
    Raw8<T> b0, b1, p0, p1;
    xr.zero();
    b0.zero();
    b1.zero();
    p0.zero();
    p1.zero();
    if (in) {
      if (p.x) xr.load(p.x + at);
      if (src[0]) b0.load(src[0] + v * 8);
      if (src[1]) b1.load(src[1] + v * 8);
      if (p.plain[0]) p0.load(p.plain[0] + at);
      if (p.plain[1]) p1.load(p.plain[1] + at);
    }
    if (it == 0 && p.routed) __syncthreads();              // the routes
    float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f}, a[8];
    if (in && p.routed) {
      for (int k0 = 0; k0 < p.top; k0 += ROUTES) {
        Raw8<T> y[ROUTES];
        float w[ROUTES];
#pragma unroll
        for (int u = 0; u < ROUTES; ++u) {
          const int at_row = k0 + u < p.top ? s_route[k0 + u] : -1;
          w[u] = at_row >= 0 ? s_w[k0 + u] : 0.f;
          if (at_row >= 0) y[u].load(p.routed + (size_t)at_row * p.ld_routed + v * 8);
          else y[u].zero();
        }
#pragma unroll
        for (int u = 0; u < ROUTES; ++u) {
          y[u].get(a);
#pragma unroll
          for (int j = 0; j < 8; ++j) f[j] = fmaf(w[u], a[j], f[j]);
        }
      }
    }
    xr.get(x[it]);
    b0.get(n0[it]);
    b1.get(n1[it]);
    p0.get(a);
#pragma unroll
    for (int j = 0; j < 8; ++j) f[j] += a[j];
    p1.get(a);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      x[it][j] += f[j] + a[j];
      if (v * 8 + j >= p.cols) n0[it][j] = n1[it][j] = 0.f;
      ss.x = fmaf(n0[it][j], n0[it][j], ss.x);
      ss.y = fmaf(n1[it][j], n1[it][j], ss.y);
    }
  }
  const float inv_n = 1.f / (float)p.cols;
  if (has0 || has1) {
    ss = block_sum2(ss, red);
    const float i0 = 1.f / sqrtf(ss.x * inv_n + p.eps), i1 = 1.f / sqrtf(ss.y * inv_n + p.eps);
#pragma unroll
    for (int it = 0; it < VEC; ++it) {
      const int v = threadIdx.x + it * blockDim.x;
      if (v >= nvec) continue;
      float w[8], s[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      if (has0) {
        load8(p.normed_w[0] + v * 8, w);
#pragma unroll
        for (int j = 0; j < 8; ++j) s[j] = n0[it][j] * i0 * w[j];
      }
      if (has1) {
        load8(p.normed_w[1] + v * 8, w);
#pragma unroll
        for (int j = 0; j < 8; ++j) s[j] = fmaf(n1[it][j] * i1, w[j], s[j]);
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) x[it][j] += s[j];
    }
  }
  float hs = 0.f;
#pragma unroll
  for (int it = 0; it < VEC; ++it) {
    const int v = threadIdx.x + it * blockDim.x;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (v * 8 + j >= p.cols) x[it][j] = 0.f;
      hs = fmaf(x[it][j], x[it][j], hs);
    }
    if (v < nvec) {
      if (p.x_out) store8(p.x_out + row * p.ld + v * 8, x[it]);
      if (p.copy_out) store8(p.copy_out + row * p.ld + v * 8, x[it]);
    }
  }
  if (!p.h_out) return;
  const float inv = 1.f / sqrtf(block_sum2(make_float2(hs, 0.f), red).x * inv_n + p.eps);
#pragma unroll
  for (int it = 0; it < VEC; ++it) {
    const int v = threadIdx.x + it * blockDim.x;
    if (v >= nvec) continue;
    float w[8];
    load8(p.weight + v * 8, w);
#pragma unroll
    for (int j = 0; j < 8; ++j) x[it][j] = rounded(x[it][j] * inv * w[j], T());
    store8(p.h_out + orow * p.ld + v * 8, x[it]);
    if (p.m_out) {
      const int keep = p.taps - 1, pos = p.positions[row];
      T* tail = p.tail + ((size_t)p.row_slot[row] * max(keep, 1)) * p.ld + v * 8;
      float m[8], f[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) m[j] = 0.f;
      for (int t = 0; t < keep; ++t) {                     // the row keep - t positions back
        const bool seen = keep - t <= pos;                 // otherwise zero: before the sequence
        if (seen) load8(tail + (size_t)t * p.ld, f);
        else
#pragma unroll
          for (int j = 0; j < 8; ++j) f[j] = 0.f;
        if (t > 0) store8(tail + (size_t)(t - 1) * p.ld, f);
        load8(p.conv_w + (size_t)t * p.ld + v * 8, w);
#pragma unroll
        for (int j = 0; j < 8; ++j) m[j] = fmaf(w[j], f[j], m[j]);
      }
      load8(p.conv_w + (size_t)keep * p.ld + v * 8, w);
#pragma unroll
      for (int j = 0; j < 8; ++j) m[j] = fmaf(w[j], x[it][j], m[j]);
      if (keep > 0) store8(tail + (size_t)(keep - 1) * p.ld, x[it]);
      store8(p.m_out + row * p.ld + v * 8, m);
    }
  }
}

template <typename T>
int run_branch_step(const float* x, float* x_out, const int* ids, const void* table, int vocab, const void* normed0, const float* normed0_w,
                    const void* normed1, const float* normed1_w, const void* plain0, const void* plain1, const void* routed, int ld_routed,
                    const int* route_row, const float* route_w, int top, void* copy_out, const float* weight, float eps, void* h_out,
                    void* m_out, const float* conv_w, void* tail, const int* row_slot, const int* positions, int taps, const int* rows,
                    int n, int ld, int cols, cudaStream_t stream) {
  BranchStepParams<T> p;
  p.x = x; p.x_out = x_out; p.ids = ids; p.table = reinterpret_cast<const T*>(table); p.vocab = vocab;
  p.normed[0] = reinterpret_cast<const T*>(normed0); p.normed[1] = reinterpret_cast<const T*>(normed1);
  p.normed_w[0] = normed0_w; p.normed_w[1] = normed1_w;
  p.plain[0] = reinterpret_cast<const T*>(plain0); p.plain[1] = reinterpret_cast<const T*>(plain1);
  p.routed = reinterpret_cast<const T*>(routed); p.ld_routed = ld_routed; p.route_row = route_row; p.route_w = route_w; p.top = top;
  p.copy_out = reinterpret_cast<T*>(copy_out); p.weight = weight; p.eps = eps; p.h_out = reinterpret_cast<T*>(h_out);
  p.m_out = reinterpret_cast<T*>(m_out); p.conv_w = conv_w; p.tail = reinterpret_cast<T*>(tail); p.row_slot = row_slot;
  p.positions = positions; p.taps = taps; p.rows = rows; p.ld = ld; p.cols = cols;
  const int nvec = ld >> 3;
  int threads = (nvec + 31) / 32 * 32;
  if (threads > 512) threads = 512;
  const int vec = (nvec + threads - 1) / threads;
  const dim3 grid(n), block(threads);
  const size_t smem = routed ? (size_t)top * 8 : 0;
  if (vec == 1) return (int)launch_pdl(branch_step_kernel<T, 1>, grid, block, smem, stream, p);
  if (vec == 2) return (int)launch_pdl(branch_step_kernel<T, 2>, grid, block, smem, stream, p);
  if (vec <= 4) return (int)launch_pdl(branch_step_kernel<T, 4>, grid, block, smem, stream, p);
  return -6;
}

}  // namespace

// n rows of width ld (a multiple of 8, at most 16384; columns past `cols` are zero); f32 != 0: activations are fp32, else bf16.
extern "C" int b200_branch_step(const float* x, float* x_out, const int* ids, const void* table, int vocab, const void* normed0,
                                const float* normed0_w, const void* normed1, const float* normed1_w, const void* plain0,
                                const void* plain1, const void* routed, int ld_routed, const int* route_row, const float* route_w,
                                int top, void* copy_out, const float* weight, float eps, void* h_out, void* m_out,
                                const float* conv_w, void* tail, const int* row_slot, const int* positions, int taps, const int* rows,
                                int n, int ld, int cols, int f32, cudaStream_t stream) {
  if (n <= 0 || ld <= 0 || (ld & 7) || ld > 16384 || cols <= 0 || cols > ld) return -6;
  if ((ids && (!table || !normed0_w || normed0)) || (normed0 && !normed0_w) || (normed1 && !normed1_w)) return -6;
  if (routed && (!route_row || !route_w || top <= 0 || (ld_routed & 7) || ld_routed < ld)) return -6;
  if ((h_out && !weight) || (m_out && (!h_out || !conv_w || !tail || !row_slot || !positions || rows || taps < 1 || taps > 64))) return -6;
  return f32 ? run_branch_step<float>(x, x_out, ids, table, vocab, normed0, normed0_w, normed1, normed1_w, plain0, plain1, routed, ld_routed,
                                      route_row, route_w, top, copy_out, weight, eps, h_out, m_out, conv_w, tail, row_slot, positions, taps,
                                      rows, n, ld, cols, stream)
             : run_branch_step<__nv_bfloat16>(x, x_out, ids, table, vocab, normed0, normed0_w, normed1, normed1_w, plain0, plain1, routed,
                                              ld_routed, route_row, route_w, top, copy_out, weight, eps, h_out, m_out, conv_w, tail,
                                              row_slot, positions, taps, rows, n, ld, cols, stream);
}
