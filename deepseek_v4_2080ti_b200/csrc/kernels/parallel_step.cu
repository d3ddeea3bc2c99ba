// Step between the layers of a decoder whose two sublayers read the same norm and are added side by side:
//
//   x' = x + mix sigmoid(g1 + b1) + ff sigmoid(g2 + b2)          element-wise gates; the residual is fp32
//   ff = sum_k w_k y_k + sigmoid(sg) shared                      routed experts, identity experts (y = h of the layer), one
//                                                                shared expert behind a gate of its own per row
//   h' = x' / rms(x') * weight                                   one weight for all columns
//   m' = h' + (h'(row before) - h') shift                        what a mixer with a token shift reads
//
// Every part is optional.  The row may start from an embedding table.  The row before is the neighbouring row of the same
// portion, the sequence's stored tail where a portion begins, or zero at position 0.  A batch of single rows is one launch, and
// replaces the tails itself (one block reads and writes a tail); with longer portions a row's predecessor is another block's
// work, so the shift is a second pass over h', and the tails are replaced by a third once every reader is done.
// h' is rounded to the activations' type before the shift, so that a stored tail and a neighbour give the same result.
#include "launch.h"
#include "ops.h"
#include "vec8.cuh"

namespace {
using namespace b200;

template <typename T>
struct ParallelStepParams {
  const float* x;            // [rows, ld]
  float* x_out;              // [rows, ld] or null (may be x)
  const int* ids;            // not null: the row starts as table[ids[row]]
  const T* table;
  int vocab;
  const T* mix;              // [rows, ld] or null
  const T* gates;            // [rows, ld_gates]: logits of the mixer's gate, then (at column ld) of the feed-forward's
  const float* gate_b;       // [2 * ld]
  int ld_gates;
  const T* h;                // [rows, ld] the layer's norm output (identity experts)
  const T* routed;           // [routes, ld_routed] or null
  const int *route_row, *route_id;   // [rows, top]
  const float* route_w;      // [rows, top]
  int ld_routed, top, experts;       // ids from `experts` on are identity experts
  const T* shared;           // [rows, ld] or null
  const float* shared_gate;  // logit of row r at shared_gate[r * ld_shared_gate], or null (factor 1)
  int ld_shared_gate;
  float weight, eps;
  T* h_out;                  // [rows, ld] or null
  T* m_out;                  // [rows, ld] or null: single rows only
  const float* shift;        // [ld]
  T* tail;                   // [slots, ld]
  const int *row_slot, *positions;
  const int* rows;           // not null: output row i is stored row rows[i]
  int ld, cols;
};

__device__ __forceinline__ float sigmoidf(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float gate_of(float z, __nv_bfloat16) { return __fdividef(1.f, 1.f + __expf(-z)); }
__device__ __forceinline__ float gate_of(float z, float) { return sigmoidf(z); }
__device__ __forceinline__ float rounded(float v, __nv_bfloat16) { return __bfloat162float(__float2bfloat16(v)); }
__device__ __forceinline__ float rounded(float v, float) { return v; }

constexpr int ROUTES = 4;      // routed rows in flight

// Loads go out first, as they lie in memory, and the occupancy is bounded from below: the kernel lives on loads in flight.
template <typename T, int VEC>
__global__ void __launch_bounds__(512, VEC == 1 ? 2 : 1) parallel_step_kernel(ParallelStepParams<T> p) {
  __shared__ float red[32];
  extern __shared__ int s_route[];           // [top] row of the routed output, -1, or -2: identity; then [top] weights
  pdl_grid_trigger();
  pdl_grid_wait();
  const int nvec = p.ld >> 3;
  const size_t orow = blockIdx.x, row = p.rows ? (size_t)p.rows[orow] : orow;
  float* s_w = reinterpret_cast<float*>(s_route + p.top);
  const bool ff = p.routed || p.shared;
  if (p.routed) {
    for (int k = threadIdx.x; k < p.top; k += blockDim.x) {
      const size_t r = row * p.top + k;
      const bool own = p.route_id[r] < p.experts;
      s_route[k] = own ? p.route_row[r] : -2;
      s_w[k] = p.route_w[r];
    }
  }
  const T* src_row = nullptr;
  if (p.ids) {
    const int id = p.ids[row];
    if (id >= 0 && id < p.vocab) src_row = p.table + (size_t)id * p.ld;
  }
  const float sg = p.shared ? (p.shared_gate ? sigmoidf(p.shared_gate[row * p.ld_shared_gate]) : 1.f) : 0.f;
  const int slot = p.m_out ? p.row_slot[row] : 0, pos = p.m_out ? p.positions[row] : 0;
  float h[VEC][8], ss = 0.f;
#pragma unroll
  for (int it = 0; it < VEC; ++it) {
    const int v = threadIdx.x + it * blockDim.x;
    const bool in = v < nvec;
    const size_t at = row * p.ld + v * 8;
    float x[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    Raw8<float> xr;
    Raw8<T> er, mr, g1, g2, sh;
    if (in) {
      if (!p.ids) xr.load(p.x + at);
      else if (src_row) er.load(src_row + v * 8);
      if (p.mix) {
        mr.load(p.mix + at);
        g1.load(p.gates + row * p.ld_gates + v * 8);
      }
      if (ff) g2.load(p.gates + row * p.ld_gates + p.ld + v * 8);
      if (p.shared) sh.load(p.shared + at);
    }
    if (it == 0) __syncthreads();            // the routes
    if (in) {
      float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f}, a[8], b[8];
      if (p.routed) {
        float id_w = 0.f;                    // weight of the identity experts
        for (int k0 = 0; k0 < p.top; k0 += ROUTES) {
          Raw8<T> y[ROUTES];
          float w[ROUTES];
#pragma unroll
          for (int u = 0; u < ROUTES; ++u) {
            const int at_row = k0 + u < p.top ? s_route[k0 + u] : -1;
            w[u] = at_row >= 0 ? s_w[k0 + u] : 0.f;
            if (at_row >= 0) y[u].load(p.routed + (size_t)at_row * p.ld_routed + v * 8);
            else y[u].zero();
            if (at_row == -2) id_w += s_w[k0 + u];
          }
#pragma unroll
          for (int u = 0; u < ROUTES; ++u) {
            y[u].get(a);
#pragma unroll
            for (int j = 0; j < 8; ++j) f[j] = fmaf(w[u], a[j], f[j]);
          }
        }
        if (id_w != 0.f) {
          load8(p.h + at, a);
#pragma unroll
          for (int j = 0; j < 8; ++j) f[j] = fmaf(id_w, a[j], f[j]);
        }
      }
      if (!p.ids) xr.get(x);
      else if (src_row) er.get(x);
      if (p.mix) {
        float m[8];
        mr.get(m);
        g1.get(a);
        load8(p.gate_b + v * 8, b);
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] = fmaf(m[j], gate_of(a[j] + b[j], T()), x[j]);
      }
      if (ff) {
        if (p.shared) {
          sh.get(a);
#pragma unroll
          for (int j = 0; j < 8; ++j) f[j] = fmaf(sg, a[j], f[j]);
        }
        g2.get(a);
        load8(p.gate_b + p.ld + v * 8, b);
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] = fmaf(f[j], gate_of(a[j] + b[j], T()), x[j]);
      }
      if (p.x_out) store8(p.x_out + at, x);
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      h[it][j] = v * 8 + j < p.cols ? x[j] : 0.f;
      ss += h[it][j] * h[it][j];
    }
  }
  if (!p.h_out) return;
  const float f = p.weight / sqrtf(block_sum_all(ss, red) / (float)p.cols + p.eps);
#pragma unroll
  for (int it = 0; it < VEC; ++it) {
    const int v = threadIdx.x + it * blockDim.x;
    if (v >= nvec) continue;
#pragma unroll
    for (int j = 0; j < 8; ++j) h[it][j] = rounded(h[it][j] * f, T());
    store8(p.h_out + orow * p.ld + v * 8, h[it]);
    if (p.m_out) {
      T* tail = p.tail + (size_t)slot * p.ld + v * 8;
      float s[8], m[8], before[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      if (pos > 0) load8(tail, before);
      load8(p.shift + v * 8, s);
#pragma unroll
      for (int j = 0; j < 8; ++j) m[j] = fmaf(before[j] - h[it][j], s[j], h[it][j]);
      store8(p.m_out + orow * p.ld + v * 8, m);
      store8(tail, h[it]);
    }
  }
}

// m = h + (h of the row before - h) shift over rows of several portions; a thread walks SHIFT_ROWS rows of eight columns.
constexpr int SHIFT_ROWS = 4;

template <typename T>
__global__ void shift_rows_kernel(const T* __restrict__ h, T* __restrict__ m, const float* __restrict__ shift, const T* __restrict__ tail,
                                  const int* __restrict__ row_first, const int* __restrict__ row_slot,
                                  const int* __restrict__ positions, int n, int ld) {
  pdl_grid_trigger();
  pdl_grid_wait();
  const int v = blockIdx.x * blockDim.x + threadIdx.x, r0 = blockIdx.y * SHIFT_ROWS;
  if (v >= ld / 8) return;
  float s[8], before[8], cur[SHIFT_ROWS][8];
  load8(shift + v * 8, s);
#pragma unroll
  for (int i = 0; i < SHIFT_ROWS; ++i)
    if (r0 + i < n) load8(h + (size_t)(r0 + i) * ld + v * 8, cur[i]);
  if (row_first[r0] != r0) load8(h + (size_t)(r0 - 1) * ld + v * 8, before);
#pragma unroll
  for (int i = 0; i < SHIFT_ROWS; ++i) {
    const int r = r0 + i;
    if (r >= n) return;
    if (row_first[r] == r) {
      if (positions[r] > 0) load8(tail + (size_t)row_slot[r] * ld + v * 8, before);
      else
#pragma unroll
        for (int j = 0; j < 8; ++j) before[j] = 0.f;
    }
    float o[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      o[j] = fmaf(before[j] - cur[i][j], s[j], cur[i][j]);
      before[j] = cur[i][j];
    }
    store8(m + (size_t)r * ld + v * 8, o);
  }
}

// tail[slot] = h[last row] of every entry.
template <typename T>
__global__ void shift_tails_kernel(const T* __restrict__ h, T* __restrict__ tail, const int* __restrict__ first,
                                   const int* __restrict__ length, const int* __restrict__ slot, int ld) {
  pdl_grid_trigger();
  pdl_grid_wait();
  const int e = blockIdx.x, n = length[e];
  const T* src = h + (size_t)(first[e] + n - 1) * ld;
  T* dst = tail + (size_t)slot[e] * ld;
  for (int v = threadIdx.x; v < ld / 8; v += blockDim.x) {
    float f[8];
    load8(src + v * 8, f);
    store8(dst + v * 8, f);
  }
}

template <typename T>
int run_parallel_step(ParallelStepParams<T> p, int n, cudaStream_t stream) {
  const int nvec = p.ld >> 3;
  int threads = (nvec + 31) / 32 * 32;
  if (threads > 512) threads = 512;
  const int vec = (nvec + threads - 1) / threads;
  const dim3 grid(n), block(threads);
  const size_t smem = p.routed ? (size_t)p.top * 8 : 0;
  if (vec == 1) return (int)launch_pdl(parallel_step_kernel<T, 1>, grid, block, smem, stream, p);
  if (vec == 2) return (int)launch_pdl(parallel_step_kernel<T, 2>, grid, block, smem, stream, p);
  if (vec <= 4) return (int)launch_pdl(parallel_step_kernel<T, 4>, grid, block, smem, stream, p);
  return -6;
}

template <typename T>
int make_parallel_step(const float* x, float* x_out, const int* ids, const void* table, int vocab, const void* mix, const void* gates,
                       int ld_gates, const float* gate_b, const void* h, const void* routed, int ld_routed, const int* route_row,
                       const int* route_id, const float* route_w, int top, int experts, const void* shared, const float* shared_gate,
                       int ld_shared_gate, float weight, float eps, void* h_out, void* m_out, const float* shift, void* tail,
                       const int* row_slot, const int* positions, const int* rows, int n, int ld, int cols, cudaStream_t stream) {
  ParallelStepParams<T> p;
  p.x = x; p.x_out = x_out; p.ids = ids; p.table = reinterpret_cast<const T*>(table); p.vocab = vocab;
  p.mix = reinterpret_cast<const T*>(mix); p.gates = reinterpret_cast<const T*>(gates); p.gate_b = gate_b; p.ld_gates = ld_gates;
  p.h = reinterpret_cast<const T*>(h); p.routed = reinterpret_cast<const T*>(routed); p.route_row = route_row;
  p.route_id = route_id; p.route_w = route_w; p.ld_routed = ld_routed; p.top = top; p.experts = experts;
  p.shared = reinterpret_cast<const T*>(shared); p.shared_gate = shared_gate; p.ld_shared_gate = ld_shared_gate;
  p.weight = weight; p.eps = eps; p.h_out = reinterpret_cast<T*>(h_out); p.m_out = reinterpret_cast<T*>(m_out); p.shift = shift;
  p.tail = reinterpret_cast<T*>(tail); p.row_slot = row_slot; p.positions = positions; p.rows = rows;
  p.ld = ld; p.cols = cols;
  return run_parallel_step(p, n, stream);
}

}  // namespace

// n rows of width ld (a multiple of 8, at most 16384; columns past `cols` are zero); f32 != 0: activations are fp32, else bf16.
extern "C" int b200_parallel_step(const float* x, float* x_out, const int* ids, const void* table, int vocab, const void* mix,
                                  const void* gates, int ld_gates, const float* gate_b, const void* h, const void* routed,
                                  int ld_routed, const int* route_row, const int* route_id, const float* route_w, int top,
                                  int experts, const void* shared, const float* shared_gate, int ld_shared_gate, float weight,
                                  float eps, void* h_out, void* m_out, const float* shift, void* tail,
                                  const int* row_slot, const int* positions, const int* rows, int n, int ld, int cols, int f32,
                                  cudaStream_t stream) {
  if (n <= 0 || ld <= 0 || (ld & 7) || ld > 16384 || cols <= 0 || cols > ld) return -6;
  if ((!ids && !x) || (ids && !table) || ((mix || routed || shared) && (!gates || !gate_b))) return -6;
  if (ld_gates & 7 || ld_routed & 7 || (routed && (!route_row || !route_id || !route_w || !h || top <= 0 || ld_routed < ld))) return -6;
  if (m_out && (!h_out || !shift || !tail || !row_slot || !positions || rows)) return -6;
  return f32 ? make_parallel_step<float>(x, x_out, ids, table, vocab, mix, gates, ld_gates, gate_b, h, routed, ld_routed, route_row,
                                         route_id, route_w, top, experts, shared, shared_gate, ld_shared_gate, weight, eps, h_out,
                                         m_out, shift, tail, row_slot, positions, rows, n, ld, cols, stream)
             : make_parallel_step<__nv_bfloat16>(x, x_out, ids, table, vocab, mix, gates, ld_gates, gate_b, h, routed, ld_routed,
                                                 route_row, route_id, route_w, top, experts, shared, shared_gate, ld_shared_gate,
                                                 weight, eps, h_out, m_out, shift, tail, row_slot, positions, rows, n, ld,
                                                 cols, stream);
}

// Rows of several portions (row_first: first row of a row's portion), then the sequences' new tails; n rows, `entries` portions.
extern "C" int b200_shift_rows(const void* h, void* m, const float* shift, void* tail, const int* row_first, const int* row_slot,
                               const int* positions, const int* first, const int* length, const int* slot, int entries, int n, int ld,
                               int f32, cudaStream_t stream) {
  if (n <= 0 || entries <= 0 || ld <= 0 || (ld & 7) || (n + SHIFT_ROWS - 1) / SHIFT_ROWS > 65535) return -6;
  const int nvec = ld / 8, threads = nvec >= 128 ? 128 : (nvec + 31) / 32 * 32;
  const dim3 grid((nvec + threads - 1) / threads, (n + SHIFT_ROWS - 1) / SHIFT_ROWS);
  if (f32) {
    auto hp = reinterpret_cast<const float*>(h);
    auto tp = reinterpret_cast<float*>(tail);
    const cudaError_t e = launch_pdl(shift_rows_kernel<float>, grid, dim3(threads), 0, stream, hp, reinterpret_cast<float*>(m), shift,
                                     tp, row_first, row_slot, positions, n, ld);
    return e != cudaSuccess ? (int)e : (int)launch_pdl(shift_tails_kernel<float>, dim3(entries), dim3(256), 0, stream, hp, tp, first,
                                                       length, slot, ld);
  }
  auto hp = reinterpret_cast<const __nv_bfloat16*>(h);
  auto tp = reinterpret_cast<__nv_bfloat16*>(tail);
  const cudaError_t e = launch_pdl(shift_rows_kernel<__nv_bfloat16>, grid, dim3(threads), 0, stream, hp,
                                   reinterpret_cast<__nv_bfloat16*>(m), shift, tp, row_first, row_slot, positions, n, ld);
  return e != cudaSuccess ? (int)e : (int)launch_pdl(shift_tails_kernel<__nv_bfloat16>, dim3(entries), dim3(256), 0, stream, hp, tp,
                                                     first, length, slot, ld);
}
