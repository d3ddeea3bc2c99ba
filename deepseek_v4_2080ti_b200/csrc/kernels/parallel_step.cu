// Step between the layers of a decoder whose two sublayers read the same norm and are added side by side:
//
//   x' = x + mix sigmoid(g1 + b1) + ff sigmoid(g2 + b2)          element-wise gates; the residual is fp32
//   ff = sum_k w_k y_k + sigmoid(sg) shared                      routed experts, identity experts (y = h of the layer), one
//                                                                shared expert behind a gate of its own per row
//   h' = x' / rms(x') * weight                                   one weight for all columns
//   m' = h' + (h'(row before) - h') shift                        what a mixer with a token shift reads
//
// one launch per layer; every part is optional.  The row may start from an embedding table.  The row before is the
// neighbouring row of the same portion, the sequence's stored tail where a portion begins, or zero at position 0.  A block
// takes a run of rows and keeps the last h' in registers; the run's first row works its predecessor out again, which is why
// the residual goes to another buffer than it comes from.  Single rows replace their sequence's tail here (one block reads
// and writes it); the tails of longer portions are replaced by shift_tails_kernel once every reader is done.
// h' is rounded to the activations' type before the shift, so that a stored tail and a neighbour give the same result.
#include "launch.h"
#include "ops.h"
#include "vec8.cuh"

namespace {
using namespace b200;

template <typename T>
struct ParallelStepParams {
  const float* x;            // [rows, ld]
  float* x_out;              // [rows, ld] or null, not x
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
  T* m_out;                  // [rows, ld] or null
  const float* shift;        // [ld]
  T* tail;                   // [slots, ld]
  const int *row_first, *row_slot, *positions;
  const int* rows;           // not null: output row i is stored row rows[i]
  int n, ld, cols, run;
};

__device__ __forceinline__ float sigmoidf(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float rounded(float v, __nv_bfloat16) { return __bfloat162float(__float2bfloat16(v)); }
__device__ __forceinline__ float rounded(float v, float) { return v; }

template <typename T, int VEC>
__global__ void parallel_step_kernel(ParallelStepParams<T> p) {
  __shared__ float red[32];
  pdl_grid_trigger();
  pdl_grid_wait();
  const int nvec = p.ld >> 3;
  const float inv_n = 1.f / (float)p.cols;
  float h[VEC][8];           // the row's norm output, rounded

  // h <- norm of the advanced residual of `row`; stores the residual when asked
  auto advance = [&](size_t row, bool store_x) {
    const T* src_row = nullptr;
    if (p.ids) {
      const int id = p.ids[row];
      if (id >= 0 && id < p.vocab) src_row = p.table + (size_t)id * p.ld;
    }
    const float sg = p.shared ? (p.shared_gate ? sigmoidf(p.shared_gate[row * p.ld_shared_gate]) : 1.f) : 0.f;
    float ss = 0.f;
#pragma unroll
    for (int it = 0; it < VEC; ++it) {
      const int v = threadIdx.x + it * blockDim.x;
      float x[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      if (v < nvec) {
        const size_t at = row * p.ld + v * 8;
        float a[8], g[8], b[8];
        if (!p.ids) load8(p.x + at, x);
        else if (src_row) load8(src_row + v * 8, x);
        if (p.mix) {
          load8(p.mix + at, a);
          load8(p.gates + row * p.ld_gates + v * 8, g);
          load8(p.gate_b + v * 8, b);
#pragma unroll
          for (int j = 0; j < 8; ++j) x[j] = fmaf(a[j], sigmoidf(g[j] + b[j]), x[j]);
        }
        if (p.routed || p.shared) {
          float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
          if (p.routed) {
            float id_w = 0.f;
            for (int k = 0; k < p.top; ++k) {
              const size_t r = row * p.top + k;
              const float w = p.route_w[r];
              if (p.route_id[r] >= p.experts) { id_w += w; continue; }
              const int at_row = p.route_row[r];
              if (at_row < 0) continue;
              load8(p.routed + (size_t)at_row * p.ld_routed + v * 8, a);
#pragma unroll
              for (int j = 0; j < 8; ++j) f[j] = fmaf(w, a[j], f[j]);
            }
            if (id_w != 0.f) {
              load8(p.h + at, a);
#pragma unroll
              for (int j = 0; j < 8; ++j) f[j] = fmaf(id_w, a[j], f[j]);
            }
          }
          if (p.shared) {
            load8(p.shared + at, a);
#pragma unroll
            for (int j = 0; j < 8; ++j) f[j] = fmaf(sg, a[j], f[j]);
          }
          load8(p.gates + row * p.ld_gates + p.ld + v * 8, g);
          load8(p.gate_b + p.ld + v * 8, b);
#pragma unroll
          for (int j = 0; j < 8; ++j) x[j] = fmaf(f[j], sigmoidf(g[j] + b[j]), x[j]);
        }
        if (store_x) store8(p.x_out + at, x);
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        h[it][j] = v * 8 + j < p.cols ? x[j] : 0.f;
        ss += h[it][j] * h[it][j];
      }
    }
    if (!p.h_out && !p.m_out) return;
    const float f = p.weight / sqrtf(block_sum_all(ss, red) * inv_n + p.eps);
#pragma unroll
    for (int it = 0; it < VEC; ++it)
#pragma unroll
      for (int j = 0; j < 8; ++j) h[it][j] = rounded(h[it][j] * f, T());
  };

  const int r0 = blockIdx.x * p.run, r1 = min(p.n, r0 + p.run);
  if (p.m_out && p.row_first[r0] != r0) advance(r0 - 1, false);
  for (int r = r0; r < r1; ++r) {
    const size_t row = p.rows ? (size_t)p.rows[r] : (size_t)r;
    float before[VEC][8];
    int first = 0, slot = 0, pos = 0;
    if (p.m_out) {
      first = p.row_first[r];
      slot = p.row_slot[r];
      pos = p.positions[r];
#pragma unroll
      for (int it = 0; it < VEC; ++it) {
        const int v = threadIdx.x + it * blockDim.x;
        if (first == r) {
          if (pos > 0 && v < nvec) load8(p.tail + (size_t)slot * p.ld + v * 8, before[it]);
          else
#pragma unroll
            for (int j = 0; j < 8; ++j) before[it][j] = 0.f;
        } else {
#pragma unroll
          for (int j = 0; j < 8; ++j) before[it][j] = h[it][j];
        }
      }
    }
    advance(row, p.x_out != nullptr);
    const bool alone = p.m_out && first == r && (r + 1 >= p.n || p.row_first[r + 1] != first);
#pragma unroll
    for (int it = 0; it < VEC; ++it) {
      const int v = threadIdx.x + it * blockDim.x;
      if (v >= nvec) continue;
      if (p.h_out) store8(p.h_out + (size_t)r * p.ld + v * 8, h[it]);
      if (p.m_out) {
        float s[8], m[8];
        load8(p.shift + v * 8, s);
#pragma unroll
        for (int j = 0; j < 8; ++j) m[j] = fmaf(before[it][j] - h[it][j], s[j], h[it][j]);
        store8(p.m_out + (size_t)r * p.ld + v * 8, m);
        if (alone) store8(p.tail + (size_t)slot * p.ld + v * 8, h[it]);
      }
    }
  }
}

// tail[slot] = h[last row] of every entry with more than one row.
template <typename T>
__global__ void shift_tails_kernel(const T* __restrict__ h, T* __restrict__ tail, const int* __restrict__ first,
                                   const int* __restrict__ length, const int* __restrict__ slot, int ld) {
  pdl_grid_trigger();
  pdl_grid_wait();
  const int e = blockIdx.x, n = length[e];
  if (n < 2) return;
  const T* src = h + (size_t)(first[e] + n - 1) * ld;
  T* dst = tail + (size_t)slot[e] * ld;
  for (int v = threadIdx.x; v < ld / 8; v += blockDim.x) {
    float f[8];
    load8(src + v * 8, f);
    store8(dst + v * 8, f);
  }
}

template <typename T>
int run_parallel_step(ParallelStepParams<T> p, cudaStream_t stream) {
  const int nvec = p.ld >> 3;
  int threads = (nvec + 31) / 32 * 32;
  if (threads > 512) threads = 512;
  const int vec = (nvec + threads - 1) / threads;
  // runs of rows only where they share a predecessor and the machine stays full
  p.run = p.m_out && !p.rows && p.n > 148 * 8 ? 8 : 1;
  const dim3 grid((p.n + p.run - 1) / p.run), block(threads);
  if (vec == 1) return (int)launch_pdl(parallel_step_kernel<T, 1>, grid, block, 0, stream, p);
  if (vec == 2) return (int)launch_pdl(parallel_step_kernel<T, 2>, grid, block, 0, stream, p);
  if (vec <= 4) return (int)launch_pdl(parallel_step_kernel<T, 4>, grid, block, 0, stream, p);
  return -6;
}

template <typename T>
int make_parallel_step(const float* x, float* x_out, const int* ids, const void* table, int vocab, const void* mix, const void* gates,
                       int ld_gates, const float* gate_b, const void* h, const void* routed, int ld_routed, const int* route_row,
                       const int* route_id, const float* route_w, int top, int experts, const void* shared, const float* shared_gate,
                       int ld_shared_gate, float weight, float eps, void* h_out, void* m_out, const float* shift, void* tail,
                       const int* row_first, const int* row_slot, const int* positions, const int* rows, int n, int ld, int cols,
                       cudaStream_t stream) {
  ParallelStepParams<T> p;
  p.x = x; p.x_out = x_out; p.ids = ids; p.table = reinterpret_cast<const T*>(table); p.vocab = vocab;
  p.mix = reinterpret_cast<const T*>(mix); p.gates = reinterpret_cast<const T*>(gates); p.gate_b = gate_b; p.ld_gates = ld_gates;
  p.h = reinterpret_cast<const T*>(h); p.routed = reinterpret_cast<const T*>(routed); p.route_row = route_row;
  p.route_id = route_id; p.route_w = route_w; p.ld_routed = ld_routed; p.top = top; p.experts = experts;
  p.shared = reinterpret_cast<const T*>(shared); p.shared_gate = shared_gate; p.ld_shared_gate = ld_shared_gate;
  p.weight = weight; p.eps = eps; p.h_out = reinterpret_cast<T*>(h_out); p.m_out = reinterpret_cast<T*>(m_out); p.shift = shift;
  p.tail = reinterpret_cast<T*>(tail); p.row_first = row_first; p.row_slot = row_slot; p.positions = positions; p.rows = rows;
  p.n = n; p.ld = ld; p.cols = cols; p.run = 1;
  return run_parallel_step(p, stream);
}

}  // namespace

// n rows of width ld (a multiple of 8, at most 16384; columns past `cols` are zero); f32 != 0: activations are fp32, else bf16.
extern "C" int b200_parallel_step(const float* x, float* x_out, const int* ids, const void* table, int vocab, const void* mix,
                                  const void* gates, int ld_gates, const float* gate_b, const void* h, const void* routed,
                                  int ld_routed, const int* route_row, const int* route_id, const float* route_w, int top,
                                  int experts, const void* shared, const float* shared_gate, int ld_shared_gate, float weight,
                                  float eps, void* h_out, void* m_out, const float* shift, void* tail, const int* row_first,
                                  const int* row_slot, const int* positions, const int* rows, int n, int ld, int cols, int f32,
                                  cudaStream_t stream) {
  if (n <= 0 || ld <= 0 || (ld & 7) || ld > 16384 || cols <= 0 || cols > ld) return -6;
  if ((!ids && !x) || (ids && !table) || (x_out && x_out == x) || ((mix || routed || shared) && (!gates || !gate_b))) return -6;
  if (ld_gates & 7 || ld_routed & 7 || (routed && (!route_row || !route_id || !route_w || !h || top <= 0 || ld_routed < ld))) return -6;
  if (m_out && (!shift || !tail || !row_first || !row_slot || !positions || rows)) return -6;
  return f32 ? make_parallel_step<float>(x, x_out, ids, table, vocab, mix, gates, ld_gates, gate_b, h, routed, ld_routed, route_row,
                                         route_id, route_w, top, experts, shared, shared_gate, ld_shared_gate, weight, eps, h_out,
                                         m_out, shift, tail, row_first, row_slot, positions, rows, n, ld, cols, stream)
             : make_parallel_step<__nv_bfloat16>(x, x_out, ids, table, vocab, mix, gates, ld_gates, gate_b, h, routed, ld_routed,
                                                 route_row, route_id, route_w, top, experts, shared, shared_gate, ld_shared_gate,
                                                 weight, eps, h_out, m_out, shift, tail, row_first, row_slot, positions, rows, n, ld,
                                                 cols, stream);
}

extern "C" int b200_shift_tails(const void* h, void* tail, const int* first, const int* length, const int* slot, int entries, int ld,
                                int f32, cudaStream_t stream) {
  if (entries <= 0 || ld <= 0 || (ld & 7)) return -6;
  if (f32)
    return (int)launch_pdl(shift_tails_kernel<float>, dim3(entries), dim3(256), 0, stream, reinterpret_cast<const float*>(h),
                           reinterpret_cast<float*>(tail), first, length, slot, ld);
  return (int)launch_pdl(shift_tails_kernel<__nv_bfloat16>, dim3(entries), dim3(256), 0, stream,
                         reinterpret_cast<const __nv_bfloat16*>(h), reinterpret_cast<__nv_bfloat16*>(tail), first, length, slot, ld);
}
