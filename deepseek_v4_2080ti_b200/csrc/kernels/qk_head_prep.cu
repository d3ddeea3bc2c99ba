// Attention prologue without a rotation, one block per token: every query and key vector (one per head, or one per head
// and map) is RMS-normalised over its own `dim` values with a weight all vectors share; queries are scaled by a
// temperature that grows with the position,  1 + coef ln(floor((p + 1) / every) + 1)  (every <= 0: none); keys and values
// are appended to the paged cache.  A layer that attends over another layer's cache passes n_k = v_width = 0.
//
// Vectors are D wide in memory (a multiple of 8; columns past `dim` are zero and stay zero).
#include "launch.h"
#include "ops.h"
#include "vec8.cuh"

namespace {
using namespace b200;

template <typename T>
struct QkHeadParams {
  const T* proj;             // [T, ld]
  int ld, q_off, k_off, v_off, n_q, n_k, v_width, D;
  const float *q_w, *k_w;    // [D]
  float inv_dim, eps, coef;
  double every;
  const int *positions, *slots;
  T* q;                      // [T, n_q * D]
  T *k_cache, *v_cache;      // [pages * page size, n_k * D], [.., v_width]
};

template <typename T>
__global__ void __launch_bounds__(256) qk_head_prep_kernel(QkHeadParams<T> p, int lanes) {
  pdl_grid_trigger();
  pdl_grid_wait();
  const int t = blockIdx.x, slot = p.slots[t];
  float temp = 1.f;
  if (p.every > 0.0) temp = 1.f + p.coef * logf((float)floor((double)(p.positions[t] + 1) / p.every) + 1.f);
  const T* row = p.proj + (size_t)t * p.ld;
  const int lane = threadIdx.x % lanes, groups = blockDim.x / lanes, n = p.n_q + p.n_k;
  // whole warps take every pass (the sums below are shuffles): the bound is rounded up to the groups of a block
  for (int base = 0; base < n; base += groups) {
    const int v = base + threadIdx.x / lanes;
    const bool on = v < n, is_q = v < p.n_q;
    const T* src = row + (is_q ? p.q_off + v * p.D : p.k_off + (v - p.n_q) * p.D);
    float ss = 0.f;
    for (int d = lane * 8; on && d < p.D; d += lanes * 8) {
      float f[8];
      load8(src + d, f);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += f[j] * f[j];
    }
    for (int o = lanes / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (!on || (!is_q && slot < 0)) continue;
    const float inv = (is_q ? temp : 1.f) / sqrtf(ss * p.inv_dim + p.eps);
    T* dst = is_q ? p.q + ((size_t)t * p.n_q + v) * p.D : p.k_cache + ((size_t)slot * p.n_k + (v - p.n_q)) * p.D;
    const float* w = is_q ? p.q_w : p.k_w;
    for (int d = lane * 8; d < p.D; d += lanes * 8) {
      float f[8], g[8];
      load8(src + d, f);
      load8(w + d, g);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] = f[j] * inv * g[j];
      store8(dst + d, f);
    }
  }
  if (slot < 0) return;
  for (int v = threadIdx.x * 8; v < p.v_width; v += blockDim.x * 8) {
    float f[8];
    load8(row + p.v_off + v, f);
    store8(p.v_cache + (size_t)slot * p.v_width + v, f);
  }
}

template <typename T>
int run_qk_head(const void* proj, int ld, int q_off, int k_off, int v_off, int n_q, int n_k, int v_width, int D, int dim,
                const float* q_w, const float* k_w, float eps, float coef, double every, const int* positions, const int* slots,
                void* q, void* k_cache, void* v_cache, int rows, cudaStream_t stream) {
  QkHeadParams<T> p;
  p.proj = reinterpret_cast<const T*>(proj); p.ld = ld; p.q_off = q_off; p.k_off = k_off; p.v_off = v_off; p.n_q = n_q;
  p.n_k = n_k; p.v_width = v_width; p.D = D; p.q_w = q_w; p.k_w = k_w; p.inv_dim = 1.f / (float)dim; p.eps = eps;
  p.coef = coef; p.every = every; p.positions = positions; p.slots = slots; p.q = reinterpret_cast<T*>(q);
  p.k_cache = reinterpret_cast<T*>(k_cache); p.v_cache = reinterpret_cast<T*>(v_cache);
  int lanes = 1;
  while (lanes < 32 && lanes * 8 < D) lanes *= 2;
  int threads = 64;
  while (threads < 256 && threads < (n_q + n_k) * lanes) threads *= 2;
  return (int)launch_pdl(qk_head_prep_kernel<T>, dim3(rows), dim3(threads), 0, stream, p, lanes);
}

}  // namespace

extern "C" int b200_qk_head_prep(const void* proj, int ld, int q_off, int k_off, int v_off, int n_q, int n_k, int v_width, int D,
                                 int dim, const float* q_w, const float* k_w, float eps, float coef, double every,
                                 const int* positions, const int* slots, void* q, void* k_cache, void* v_cache, int rows, int f32,
                                 cudaStream_t stream) {
  if (rows <= 0 || n_q <= 0 || n_k < 0 || v_width < 0 || D <= 0 || (D & 7) || dim <= 0 || dim > D || (ld & 7) || (q_off & 7) ||
      (k_off & 7) || (v_off & 7) || (v_width & 7) || !q || (n_k > 0 && (!k_cache || !k_w)) || (v_width > 0 && !v_cache))
    return -6;
  return f32 ? run_qk_head<float>(proj, ld, q_off, k_off, v_off, n_q, n_k, v_width, D, dim, q_w, k_w, eps, coef, every, positions,
                                  slots, q, k_cache, v_cache, rows, stream)
             : run_qk_head<__nv_bfloat16>(proj, ld, q_off, k_off, v_off, n_q, n_k, v_width, D, dim, q_w, k_w, eps, coef, every,
                                          positions, slots, q, k_cache, v_cache, rows, stream);
}
