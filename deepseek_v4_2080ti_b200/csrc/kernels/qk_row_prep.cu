// Attention prologue for heads whose scores are mixed across heads: one block per token.
//
//   q, k   RMS-normalised over the WHOLE projection row (all heads at once), weights per (head, dim)
//          then rotated: interleaved pairs (2i, 2i + 1) of the first `rot` dims of every head, frequency table and one
//          factor on cos and sin given by the caller (angles in fp64, sine and cosine in fp32)
//   cache  k as rotated; v as given (for shared key/value projections the caller passes the raw key columns)
//   q_mix  [n_mix, H, G * D] bf16 (first n_mix tokens): row h is the H x H head mixing folded into the query,
//          q_mix[h, c * D + d] = sum over the query heads g of group c of talk[h, g] q[g, d], so that
//          q_mix[h] . (all key heads of a token side by side) = sum_g talk[h, g] (q_g . k_group(g))
//   q_row  [T - n_mix, H, D] fp32 (the other tokens): plain rotated queries
//
// D is a multiple of 8 (heads padded with zero rows by the loader); the norm's mean runs over q_count / k_count values.
#include "launch.h"
#include "ops.h"
#include "per_device.h"
#include "vec8.cuh"

namespace {
using namespace b200;

template <typename T>
struct QkRowParams {
  const T* proj;             // [T, ld]: q at q_off, k at k_off, v at v_off
  int ld, q_off, k_off, v_off;
  const float *q_w, *k_w;    // [H * D], [G * D]
  float q_count, k_count, eps;
  const double* freq;        // [rot / 2]
  int rot;
  float mscale;
  const float* talk_t;       // [H (g), H4 (h)]: transposed mixing matrix, rows padded to a multiple of 4
  const int *positions, *slots;
  __nv_bfloat16* q_mix;
  float* q_row;
  T *k_cache, *v_cache;      // [pages * page size, G * D]
  int T_, n_mix, H, G, D;
};

template <typename T>
__global__ void __launch_bounds__(256) qk_row_prep_kernel(QkRowParams<T> p) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[32];
  pdl_grid_trigger();
  pdl_grid_wait();
  const int t = blockIdx.x, H = p.H, D = p.D, KW = p.G * p.D, QW = H * D;
  float* sq = sm;                 // [QW]
  float* cs = sm + QW;            // [rot / 2] cos, then sin
  float* sn = cs + p.rot / 2;
  const int pos = p.positions[t], slot = p.slots[t];
  for (int i = threadIdx.x; i < p.rot / 2; i += blockDim.x) {
    double a = (double)pos * p.freq[i];
    a -= 6.283185307179586 * rint(a * 0.15915494309189535);
    float s, c;
    sincosf((float)a, &s, &c);
    cs[i] = c * p.mscale;
    sn[i] = s * p.mscale;
  }
  const T* row = p.proj + (size_t)t * p.ld;
  float ss = 0.f, kk = 0.f;
  for (int v = threadIdx.x; v < QW / 8; v += blockDim.x) {
    float f[8];
    load8(row + p.q_off + v * 8, f);
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += f[j] * f[j];
    store8(sq + v * 8, f);
  }
  for (int v = threadIdx.x; v < KW / 8; v += blockDim.x) {
    float f[8];
    load8(row + p.k_off + v * 8, f);
#pragma unroll
    for (int j = 0; j < 8; ++j) kk += f[j] * f[j];
  }
  const float qi = 1.f / sqrtf(block_sum_all(ss, red) / p.q_count + p.eps);
  const float ki = 1.f / sqrtf(block_sum_all(kk, red) / p.k_count + p.eps);   // its barriers also publish cs / sn / sq

  auto finish = [&](float (&f)[8], const float* w, int v, float inv) {
    float g[8];
    load8(w + v * 8, g);
#pragma unroll
    for (int j = 0; j < 8; ++j) f[j] = f[j] * inv * g[j];
    const int d0 = (v * 8) % D;
#pragma unroll
    for (int j = 0; j < 8; j += 2) {
      if (d0 + j < p.rot) {
        const float c = cs[(d0 + j) >> 1], s = sn[(d0 + j) >> 1], a = f[j], b = f[j + 1];
        f[j] = a * c - b * s;
        f[j + 1] = b * c + a * s;
      }
    }
  };
  const bool mix = t < p.n_mix;
  for (int v = threadIdx.x; v < QW / 8; v += blockDim.x) {      // same thread wrote this vector of sq
    float f[8];
    load8(sq + v * 8, f);
    finish(f, p.q_w, v, qi);
    if (mix) store8(sq + v * 8, f);
    else store8(p.q_row + ((size_t)(t - p.n_mix) * QW + v * 8), f);
  }
  if (slot >= 0) {
    for (int v = threadIdx.x; v < KW / 8; v += blockDim.x) {
      float f[8];
      load8(row + p.k_off + v * 8, f);
      finish(f, p.k_w, v, ki);
      store8(p.k_cache + (size_t)slot * KW + v * 8, f);
      load8(row + p.v_off + v * 8, f);
      store8(p.v_cache + (size_t)slot * KW + v * 8, f);
    }
  }
  if (!mix) return;
  __syncthreads();
  const int R = H / p.G, H4 = (H + 3) & ~3, cols = KW / 8;
  for (int i = threadIdx.x; i < cols * (H4 / 4); i += blockDim.x) {
    const int v = i % cols, h0 = (i / cols) * 4;
    const int c = (v * 8) / D, d = (v * 8) % D;
    float acc[4][8] = {};
    for (int r = 0; r < R; ++r) {
      const int g = c * R + r;
      const float4 tk = __ldg(reinterpret_cast<const float4*>(p.talk_t + (size_t)g * H4 + h0));
      float f[8];
      load8(sq + g * D + d, f);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        acc[0][j] = fmaf(tk.x, f[j], acc[0][j]);
        acc[1][j] = fmaf(tk.y, f[j], acc[1][j]);
        acc[2][j] = fmaf(tk.z, f[j], acc[2][j]);
        acc[3][j] = fmaf(tk.w, f[j], acc[3][j]);
      }
    }
#pragma unroll
    for (int u = 0; u < 4; ++u)
      if (h0 + u < H) store8(p.q_mix + ((size_t)t * H + h0 + u) * KW + v * 8, acc[u]);
  }
}

template <typename T>
int launch_qk_row(QkRowParams<T> p, cudaStream_t stream) {
  const size_t smem = ((size_t)p.H * p.D + p.rot) * sizeof(float);
  if (smem > 227 * 1024 - 256) return -6;
  static PerDeviceOnce once_;
  bool& configured = once_.slot();
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(qk_row_prep_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024 - 256);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  return (int)launch_pdl(qk_row_prep_kernel<T>, dim3(p.T_), dim3(256), smem, stream, p);
}

}  // namespace

extern "C" int b200_qk_row_prep(const void* proj, int ld, int q_off, int k_off, int v_off, const float* q_w, const float* k_w,
                                int q_count, int k_count, float eps, const double* freq, int rot, float mscale,
                                const float* talk_t, const int* positions, const int* slots, void* q_mix, float* q_row,
                                void* k_cache, void* v_cache, int T, int n_mix, int H, int G, int D, int f32,
                                cudaStream_t stream) {
  if (T <= 0 || H <= 0 || G <= 0 || H % G || D <= 0 || (D & 7) || (ld & 7) || (q_off & 7) || (k_off & 7) || (v_off & 7) ||
      rot < 0 || (rot & 1) || rot > D || n_mix < 0 || n_mix > T || (n_mix > 0 && (!q_mix || !talk_t)) || (n_mix < T && !q_row))
    return -6;
#define B200_FILL(TT)                                                                                                       \
  QkRowParams<TT> p;                                                                                                        \
  p.proj = reinterpret_cast<const TT*>(proj); p.ld = ld; p.q_off = q_off; p.k_off = k_off; p.v_off = v_off;                 \
  p.q_w = q_w; p.k_w = k_w; p.q_count = (float)q_count; p.k_count = (float)k_count; p.eps = eps; p.freq = freq; p.rot = rot; \
  p.mscale = mscale; p.talk_t = talk_t; p.positions = positions; p.slots = slots;                                           \
  p.q_mix = reinterpret_cast<__nv_bfloat16*>(q_mix); p.q_row = q_row; p.k_cache = reinterpret_cast<TT*>(k_cache);           \
  p.v_cache = reinterpret_cast<TT*>(v_cache); p.T_ = T; p.n_mix = n_mix; p.H = H; p.G = G; p.D = D;                         \
  return launch_qk_row(p, stream);
  if (f32) {
    B200_FILL(float)
  } else {
    B200_FILL(__nv_bfloat16)
  }
#undef B200_FILL
}
