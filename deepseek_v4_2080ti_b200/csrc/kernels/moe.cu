// Routed-expert plumbing around the grouped GEMM (gemm_wdec.cu, grouped mode):
//   moe_route        - scores (softmax | sigmoid | sqrt-softplus) + selection bias + top-k + weight normalisation;
//   moe_plan         - counting sort of the (token, k) routes by local expert: per-expert offsets, the row of every
//                      route in expert-sorted order, and the (expert, m_tile, row0, rows) work table of both grouped
//                      GEMMs, all on the device (nothing is read back by the host);
//   moe_gather       - token rows -> expert-sorted rows;
//   moe_glu          - gated unit on the sorted rows: silu(gate) * up (with the DeepSeek clamp) or the one-plus form;
//   moe_combine      - out[t] = (shared[t]) + sum_k w[t,k] * y[row(t,k)], k ascending (deterministic).
// Routes whose expert lives on another rank are dropped locally (expert-range sharding) or carried by the
// dispatch kernels of csrc/comm.
// Reference counterparts: gate_topk_finalize (cpp_engine/backends/cuda/kernels/bf16_ops.cu:179-295),
// moe_route_count/prefix/fill (fp4_ops.cu:100-137), gather/scatter routes (src/csrc/cuda_kernel_impl.cu:264-331),
// moe_finalize_reduce (:4917).
#include <cuda_bf16.h>
#include <stdint.h>
#include "glu.cuh"
#include "ops.h"
#include "vec8.cuh"

namespace {

constexpr int MAX_EXPERTS = 1024;

__device__ __forceinline__ float score_fn(float x, int fn) {
  if (fn == 1) return 1.f / (1.f + expf(-x));                         // sigmoid
  if (fn == 2) return sqrtf(x > 20.f ? x : log1pf(expf(x)));          // sqrt(softplus)
  return x;                                                           // the softmaxes are handled by the caller
}

// One warp per token. logits fp32 [T, ld], the first E of a row; bias fp32 [E] or null; E <= 32 J.
template <int J>
__global__ void moe_route_kernel(const float* __restrict__ logits, int ld, const float* __restrict__ bias, int T, int E, int K,
                                 int fn, int norm_topk, float route_scale, int* __restrict__ idx,
                                 float* __restrict__ wts) {
  const int t = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (t >= T) return;
  const float* row = logits + (size_t)t * ld;
  // softmax statistics
  float mx = -INFINITY, den = 1.f;
  if (fn == 0) {
    for (int e = lane; e < E; e += 32) mx = fmaxf(mx, row[e]);
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    den = 0.f;
    for (int e = lane; e < E; e += 32) den += expf(row[e] - mx);
    for (int o = 16; o > 0; o >>= 1) den += __shfl_xor_sync(0xffffffffu, den, o);
  }
  // each lane keeps the scores of experts lane, lane + 32, ...
  float sc[J], sel[J];
#pragma unroll
  for (int j = 0; j < J; ++j) {
    const int e = j * 32 + lane;
    if (e < E) {
      sc[j] = fn == 0 ? expf(row[e] - mx) / den : score_fn(row[e], fn);
      sel[j] = sc[j] + (bias ? bias[e] : 0.f);
      if (fn == 3) sc[j] = sel[j];                                    // the bias belongs to the logit
    } else {
      sc[j] = 0.f;
      sel[j] = -INFINITY;
    }
  }
  float wsum = 0.f, top = 0.f;
  for (int k = 0; k < K; ++k) {
    float best = -INFINITY;
    int be = 0x7fffffff;
#pragma unroll
    for (int j = 0; j < J; ++j) {
      const int e = j * 32 + lane;
      if (sel[j] > best || (sel[j] == best && e < be)) { best = sel[j]; be = e; }
    }
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oe = __shfl_xor_sync(0xffffffffu, be, o);
      if (ob > best || (ob == best && oe < be)) { best = ob; be = oe; }
    }
    // the owning lane reports the unbiased score and retires the expert
    float w = 0.f;
#pragma unroll
    for (int j = 0; j < J; ++j)
      if (j * 32 + lane == be) { w = sc[j]; sel[j] = -INFINITY; }
    for (int o = 16; o > 0; o >>= 1) w += __shfl_xor_sync(0xffffffffu, w, o);
    if (fn == 3) {                                                    // softmax over the chosen: the first is the largest
      if (k == 0) top = w;
      w = expf(w - top);
    }
    wsum += w;
    if (lane == (k & 31)) {
      idx[(size_t)t * K + k] = be;
      wts[(size_t)t * K + k] = w * route_scale;
    }
  }
  if (fn != 0 && norm_topk)
    for (int k = lane; k < K; k += 32) wts[(size_t)t * K + k] /= wsum;     // lane k & 31 wrote entry k
}

__device__ __forceinline__ int warp_scan(int v, int lane) {                // inclusive
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int u = __shfl_up_sync(0xffffffffu, v, o);
    if (lane >= o) v += u;
  }
  return v;
}
// Exclusive prefix sum over a block of 1024 threads; `ws` holds 32 ints; total: the block's sum.
__device__ __forceinline__ int block_scan(int v, int* ws, int& total) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int inc = warp_scan(v, lane);
  if (lane == 31) ws[warp] = inc;
  __syncthreads();
  if (warp == 0) ws[lane] = warp_scan(ws[lane], lane);
  __syncthreads();
  const int base = warp ? ws[warp - 1] : 0;
  total = ws[31];
  __syncthreads();
  return base + inc - v;
}

// One block of 1024 threads per local expert.  idx [R] global expert ids (R = T*K); experts [lo, hi) are local.
// Outputs: offsets [EL+1], route_row [R] (row in sorted order or -1), row_token [rows] (source token of a sorted row),
// work tables for token tiles of bn13 / bn2 rows, counts.  Every block counts all routes, so that it knows where its expert's
// rows and work entries begin, and places its own expert's routes in their order (stable: results are run-to-run identical).
__global__ void __launch_bounds__(1024)
moe_plan_kernel(const int* __restrict__ idx, int R, int K, int lo, int hi, int* __restrict__ offsets,
                int* __restrict__ route_row, int* __restrict__ row_token, int4* __restrict__ work13, int* __restrict__ n13,
                int m_tiles13, int bn13, int4* __restrict__ work2, int* __restrict__ n2, int m_tiles2, int bn2,
                int max_work) {
  __shared__ int cnt[MAX_EXPERTS], ws[32], mine[4];
  const int EL = hi - lo, e = blockIdx.x, tid = threadIdx.x;
  cnt[tid] = 0;
  __syncthreads();
  constexpr int U = 8;                     // neighbouring routes per thread and round, two 16-byte loads
  auto load = [&](int r, int (&x)[U]) {    // local expert of routes r .. r + 7; -1: none
#pragma unroll
    for (int u = 0; u < U; u += 4) {
      int4 v = make_int4(-1, -1, -1, -1);
      if (r + u + 4 <= R) {
        v = *reinterpret_cast<const int4*>(idx + r + u);
      } else {
        if (r + u < R) v.x = idx[r + u];
        if (r + u + 1 < R) v.y = idx[r + u + 1];
        if (r + u + 2 < R) v.z = idx[r + u + 2];
      }
      x[u] = v.x - lo; x[u + 1] = v.y - lo; x[u + 2] = v.z - lo; x[u + 3] = v.w - lo;
    }
  };
#pragma unroll 2
  for (int r = tid * U; r < R; r += 1024 * U) {
    int x[U];
    load(r, x);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (r + u >= R) break;
      if (x[u] >= 0 && x[u] < EL) atomicAdd(&cnt[x[u]], 1);
      else if (e == 0) route_row[r + u] = -1;
    }
  }
  __syncthreads();
  const int c_t = tid < EL ? cnt[tid] : 0;                                 // thread t stands for expert t here
  int total, total13, total2;
  const int off_t = block_scan(c_t, ws, total);
  const int w13_t = block_scan(m_tiles13 * ((c_t + bn13 - 1) / bn13), ws, total13);
  const int w2_t = block_scan(m_tiles2 * ((c_t + bn2 - 1) / bn2), ws, total2);
  if (e == 0) {
    if (tid < EL) offsets[tid] = off_t;
    if (tid == 0) {
      offsets[EL] = total;
      *n13 = min(total13, max_work);
      *n2 = min(total2, max_work);
    }
  }
  if (tid == e) { mine[0] = c_t; mine[1] = off_t; mine[2] = w13_t; mine[3] = w2_t; }
  __syncthreads();
  const int c = mine[0], off = mine[1];
  if (c == 0) return;
  int placed = 0;
  for (int r0 = 0; r0 < R && placed < c; r0 += 1024 * U) {
    const int r = r0 + tid * U;
    int x[U], hits = 0, n;
    load(r, x);
#pragma unroll
    for (int u = 0; u < U; ++u) hits |= (r + u < R && x[u] == e) << u;
    int at = off + placed + block_scan(__popc(hits), ws, n);
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (hits >> u & 1) {
        route_row[r + u] = at;
        row_token[at++] = (r + u) / K;
      }
    placed += n;
  }
  // work tables: m-tile fastest inside a token tile so one expert's weight tiles are swept once per token tile
  auto emit = [&](int4* work, int base, int m_tiles, int bn) {
    const int n = m_tiles * ((c + bn - 1) / bn);
    for (int i = tid; i < n; i += 1024) {
      const int nt = i / m_tiles;
      if (base + i < max_work) work[base + i] = make_int4(e, i - nt * m_tiles, off + nt * bn, min(bn, c - nt * bn));
    }
  };
  emit(work13, mine[2], m_tiles13, bn13);
  emit(work2, mine[3], m_tiles2, bn2);
}

// xs[row, :] = x[row_token[row], :]; one block per sorted row; H % 8 == 0.
__global__ void moe_gather_kernel(const __nv_bfloat16* __restrict__ x, const int* __restrict__ row_token,
                                  const int* __restrict__ offsets, int EL, __nv_bfloat16* __restrict__ xs, int H) {
  const int row = blockIdx.x;
  if (row >= offsets[EL]) return;
  const uint4* src = reinterpret_cast<const uint4*>(x + (size_t)row_token[row] * H);
  uint4* dst = reinterpret_cast<uint4*>(xs + (size_t)row * H);
  for (int i = threadIdx.x; i < H / 8; i += blockDim.x) dst[i] = src[i];
}

// rows [gate | up] of 2 I columns -> gated unit (glu.cuh); slope 0: silu(min(g, limit)) clamp(u), the limit optional.
template <typename T>
__global__ void moe_glu_kernel(const T* __restrict__ gu, const int* __restrict__ offsets, int EL, T* __restrict__ act, int I,
                               float limit, float slope) {
  const int row = blockIdx.x;
  if (row >= offsets[EL]) return;
  const T* g = gu + (size_t)row * 2 * I;
  const b200::GluShape shape = {limit, slope};
  for (int i = threadIdx.x * 8; i < I; i += blockDim.x * 8) {
    float gv[8], uv[8];
    b200::load8(g + i, gv);
    b200::load8(g + I + i, uv);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (slope > 0.f) {
        gv[j] = b200::glu<sizeof(T) == 2>(gv[j], uv[j], shape);
        continue;
      }
      if (limit > 0.f) {
        uv[j] = fminf(fmaxf(uv[j], -limit), limit);
        gv[j] = fminf(gv[j], limit);
      }
      gv[j] = __fdividef(gv[j], 1.f + __expf(-gv[j])) * uv[j];
    }
    b200::store8(act + (size_t)row * I + i, gv);
  }
}

// out[t, :] = base[t, :] (optional) + sum_k wts[t,k] * y[route_row[t,k], :]
__global__ void moe_combine_kernel(const __nv_bfloat16* __restrict__ y, const int* __restrict__ route_row,
                                   const float* __restrict__ wts, const __nv_bfloat16* __restrict__ base,
                                   __nv_bfloat16* __restrict__ out, int K, int H) {
  const int t = blockIdx.x;
  for (int h = threadIdx.x; h < H; h += blockDim.x) {
    float acc = base ? __bfloat162float(base[(size_t)t * H + h]) : 0.f;
    for (int k = 0; k < K; ++k) {
      const int r = route_row[(size_t)t * K + k];
      if (r >= 0) acc += wts[(size_t)t * K + k] * __bfloat162float(y[(size_t)r * H + h]);
    }
    out[(size_t)t * H + h] = __float2bfloat16(acc);
  }
}

}  // namespace

extern "C" {

// score_fn: 0 softmax, 1 sigmoid, 2 sqrt(softplus). logits rows of `ld` floats; idx int32 [T, K], wts fp32 [T, K].
int b200_moe_route(const float* logits, int ld, const float* bias, int T, int E, int K, int score_fn, int norm_topk,
                   float route_scale, int* idx, float* wts, cudaStream_t stream) {
  if (T <= 0 || E <= 0 || E > MAX_EXPERTS || K <= 0 || K > E || ld < E) return -6;
  const int wpb = 4;
  const dim3 grid((T + wpb - 1) / wpb), block(wpb * 32);
#define B200_ROUTE(J)                                                                                                 \
  if (E <= 32 * J) {                                                                                                  \
    moe_route_kernel<J><<<grid, block, 0, stream>>>(logits, ld, bias, T, E, K, score_fn, norm_topk, route_scale, idx, wts); \
    return (int)cudaGetLastError();                                                                                   \
  }
  B200_ROUTE(1) B200_ROUTE(2) B200_ROUTE(4) B200_ROUTE(8) B200_ROUTE(16) B200_ROUTE(32)
#undef B200_ROUTE
  return -6;
}

// Plans the grouped GEMMs of this rank's experts [expert_lo, expert_hi).  All outputs are device buffers:
// offsets int32 [EL+1]; route_row int32 [T*K]; row_token int32 [T*K]; work13 / work2: int4 [max_work]; n13 / n2: int32 [1].
int b200_moe_plan(const int* idx, int T, int K, int expert_lo, int expert_hi, int* offsets, int* route_row,
                  int* row_token, void* work13, int* n13, int m_tiles13, int bn13, void* work2, int* n2, int m_tiles2,
                  int bn2, int max_work, cudaStream_t stream) {
  const int EL = expert_hi - expert_lo;
  if (T <= 0 || K <= 0 || EL <= 0 || EL > MAX_EXPERTS || max_work <= 0) return -6;
  moe_plan_kernel<<<EL, 1024, 0, stream>>>(idx, T * K, K, expert_lo, expert_hi, offsets, route_row, row_token,
                                          reinterpret_cast<int4*>(work13), n13, m_tiles13, bn13,
                                          reinterpret_cast<int4*>(work2), n2, m_tiles2, bn2, max_work);
  return (int)cudaGetLastError();
}

int b200_moe_gather(const void* x, const int* row_token, const int* offsets, int EL, void* xs, int max_rows, int H,
                    cudaStream_t stream) {
  if (max_rows <= 0 || H % 8) return -6;
  moe_gather_kernel<<<max_rows, 128, 0, stream>>>(reinterpret_cast<const __nv_bfloat16*>(x), row_token, offsets, EL,
                                                  reinterpret_cast<__nv_bfloat16*>(xs), H);
  return (int)cudaGetLastError();
}

// slope > 0: the clamped one-plus unit of glu.cuh, else SwiGLU with the optional clamp.  I % 8 == 0.
int b200_moe_glu(const void* gu, const int* offsets, int EL, void* act, int max_rows, int I, float limit, float slope, int f32,
                 cudaStream_t stream) {
  if (max_rows <= 0 || I <= 0 || (I & 7)) return -6;
  const int threads = I >= 2048 ? 256 : I >= 1024 ? 128 : I >= 512 ? 64 : 32;
  if (f32)
    moe_glu_kernel<float><<<max_rows, threads, 0, stream>>>(reinterpret_cast<const float*>(gu), offsets, EL,
                                                            reinterpret_cast<float*>(act), I, limit, slope);
  else
    moe_glu_kernel<__nv_bfloat16><<<max_rows, threads, 0, stream>>>(reinterpret_cast<const __nv_bfloat16*>(gu), offsets, EL,
                                                                    reinterpret_cast<__nv_bfloat16*>(act), I, limit, slope);
  return (int)cudaGetLastError();
}

int b200_moe_combine(const void* y, const int* route_row, const float* wts, const void* base, void* out, int T, int K,
                     int H, cudaStream_t stream) {
  if (T <= 0 || K <= 0 || H <= 0) return -6;
  moe_combine_kernel<<<T, 256, 0, stream>>>(reinterpret_cast<const __nv_bfloat16*>(y), route_row, wts,
                                            reinterpret_cast<const __nv_bfloat16*>(base),
                                            reinterpret_cast<__nv_bfloat16*>(out), K, H);
  return (int)cudaGetLastError();
}

}  // extern "C"
