// Gated linear attention: per head a state S [D, V] in fp32 with a decay per key channel,
//
//   S_t = diag(alpha_t) S_(t-1) + k_t v_t^T,     o_t = S_t^T q_t,     alpha = sigmoid(z)^(1 / tau)
//
// over a batch of rows of several sequences (entries of neighbouring rows, one state slot each; a portion that begins at
// position 0 starts from zero).  Head widths are padded to multiples of 16 with zero channels.
//
//   gla_decay    log alpha from the low-rank logits z = W2 a + b, fp32
//   gla_scan     one token after the other; the state's columns are independent, so a block takes 32 of them, a lane per
//                column, and the warps share the rows.  For fp32, and for bf16 portions too short for gla_chunk.cu
//   gla_step     one token of many sequences: a block per head and sequence reads, updates and writes the state once and
//                finishes the row (norm, gate) itself
//   gla_finish   per head o / rms(o) * weight * silu(g)
#include "launch.h"
#include "ops.h"
#include "per_device.h"
#include "vec8.cuh"

namespace {
using namespace b200;

__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

constexpr int DR = 8;           // rows per block of gla_decay

// a: [rows, >= rank] (row stride ld); w2 [channels, rank]; la [rows, channels].  rank a multiple of 8.
template <typename T>
__global__ void gla_decay_kernel(const T* __restrict__ a, int ld, const T* __restrict__ w2, const float* __restrict__ bias,
                                 float inv_tau, float* __restrict__ la, int rows, int channels, int rank) {
  extern __shared__ __align__(16) float sa[];   // [DR][rank]
  pdl_grid_trigger();
  pdl_grid_wait();
  const int r0 = blockIdx.x * DR, n = min(DR, rows - r0);
  for (int i = threadIdx.x; i < DR * rank; i += blockDim.x)
    sa[i] = i / rank < n ? (float)a[(size_t)(r0 + i / rank) * ld + i % rank] : 0.f;
  __syncthreads();
  for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < channels; c += gridDim.y * blockDim.x) {
    float z[DR];
#pragma unroll
    for (int r = 0; r < DR; ++r) z[r] = bias[c];
    for (int k = 0; k < rank; k += 8) {
      float w[8];
      load8(w2 + (size_t)c * rank + k, w);
#pragma unroll
      for (int r = 0; r < DR; ++r) {
        float a8[8];
        load8(sa + r * rank + k, a8);
#pragma unroll
        for (int j = 0; j < 8; ++j) z[r] = fmaf(w[j], a8[j], z[r]);
      }
    }
#pragma unroll
    for (int r = 0; r < DR; ++r)
      if (r < n) la[(size_t)(r0 + r) * channels + c] = log_sigmoid(z[r]) * inv_tau;
  }
}

template <typename T>
struct GlaParams {
  const T *q, *k, *v;        // head h of row t at ptr + t * ld + h * D (V)
  const float* la;           // [rows, H * D]
  float* state;              // [slots, H, D, V]
  float* o;                  // [rows, H * V]
  const int *first, *length, *slot, *positions;
  int ld, H, D, V;
  int max_len;               // longer entries are left alone (0: none)
  float scale;
};

constexpr int CT = 16;          // rows staged together
constexpr int SW = 8;           // warps

// grid (ceil(V / 32), H, entries).  RD: state rows per warp (and per thread).
template <typename T, int RD>
__global__ void __launch_bounds__(SW * 32) gla_scan_kernel(GlaParams<T> p) {
  extern __shared__ float sm[];
  pdl_grid_trigger();
  const int D = p.D, V = p.V, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  float* sq = sm;                          // [CT][D]
  float* sk = sq + CT * D;
  float* sg = sk + CT * D;
  float* sv = sg + CT * D;                 // [CT][32]
  float* red = sv + CT * 32;               // [CT][SW][32]
  const int h = blockIdx.y, e = blockIdx.z, c = blockIdx.x * 32 + lane;
  pdl_grid_wait();
  const int t0 = p.first[e], n = p.length[e];
  if (p.max_len && n > p.max_len) return;
  float* st = p.state + ((size_t)p.slot[e] * p.H + h) * D * V;
  const bool fresh = p.positions[t0] == 0;
  float s[RD];
#pragma unroll
  for (int i = 0; i < RD; ++i) {
    const int d = i * SW + warp;
    s[i] = !fresh && d < D && c < V ? st[(size_t)d * V + c] : 0.f;
  }
  for (int r0 = 0; r0 < n; r0 += CT) {
    const int m = min(CT, n - r0);
    __syncthreads();
    for (int i = tid; i < m * D; i += SW * 32) {
      const int r = i / D, d = i - r * D;
      const size_t row = (size_t)(t0 + r0 + r);
      sq[i] = (float)p.q[row * p.ld + h * D + d] * p.scale;
      sk[i] = (float)p.k[row * p.ld + h * D + d];
      sg[i] = expf(p.la[(row * p.H + h) * D + d]);
    }
    for (int i = tid; i < m * 32; i += SW * 32)
      sv[i] = blockIdx.x * 32 + (i & 31) < V ? (float)p.v[(size_t)(t0 + r0 + (i >> 5)) * p.ld + h * V + blockIdx.x * 32 + (i & 31)] : 0.f;
    __syncthreads();
    for (int r = 0; r < m; ++r) {
      const float v = sv[r * 32 + lane];
      float acc = 0.f;
#pragma unroll
      for (int i = 0; i < RD; ++i) {
        const int d = i * SW + warp;
        if (d < D) {
          s[i] = fmaf(sg[r * D + d], s[i], sk[r * D + d] * v);
          acc = fmaf(s[i], sq[r * D + d], acc);
        }
      }
      red[(r * SW + warp) * 32 + lane] = acc;
    }
    __syncthreads();
    for (int i = tid; i < m * 32; i += SW * 32) {
      const int r = i >> 5, col = blockIdx.x * 32 + (i & 31);
      float a = 0.f;
#pragma unroll
      for (int w = 0; w < SW; ++w) a += red[(r * SW + w) * 32 + (i & 31)];
      if (col < V) p.o[((size_t)(t0 + r0 + r) * p.H + h) * V + col] = a;
    }
  }
#pragma unroll
  for (int i = 0; i < RD; ++i) {
    const int d = i * SW + warp;
    if (d < D && c < V) st[(size_t)d * V + c] = s[i];
  }
}

template <typename T>
struct GlaStepParams {
  GlaParams<T> b;
  const T *a, *gate;         // decay latent and gate columns of the projection
  const T* w2;               // [H * D, rank]
  const float *bias, *norm_w;
  T* out;                    // [rows, ldo]
  int rank, vdim, ldo;
  float inv_tau, eps;
};

constexpr int STEP_THREADS = 256;

// grid (H, entries): one row per entry.  A thread owns four value columns and every (threads / (V / 4))-th channel.
template <typename T>
__global__ void __launch_bounds__(STEP_THREADS) gla_step_kernel(GlaStepParams<T> p) {
  extern __shared__ float sm[];
  __shared__ float red[32];
  pdl_grid_trigger();
  const int D = p.b.D, V = p.b.V, nq = V / 4, groups = STEP_THREADS / nq, tid = threadIdx.x;
  float* sq = sm;                          // [D] query, key, decay
  float* sk = sq + D;
  float* sg = sk + D;
  float* sa = sg + D;                      // [rank]
  float* so = sa + p.rank;                 // [groups][V]
  const int h = blockIdx.x, e = blockIdx.y;
  pdl_grid_wait();
  const size_t row = p.b.first[e];
  float* st = p.b.state + ((size_t)p.b.slot[e] * p.b.H + h) * D * V;
  const bool fresh = p.b.positions[row] == 0;
  for (int i = tid; i < p.rank; i += STEP_THREADS) sa[i] = (float)p.a[row * p.b.ld + i];
  for (int d = tid; d < D; d += STEP_THREADS) {
    sq[d] = (float)p.b.q[row * p.b.ld + h * D + d] * p.b.scale;
    sk[d] = (float)p.b.k[row * p.b.ld + h * D + d];
  }
  const int col = tid % nq, grp = tid / nq;
  const bool on = grp < groups;
  float v[4] = {0.f, 0.f, 0.f, 0.f};
  if (on)
#pragma unroll
    for (int j = 0; j < 4; ++j) v[j] = (float)p.b.v[row * p.b.ld + h * V + col * 4 + j];
  __syncthreads();
  for (int d = tid; d < D; d += STEP_THREADS) {
    float z = p.bias[h * D + d];
    for (int k = 0; k < p.rank; k += 8) {
      float w[8];
      load8(p.w2 + (size_t)(h * D + d) * p.rank + k, w);
#pragma unroll
      for (int j = 0; j < 8; ++j) z = fmaf(w[j], sa[k + j], z);
    }
    sg[d] = expf(log_sigmoid(z) * p.inv_tau);
  }
  __syncthreads();
  float acc[4] = {0.f, 0.f, 0.f, 0.f};
  if (on) {
    constexpr int U = 8;                   // channels in flight
    for (int d0 = grp; d0 < D; d0 += groups * U) {
      float4 s[U];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int d = d0 + u * groups;
        s[u] = !fresh && d < D ? *reinterpret_cast<const float4*>(st + (size_t)d * V + col * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int d = d0 + u * groups;
        if (d < D) {
          const float a = sg[d], k = sk[d], q = sq[d];
          s[u].x = fmaf(a, s[u].x, k * v[0]); s[u].y = fmaf(a, s[u].y, k * v[1]);
          s[u].z = fmaf(a, s[u].z, k * v[2]); s[u].w = fmaf(a, s[u].w, k * v[3]);
          acc[0] = fmaf(s[u].x, q, acc[0]); acc[1] = fmaf(s[u].y, q, acc[1]);
          acc[2] = fmaf(s[u].z, q, acc[2]); acc[3] = fmaf(s[u].w, q, acc[3]);
          *reinterpret_cast<float4*>(st + (size_t)d * V + col * 4) = s[u];
        }
      }
    }
    *reinterpret_cast<float4*>(so + grp * V + col * 4) = make_float4(acc[0], acc[1], acc[2], acc[3]);
  }
  __syncthreads();
  float o[4], ss = 0.f;                    // V <= 4 * STEP_THREADS
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int c = tid + j * STEP_THREADS;
    o[j] = 0.f;
    if (c < V)
      for (int w = 0; w < groups; ++w) o[j] += so[w * V + c];
    ss += o[j] * o[j];
  }
  const float inv = 1.f / sqrtf(block_sum_all(ss, red) / (float)p.vdim + p.eps);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int c = tid + j * STEP_THREADS;
    if (c < V) {
      const float g = (float)p.gate[row * p.b.ld + h * V + c];
      p.out[row * p.ldo + h * V + c] = (T)(o[j] * inv * p.norm_w[c] * (g / (1.f + expf(-g))));
    }
  }
  if (h == 0)
    for (int c = p.b.H * V + tid; c < p.ldo; c += STEP_THREADS) p.out[row * p.ldo + c] = (T)0.f;
}

__device__ __forceinline__ float silu_of(float z, __nv_bfloat16) { return __fdividef(z, 1.f + __expf(-z)); }
__device__ __forceinline__ float silu_of(float z, float) { return z / (1.f + expf(-z)); }

// LANES lanes per (row, head): out[row, h * V + c] = o / rms over the head's vdim values * weight * silu(gate).
template <typename T, int KEEP, int LANES>  // KEEP: rounds of 8 LANES columns held in registers
__global__ void gla_finish_kernel(const float* __restrict__ o, const T* __restrict__ gate, int ld_gate, const float* __restrict__ w,
                                  T* __restrict__ out, int ldo, int rows, int H, int V, int vdim, float eps) {
  pdl_grid_trigger();
  pdl_grid_wait();
  const int lane = threadIdx.x % LANES;
  const long long item = (long long)blockIdx.x * (blockDim.x / LANES) + threadIdx.x / LANES;
  const bool on = item < (long long)rows * H;               // the sums below are shuffles of whole warps
  const size_t row = on ? item / H : 0;
  const int h = on ? (int)(item - (long long)row * H) : 0;
  const float* src = o + (on ? item : 0) * V;
  const T* gsrc = gate + row * ld_gate + h * V;
  float f[KEEP][8], g[KEEP][8], ss = 0.f;
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int c = i * 8 * LANES + lane * 8;
    if (c < V) {
      load8(src + c, f[i]);
      load8(gsrc + c, g[i]);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += f[i][j] * f[i][j];               // padded columns are zero
    }
  }
  for (int c = KEEP * 8 * LANES + lane * 8; c < V; c += 8 * LANES) {
    float t[8];
    load8(src + c, t);
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += t[j] * t[j];
  }
#pragma unroll
  for (int x = LANES / 2; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);
  if (!on) return;
  const float inv = 1.f / sqrtf(ss / (float)vdim + eps);
  auto finish = [&](int c, float (&v)[8], const float (&gv)[8]) {
    float ww[8];
    load8(w + c, ww);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = v[j] * inv * ww[j] * silu_of(gv[j], T());
    store8(out + row * ldo + h * V + c, v);
  };
#pragma unroll
  for (int i = 0; i < KEEP; ++i)
    if (i * 8 * LANES + lane * 8 < V) finish(i * 8 * LANES + lane * 8, f[i], g[i]);
  for (int c = KEEP * 8 * LANES + lane * 8; c < V; c += 8 * LANES) {
    float v[8], gv[8];
    load8(src + c, v);
    load8(gsrc + c, gv);
    finish(c, v, gv);
  }
  if (h == H - 1)
    for (int c = H * V + lane; c < ldo; c += LANES) out[row * ldo + c] = (T)0.f;
}

template <typename T, int RD>
int launch_scan(const GlaParams<T>& p, int entries, cudaStream_t stream) {
  const size_t smem = (size_t)(3 * CT * p.D + CT * 32 + CT * SW * 32) * 4;
  static PerDeviceOnce once_;
  bool& configured = once_.slot();
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(gla_scan_kernel<T, RD>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  return (int)launch_pdl(gla_scan_kernel<T, RD>, dim3((p.V + 31) / 32, p.H, entries), dim3(SW * 32), smem, stream, p);
}

template <typename T>
int run_scan(const void* q, const void* k, const void* v, int ld, const float* la, float* state, float* o, const int* first,
             const int* length, const int* slot, const int* positions, int entries, int max_len, int H, int D, int V, float scale,
             cudaStream_t stream) {
  GlaParams<T> p;
  p.max_len = max_len;
  p.q = reinterpret_cast<const T*>(q); p.k = reinterpret_cast<const T*>(k); p.v = reinterpret_cast<const T*>(v); p.la = la;
  p.state = state; p.o = o; p.first = first; p.length = length; p.slot = slot; p.positions = positions; p.ld = ld; p.H = H; p.D = D;
  p.V = V; p.scale = scale;
  if (D <= 4 * SW) return launch_scan<T, 4>(p, entries, stream);
  if (D <= 8 * SW) return launch_scan<T, 8>(p, entries, stream);
  if (D <= 16 * SW) return launch_scan<T, 16>(p, entries, stream);
  if (D <= 32 * SW) return launch_scan<T, 32>(p, entries, stream);
  if (D <= 64 * SW) return launch_scan<T, 64>(p, entries, stream);
  return -6;
}

template <typename T>
int run_decay(const void* a, int ld, const void* w2, const float* bias, float inv_tau, float* la, int rows, int channels, int rank,
              cudaStream_t stream) {
  const int threads = channels >= 256 ? 256 : (channels + 31) / 32 * 32;
  int cols = (channels + threads - 1) / threads;
  const dim3 grid((rows + DR - 1) / DR, cols);
  return (int)launch_pdl(gla_decay_kernel<T>, grid, dim3(threads), (size_t)DR * rank * 4, stream, reinterpret_cast<const T*>(a), ld,
                         reinterpret_cast<const T*>(w2), bias, inv_tau, la, rows, channels, rank);
}

template <typename T>
int run_finish(const float* o, const void* gate, int ld_gate, const float* w, void* out, int ldo, int rows, int H, int V, int vdim,
               float eps, cudaStream_t stream) {
  const long long items = (long long)rows * H;
  const int lanes = V <= 64 ? 8 : V <= 128 ? 16 : 32, per = 256 / lanes;
  const dim3 grid((unsigned)((items + per - 1) / per)), block(256);
  auto gp = reinterpret_cast<const T*>(gate);
  auto op = reinterpret_cast<T*>(out);
  if (lanes == 8) return (int)launch_pdl(gla_finish_kernel<T, 1, 8>, grid, block, 0, stream, o, gp, ld_gate, w, op, ldo, rows, H, V, vdim, eps);
  if (lanes == 16) return (int)launch_pdl(gla_finish_kernel<T, 1, 16>, grid, block, 0, stream, o, gp, ld_gate, w, op, ldo, rows, H, V, vdim, eps);
  if (V <= 256) return (int)launch_pdl(gla_finish_kernel<T, 1, 32>, grid, block, 0, stream, o, gp, ld_gate, w, op, ldo, rows, H, V, vdim, eps);
  return (int)launch_pdl(gla_finish_kernel<T, 2, 32>, grid, block, 0, stream, o, gp, ld_gate, w, op, ldo, rows, H, V, vdim, eps);
}

template <typename T>
int run_step(const void* q, const void* k, const void* v, const void* gate, const void* a, int ld, const void* w2, const float* bias,
             float inv_tau, int rank, float* state, const int* first, const int* slot, const int* positions, int entries, int H, int D,
             int V, int vdim, float scale, const float* norm_w, float eps, void* out, int ldo, cudaStream_t stream) {
  GlaStepParams<T> p;
  p.b.q = reinterpret_cast<const T*>(q); p.b.k = reinterpret_cast<const T*>(k); p.b.v = reinterpret_cast<const T*>(v); p.b.la = nullptr;
  p.b.state = state; p.b.o = nullptr; p.b.first = first; p.b.length = nullptr; p.b.slot = slot; p.b.positions = positions; p.b.ld = ld;
  p.b.H = H; p.b.D = D; p.b.V = V; p.b.max_len = 0; p.b.scale = scale;
  p.a = reinterpret_cast<const T*>(a); p.gate = reinterpret_cast<const T*>(gate); p.w2 = reinterpret_cast<const T*>(w2); p.bias = bias;
  p.norm_w = norm_w; p.out = reinterpret_cast<T*>(out); p.rank = rank; p.vdim = vdim; p.ldo = ldo; p.inv_tau = inv_tau; p.eps = eps;
  const size_t smem = (size_t)(3 * D + rank + STEP_THREADS / (V / 4) * V) * 4;
  return (int)launch_pdl(gla_step_kernel<T>, dim3(H, entries), dim3(STEP_THREADS), smem, stream, p);
}

}  // namespace

// a rows `ld` apart, w2 [channels, rank] in the activations' type, la fp32 [rows, channels]; rank % 8 == 0, at most 1024.
extern "C" int b200_gla_decay(const void* a, int ld, const void* w2, const float* bias, float inv_tau, float* la, int rows,
                              int channels, int rank, int f32, cudaStream_t stream) {
  if (rows <= 0 || channels <= 0 || rank <= 0 || (rank & 7) || rank > 1024) return -6;
  return f32 ? run_decay<float>(a, ld, w2, bias, inv_tau, la, rows, channels, rank, stream)
             : run_decay<__nv_bfloat16>(a, ld, w2, bias, inv_tau, la, rows, channels, rank, stream);
}

// D at most 512; entries of at most max_len rows (0: all); state [slots, H, D, V] fp32 in place; o fp32 [rows, H * V].
extern "C" int b200_gla_scan(const void* q, const void* k, const void* v, int ld, const float* la, float* state, float* o,
                             const int* first, const int* length, const int* slot, const int* positions, int entries, int max_len,
                             int H, int D, int V, float scale, int f32, cudaStream_t stream) {
  if (entries <= 0 || entries > 65535 || H <= 0 || H > 65535 || D <= 0 || V <= 0) return -6;
  return f32 ? run_scan<float>(q, k, v, ld, la, state, o, first, length, slot, positions, entries, max_len, H, D, V, scale, stream)
             : run_scan<__nv_bfloat16>(q, k, v, ld, la, state, o, first, length, slot, positions, entries, max_len, H, D, V, scale, stream);
}

// V % 16 == 0; out [rows, ldo] (columns behind the heads are zeroed).
extern "C" int b200_gla_finish(const float* o, const void* gate, int ld_gate, const float* w, void* out, int ldo, int rows, int H,
                               int V, int vdim, float eps, int f32, cudaStream_t stream) {
  if (rows <= 0 || H <= 0 || V <= 0 || (V & 15) || vdim <= 0 || vdim > V || ldo < H * V || (ldo & 7) || (ld_gate & 7)) return -6;
  return f32 ? run_finish<float>(o, gate, ld_gate, w, out, ldo, rows, H, V, vdim, eps, stream)
             : run_finish<__nv_bfloat16>(o, gate, ld_gate, w, out, ldo, rows, H, V, vdim, eps, stream);
}

// One row per entry (row first[e]): decay, state update, norm and gate in one launch.  V % 16 == 0, at most 1024; D at most 2048.
extern "C" int b200_gla_step(const void* q, const void* k, const void* v, const void* gate, const void* a, int ld, const void* w2,
                             const float* bias, float inv_tau, int rank, float* state, const int* first, const int* slot,
                             const int* positions, int entries, int H, int D, int V, int vdim, float scale, const float* norm_w,
                             float eps, void* out, int ldo, int f32, cudaStream_t stream) {
  if (entries <= 0 || entries > 65535 || H <= 0 || D <= 0 || D > 2048 || V <= 0 || (V & 15) || V > 4 * STEP_THREADS || vdim <= 0 ||
      vdim > V || rank <= 0 || (rank & 7) || rank > 1024 || ldo < H * V)
    return -6;
  return f32 ? run_step<float>(q, k, v, gate, a, ld, w2, bias, inv_tau, rank, state, first, slot, positions, entries, H, D, V, vdim, scale,
                               norm_w, eps, out, ldo, stream)
             : run_step<__nv_bfloat16>(q, k, v, gate, a, ld, w2, bias, inv_tau, rank, state, first, slot, positions, entries, H, D, V,
                                       vdim, scale, norm_w, eps, out, ldo, stream);
}
