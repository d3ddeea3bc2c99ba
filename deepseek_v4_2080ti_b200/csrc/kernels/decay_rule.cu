// Linear recurrences with one decay per head and a state S [D, V] per head in fp32:
//
//   retention     S <- g S + k v^T                     o = S^T q          g fixed per head; q, k rotated
//   delta rule    S <- g S,  S <- S + k (beta (v - S^T k))^T,  o = S^T q    g = exp(-exp(A) softplus(a + b)), unit q, k
//
// over a batch of rows of several sequences (entries of neighbouring rows, one state slot each; a portion that begins at
// position 0 starts from zero).  Query / key head of head h: h / (H / G).  Head widths are padded with zero channels.
//
//   delta_prep      unit queries and keys, log decays and step sizes of every row, fp32
//   rotate_prep     rotated queries and keys of every row, fp32
//   decay_scan      one token after the other: eight lanes share a column of the state.  For fp32, and for bf16 portions too
//                   short for retention_chunk.cu and delta_chunk.cu
//   decay_step      one token of many sequences: a block per head and sequence reads, updates and writes the state once,
//                   with the row's preparation in front and norm and gate behind
// The norm and the gate of prepared rows are gla_finish (gated_linear.cu).
#include "launch.h"
#include "ops.h"
#include "per_device.h"
#include "rotary.cuh"
#include "vec8.cuh"

namespace {
using namespace b200;

__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float sigmoidf(float z) { return 1.f / (1.f + expf(-z)); }

constexpr float UNIT_EPS = 1e-6f;

template <typename T>
struct DeltaPrepParams {
  const T* qk;               // [rows, >= 2 G D]: queries, then keys
  const T *a, *b;            // [rows, H] columns of the projection
  const float *neg_a, *dt;   // [H] -exp(A), bias of the step
  float *q_out, *k_out;      // [rows, G, D]
  float *log_decay, *beta;   // [rows, H]
  int ld_qk, ld_ab, rows, H, G, D;
  float scale;               // of the unit queries
};

// A block per row; a group of `lanes` lanes per vector.
template <typename T>
__global__ void __launch_bounds__(256) delta_prep_kernel(DeltaPrepParams<T> p, int lanes) {
  pdl_grid_trigger();
  pdl_grid_wait();
  const size_t row = blockIdx.x;
  const int lane = threadIdx.x % lanes, groups = blockDim.x / lanes, n = 2 * p.G;
  for (int base = 0; base < n; base += groups) {            // whole warps take every pass
    const int v = base + threadIdx.x / lanes;
    const bool on = v < n;
    const T* src = p.qk + row * p.ld_qk + (size_t)v * p.D;
    float ss = 0.f;
    for (int d = lane * 8; on && d < p.D; d += lanes * 8) {
      float f[8];
      load8(src + d, f);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss = fmaf(f[j], f[j], ss);
    }
    for (int o = lanes / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (!on) continue;
    const float inv = (v < p.G ? p.scale : 1.f) / sqrtf(ss + UNIT_EPS);
    float* dst = (v < p.G ? p.q_out + (row * p.G + v) * p.D : p.k_out + (row * p.G + v - p.G) * p.D);
    for (int d = lane * 8; d < p.D; d += lanes * 8) {
      float f[8];
      load8(src + d, f);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] *= inv;
      store8(dst + d, f);
    }
  }
  for (int h = threadIdx.x; h < p.H; h += blockDim.x) {
    p.log_decay[row * p.H + h] = p.neg_a[h] * softplus((float)p.a[row * p.ld_ab + h] + p.dt[h]);
    p.beta[row * p.H + h] = sigmoidf((float)p.b[row * p.ld_ab + h]);
  }
}

// A block per row.  Pairs (i, i + rot / 2) of every query and key vector are rotated, the rest passes; keys are scaled.  A thread
// takes eight neighbouring channels (and their partners where those are eight neighbours as well).
template <typename T>
__global__ void __launch_bounds__(256) rotate_prep_kernel(const T* __restrict__ q, const T* __restrict__ k, int ld,
                                                          const int* __restrict__ positions, const double* __restrict__ freq, int rot,
                                                          float k_scale, float* __restrict__ q_out, float* __restrict__ k_out, int H,
                                                          int D) {
  extern __shared__ float2 cs[];              // [rot / 2]
  pdl_grid_trigger();
  const int half = rot / 2, n = H * D;
  pdl_grid_wait();
  const size_t row = blockIdx.x;
  const int pos = positions[row];
  for (int i = threadIdx.x; i < half; i += blockDim.x) rotary_angle(pos, freq[i], 1.f, cs[i].x, cs[i].y);
  __syncthreads();
  const bool vectors = half % 8 == 0;
  for (int i = threadIdx.x * 8; i < 2 * n; i += blockDim.x * 8) {
    const bool is_k = i >= n;
    const int c = is_k ? i - n : i, d = c % D;
    const T* src = (is_k ? k : q) + row * ld + c;
    float f[8];
    load8(src, f);
    if (vectors) {
      if (d < rot) {
        const bool low = d < half;
        float o[8];
        load8(src + (low ? half : -half), o);
        const float2* a = cs + (low ? d : d - half);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] = f[j] * a[j].x + (low ? -o[j] : o[j]) * a[j].y;
      }
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        if (d + j < half) f[j] = f[j] * cs[d + j].x - (float)src[j + half] * cs[d + j].y;
        else if (d + j < rot) f[j] = f[j] * cs[d + j - half].x + (float)src[j - half] * cs[d + j - half].y;
      }
    }
    const float s = is_k ? k_scale : 1.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) f[j] *= s;
    store8((is_k ? k_out : q_out) + row * n + c, f);
  }
}

template <typename T>
struct DecayScanParams {
  const float *q, *k;        // [rows, G, D] prepared
  const T* v;                // head h of row t at v + t * ldv + h * V
  const float* log_decay;    // [rows, H], or null: `decay`
  const float* decay;        // [H] fixed factors
  const float* beta;         // [rows, H] (delta rule)
  float* state;              // [slots, H, D, V]
  float* o;                  // [rows, H * V]
  const int *first, *length, *slot, *positions;
  int ldv, H, G, D, V;
  int max_len;               // longer entries are left alone (0: none)
};

constexpr int CT = 16;          // rows staged together
constexpr int SW = 8;           // warps; a warp owns four columns

// grid (ceil(V / 32), H, entries).  RD: state values per lane; lane 8 c + s holds channels s, s + 8, ... of column c.
template <typename T, int RD, bool DELTA>
__global__ void __launch_bounds__(SW * 32) decay_scan_kernel(DecayScanParams<T> p) {
  extern __shared__ float sm[];
  pdl_grid_trigger();
  const int D = p.D, V = p.V, tid = threadIdx.x, sub = tid & 7, lc = tid >> 3;       // lc: column of the block
  float* sq = sm;                          // [CT][D]
  float* sk = sq + CT * D;
  float* sv = sk + CT * D;                 // [CT][32]
  float* sg = sv + CT * 32;                // [CT] decay, [CT] step size
  float* sb = sg + CT;
  const int h = blockIdx.y, e = blockIdx.z, c = blockIdx.x * 32 + lc, g = h / (p.H / p.G);
  pdl_grid_wait();
  const int t0 = p.first[e], n = p.length[e];
  if (p.max_len && n > p.max_len) return;
  float* st = p.state + ((size_t)p.slot[e] * p.H + h) * D * V;
  const bool fresh = p.positions[t0] == 0, on = c < V;
  float s[RD];
#pragma unroll
  for (int i = 0; i < RD; ++i) {
    const int d = i * 8 + sub;
    s[i] = !fresh && d < D && on ? st[(size_t)d * V + c] : 0.f;
  }
  for (int r0 = 0; r0 < n; r0 += CT) {
    const int m = min(CT, n - r0);
    __syncthreads();
    for (int i = tid; i < m * D; i += SW * 32) {
      const int r = i / D;
      const size_t at = ((size_t)(t0 + r0 + r) * p.G + g) * D + i - r * D;
      sq[i] = p.q[at];
      sk[i] = p.k[at];
    }
    for (int i = tid; i < m * 32; i += SW * 32)
      sv[i] = blockIdx.x * 32 + (i & 31) < V ? (float)p.v[(size_t)(t0 + r0 + (i >> 5)) * p.ldv + h * V + blockIdx.x * 32 + (i & 31)] : 0.f;
    if (tid < m) {
      const size_t at = (size_t)(t0 + r0 + tid) * p.H + h;
      sg[tid] = p.log_decay ? expf(p.log_decay[at]) : p.decay[h];
      if (DELTA) sb[tid] = p.beta[at];
    }
    __syncthreads();
    for (int r = 0; r < m; ++r) {
      const float gr = sg[r];
      float u = sv[r * 32 + lc];
      const float *kr = sk + r * D, *qr = sq + r * D;
      if (DELTA) {
        float dot = 0.f;
#pragma unroll
        for (int i = 0; i < RD; ++i) {
          const int d = i * 8 + sub;
          s[i] *= gr;
          if (d < D) dot = fmaf(s[i], kr[d], dot);
        }
        dot += __shfl_xor_sync(0xffffffffu, dot, 1);
        dot += __shfl_xor_sync(0xffffffffu, dot, 2);
        dot += __shfl_xor_sync(0xffffffffu, dot, 4);
        u = sb[r] * (u - dot);
      }
      float acc = 0.f;
#pragma unroll
      for (int i = 0; i < RD; ++i) {
        const int d = i * 8 + sub;
        if (d < D) {
          s[i] = fmaf(kr[d], u, DELTA ? s[i] : s[i] * gr);
          acc = fmaf(s[i], qr[d], acc);
        }
      }
      acc += __shfl_xor_sync(0xffffffffu, acc, 1);
      acc += __shfl_xor_sync(0xffffffffu, acc, 2);
      acc += __shfl_xor_sync(0xffffffffu, acc, 4);
      if (sub == 0 && on) p.o[((size_t)(t0 + r0 + r) * p.H + h) * V + c] = acc;
    }
  }
#pragma unroll
  for (int i = 0; i < RD; ++i) {
    const int d = i * 8 + sub;
    if (d < D && on) st[(size_t)d * V + c] = s[i];
  }
}

template <typename T>
struct DecayStepParams {
  const T *q, *k, *v, *gate; // head h (query / key head g) at ptr + row * ld + h V (g D); the gate in rows of ldg
  const T *a, *b;            // [rows, H] columns in rows of ldg (delta rule)
  const float *neg_a, *dt;   // [H]
  const float* decay;        // [H] (retention)
  const double* freq;        // [rot / 2]
  const float* norm_w;       // [V]
  float* state;              // [slots, H, D, V]
  T* out;                    // [rows, ldo]
  const int *first, *slot, *positions;
  int ld, ldg, H, G, D, V, vdim, rot, ldo;
  float scale, eps;
};

constexpr int KEEP_ROWS = 16;   // state rows of a thread that stay in registers

// grid (H, entries): one row per entry.  A thread owns four value columns and every (threads / (V / 4))-th channel.
template <typename T, bool DELTA>
__global__ void __launch_bounds__(512) decay_step_kernel(DecayStepParams<T> p) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[32];
  pdl_grid_trigger();
  const int D = p.D, V = p.V, nq = V / 4, nt = blockDim.x, groups = nt / nq, tid = threadIdx.x;
  float* sq = sm;                          // [D]
  float* sk = sq + D;
  float2* cs = reinterpret_cast<float2*>(sk + D);      // [rot / 2]
  float* so = sk + D + (DELTA ? 0 : (p.rot + 3) / 4 * 4);      // [groups][V]
  const int h = blockIdx.x, e = blockIdx.y, g = h / (p.H / p.G);
  pdl_grid_wait();
  const size_t row = p.first[e];
  float* st = p.state + ((size_t)p.slot[e] * p.H + h) * D * V;
  const int pos = p.positions[row];
  const int col = tid % nq, grp = tid / nq;
  const bool on = grp < groups, fresh = pos == 0, kept = groups * KEEP_ROWS >= D;
  float4 s[KEEP_ROWS];
  if (kept)
#pragma unroll
    for (int i = 0; i < KEEP_ROWS; ++i) {
      const int d = grp + i * groups;
      s[i] = on && !fresh && d < D ? *reinterpret_cast<const float4*>(st + (size_t)d * V + col * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  const T *qr = p.q + row * p.ld + (size_t)g * D, *kr = p.k + row * p.ld + (size_t)g * D;
  float decay, beta = 1.f;
  if (DELTA) {
    float qs = 0.f, ks = 0.f;
    for (int d = tid; d < D; d += nt) {
      sq[d] = (float)qr[d];
      sk[d] = (float)kr[d];
      qs = fmaf(sq[d], sq[d], qs);
      ks = fmaf(sk[d], sk[d], ks);
    }
    const float qn = p.scale / sqrtf(block_sum_all(qs, red) + UNIT_EPS), kn = 1.f / sqrtf(block_sum_all(ks, red) + UNIT_EPS);
    for (int d = tid; d < D; d += nt) {
      sq[d] *= qn;
      sk[d] *= kn;
    }
    decay = expf(p.neg_a[h] * softplus((float)p.a[row * p.ldg + h] + p.dt[h]));
    beta = sigmoidf((float)p.b[row * p.ldg + h]);
  } else {
    const int half = p.rot / 2;
    for (int i = tid; i < half; i += nt) rotary_angle(pos, p.freq[i], 1.f, cs[i].x, cs[i].y);
    __syncthreads();
    for (int d = tid; d < D; d += nt) {
      float q = (float)qr[d], k = (float)kr[d];
      if (d < half) {
        q = q * cs[d].x - (float)qr[d + half] * cs[d].y;
        k = k * cs[d].x - (float)kr[d + half] * cs[d].y;
      } else if (d < p.rot) {
        q = q * cs[d - half].x + (float)qr[d - half] * cs[d - half].y;
        k = k * cs[d - half].x + (float)kr[d - half] * cs[d - half].y;
      }
      sq[d] = q;
      sk[d] = k * p.scale;
    }
    decay = p.decay[h];
  }
  float u[4] = {0.f, 0.f, 0.f, 0.f};
  if (on)
#pragma unroll
    for (int j = 0; j < 4; ++j) u[j] = (float)p.v[row * p.ld + (size_t)h * V + col * 4 + j];
  __syncthreads();
  auto load = [&](int d) {
    return fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(st + (size_t)d * V + col * 4);
  };
  if (DELTA) {
    float4 dot = make_float4(0.f, 0.f, 0.f, 0.f);
    if (on) {
      if (kept) {
#pragma unroll
        for (int i = 0; i < KEEP_ROWS; ++i) {
          const int d = grp + i * groups;
          const float k = d < D ? sk[d] : 0.f;
          s[i].x *= decay; s[i].y *= decay; s[i].z *= decay; s[i].w *= decay;
          dot.x = fmaf(s[i].x, k, dot.x); dot.y = fmaf(s[i].y, k, dot.y);
          dot.z = fmaf(s[i].z, k, dot.z); dot.w = fmaf(s[i].w, k, dot.w);
        }
      } else {
        for (int d = grp; d < D; d += groups) {
          const float4 w = load(d);
          const float k = sk[d] * decay;
          dot.x = fmaf(w.x, k, dot.x); dot.y = fmaf(w.y, k, dot.y); dot.z = fmaf(w.z, k, dot.z); dot.w = fmaf(w.w, k, dot.w);
        }
      }
      *reinterpret_cast<float4*>(so + grp * V + col * 4) = dot;
    }
    __syncthreads();
    if (on) {
      dot = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int w = 0; w < groups; ++w) {
        const float4 f = *reinterpret_cast<const float4*>(so + w * V + col * 4);
        dot.x += f.x; dot.y += f.y; dot.z += f.z; dot.w += f.w;
      }
      u[0] = beta * (u[0] - dot.x); u[1] = beta * (u[1] - dot.y); u[2] = beta * (u[2] - dot.z); u[3] = beta * (u[3] - dot.w);
    }
    __syncthreads();
  }
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
  auto update = [&](float4& w, int d, float f) {
    const float k = sk[d], q = sq[d];
    w.x = fmaf(f, w.x, k * u[0]); w.y = fmaf(f, w.y, k * u[1]); w.z = fmaf(f, w.z, k * u[2]); w.w = fmaf(f, w.w, k * u[3]);
    acc.x = fmaf(w.x, q, acc.x); acc.y = fmaf(w.y, q, acc.y); acc.z = fmaf(w.z, q, acc.z); acc.w = fmaf(w.w, q, acc.w);
    *reinterpret_cast<float4*>(st + (size_t)d * V + col * 4) = w;
  };
  if (on) {
    if (kept) {
#pragma unroll
      for (int i = 0; i < KEEP_ROWS; ++i) {
        const int d = grp + i * groups;
        if (d < D) update(s[i], d, DELTA ? 1.f : decay);
      }
    } else {
      for (int d = grp; d < D; d += groups) {
        float4 w = load(d);
        update(w, d, decay);
      }
    }
    *reinterpret_cast<float4*>(so + grp * V + col * 4) = acc;
  }
  __syncthreads();
  constexpr int OV = 4;                    // columns of a thread: V <= OV * threads
  float o[OV], ss = 0.f;
#pragma unroll
  for (int j = 0; j < OV; ++j) {
    const int c = tid + j * nt;
    o[j] = 0.f;
    if (c < V)
      for (int w = 0; w < groups; ++w) o[j] += so[w * V + c];
    ss = fmaf(o[j], o[j], ss);
  }
  const float inv = 1.f / sqrtf(block_sum_all(ss, red) / (float)p.vdim + p.eps);
#pragma unroll
  for (int j = 0; j < OV; ++j) {
    const int c = tid + j * nt;
    if (c < V) {
      const float z = (float)p.gate[row * p.ldg + (size_t)h * V + c];
      p.out[row * p.ldo + (size_t)h * V + c] = (T)(o[j] * inv * p.norm_w[c] * (z * sigmoidf(z)));
    }
  }
  if (h == 0)
    for (int c = p.H * V + tid; c < p.ldo; c += nt) p.out[row * p.ldo + c] = (T)0.f;
}

template <typename T, int RD, bool DELTA>
int launch_scan(const DecayScanParams<T>& p, int entries, cudaStream_t stream) {
  const size_t smem = (size_t)(2 * CT * p.D + CT * 32 + 2 * CT) * 4;
  static PerDeviceOnce once_;
  bool& configured = once_.slot();
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(decay_scan_kernel<T, RD, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  return (int)launch_pdl(decay_scan_kernel<T, RD, DELTA>, dim3((p.V + 31) / 32, p.H, entries), dim3(SW * 32), smem, stream, p);
}

template <typename T, bool DELTA>
int pick_scan(const DecayScanParams<T>& p, int entries, cudaStream_t stream) {
  if (p.D <= 32) return launch_scan<T, 4, DELTA>(p, entries, stream);
  if (p.D <= 64) return launch_scan<T, 8, DELTA>(p, entries, stream);
  if (p.D <= 128) return launch_scan<T, 16, DELTA>(p, entries, stream);
  if (p.D <= 256) return launch_scan<T, 32, DELTA>(p, entries, stream);
  if (p.D <= 512) return launch_scan<T, 64, DELTA>(p, entries, stream);
  return -6;
}

template <typename T>
int run_scan(const float* q, const float* k, const void* v, int ldv, const float* log_decay, const float* decay, const float* beta,
             float* state, float* o, const int* first, const int* length, const int* slot, const int* positions, int entries, int max_len,
             int H, int G, int D, int V, cudaStream_t stream) {
  DecayScanParams<T> p;
  p.q = q; p.k = k; p.v = reinterpret_cast<const T*>(v); p.log_decay = log_decay; p.decay = decay; p.beta = beta; p.state = state; p.o = o;
  p.first = first; p.length = length; p.slot = slot; p.positions = positions; p.ldv = ldv; p.H = H; p.G = G; p.D = D; p.V = V;
  p.max_len = max_len;
  return beta ? pick_scan<T, true>(p, entries, stream) : pick_scan<T, false>(p, entries, stream);
}

template <typename T>
int run_delta_prep(const void* qk, int ld_qk, const void* a, const void* b, int ld_ab, const float* neg_a, const float* dt, float* q_out,
                   float* k_out, float* log_decay, float* beta, int rows, int H, int G, int D, float scale, cudaStream_t stream) {
  DeltaPrepParams<T> p;
  p.qk = reinterpret_cast<const T*>(qk); p.a = reinterpret_cast<const T*>(a); p.b = reinterpret_cast<const T*>(b); p.neg_a = neg_a;
  p.dt = dt; p.q_out = q_out; p.k_out = k_out; p.log_decay = log_decay; p.beta = beta; p.ld_qk = ld_qk; p.ld_ab = ld_ab; p.rows = rows;
  p.H = H; p.G = G; p.D = D; p.scale = scale;
  int lanes = 1;
  while (lanes < 32 && lanes * 8 < D) lanes *= 2;
  int threads = 64;
  while (threads < 256 && threads < 2 * G * lanes) threads *= 2;
  return (int)launch_pdl(delta_prep_kernel<T>, dim3(rows), dim3(threads), 0, stream, p, lanes);
}

// Threads of a step: every channel of four columns in registers where that is possible.
int step_threads(int D, int V) {
  int nt = 128;
  while (nt < 512 && (nt / (V / 4) * KEEP_ROWS < D || nt * 4 < V)) nt *= 2;
  return nt;
}

template <typename T, bool DELTA>
int launch_step(const DecayStepParams<T>& p, int entries, cudaStream_t stream) {
  const int nt = step_threads(p.D, p.V);
  const size_t smem = (size_t)(2 * p.D + (DELTA ? 0 : (p.rot + 3) / 4 * 4) + nt / (p.V / 4) * p.V) * 4;
  return (int)launch_pdl(decay_step_kernel<T, DELTA>, dim3(p.H, entries), dim3(nt), smem, stream, p);
}

template <typename T>
int run_step(const void* q, const void* k, const void* v, int ld, const void* gate, const void* a, const void* b, int ldg,
             const float* neg_a, const float* dt, const float* decay, const double* freq, int rot, float* state, const int* first,
             const int* slot, const int* positions, int entries, int H, int G, int D, int V, int vdim, float scale, const float* norm_w,
             float eps, void* out, int ldo, cudaStream_t stream) {
  DecayStepParams<T> p;
  p.q = reinterpret_cast<const T*>(q); p.k = reinterpret_cast<const T*>(k); p.v = reinterpret_cast<const T*>(v);
  p.gate = reinterpret_cast<const T*>(gate); p.a = reinterpret_cast<const T*>(a); p.b = reinterpret_cast<const T*>(b); p.neg_a = neg_a;
  p.dt = dt; p.decay = decay; p.freq = freq; p.norm_w = norm_w; p.state = state; p.out = reinterpret_cast<T*>(out); p.first = first;
  p.slot = slot; p.positions = positions; p.ld = ld; p.ldg = ldg; p.H = H; p.G = G; p.D = D; p.V = V; p.vdim = vdim; p.rot = rot;
  p.ldo = ldo; p.scale = scale; p.eps = eps;
  return decay ? launch_step<T, false>(p, entries, stream) : launch_step<T, true>(p, entries, stream);
}

}  // namespace

// qk rows of [queries | keys], G heads of D channels each; a, b: H columns in rows `ld_ab` apart.  D a multiple of 8.
extern "C" int b200_delta_prep(const void* qk, int ld_qk, const void* a, const void* b, int ld_ab, const float* neg_a, const float* dt,
                               float* q_out, float* k_out, float* log_decay, float* beta, int rows, int H, int G, int D, float scale,
                               int f32, cudaStream_t stream) {
  if (rows <= 0 || H <= 0 || G <= 0 || H % G || D <= 0 || (D & 7) || (ld_qk & 7) || ld_qk < 2 * G * D) return -6;
  return f32 ? run_delta_prep<float>(qk, ld_qk, a, b, ld_ab, neg_a, dt, q_out, k_out, log_decay, beta, rows, H, G, D, scale, stream)
             : run_delta_prep<__nv_bfloat16>(qk, ld_qk, a, b, ld_ab, neg_a, dt, q_out, k_out, log_decay, beta, rows, H, G, D, scale, stream);
}

// q, k: H heads of D channels in rows `ld` apart, the first `rot` (even) rotated in pairs (i, i + rot / 2); fp32 out [rows, H, D].
extern "C" int b200_rotate_prep(const void* q, const void* k, int ld, const int* positions, const double* freq, int rot, float k_scale,
                                float* q_out, float* k_out, int rows, int H, int D, int f32, cudaStream_t stream) {
  if (rows <= 0 || H <= 0 || D <= 0 || (D & 7) || (ld & 7) || rot < 0 || (rot & 1) || rot > D || rot > 4096 || ld < H * D) return -6;
  const size_t smem = (size_t)(rot / 2) * 8;
  if (f32)
    return (int)launch_pdl(rotate_prep_kernel<float>, dim3(rows), dim3(256), smem, stream, reinterpret_cast<const float*>(q),
                           reinterpret_cast<const float*>(k), ld, positions, freq, rot, k_scale, q_out, k_out, H, D);
  return (int)launch_pdl(rotate_prep_kernel<__nv_bfloat16>, dim3(rows), dim3(256), smem, stream, reinterpret_cast<const __nv_bfloat16*>(q),
                         reinterpret_cast<const __nv_bfloat16*>(k), ld, positions, freq, rot, k_scale, q_out, k_out, H, D);
}

// q, k fp32 [rows, G, D] (b200_delta_prep, b200_rotate_prep); log_decay [rows, H] or decay [H]; beta: the delta rule.  D at most
// 512; entries of at most max_len rows (0: all); state [slots, H, D, V] fp32 in place; o fp32 [rows, H * V].
extern "C" int b200_decay_scan(const float* q, const float* k, const void* v, int ldv, const float* log_decay, const float* decay,
                               const float* beta, float* state, float* o, const int* first, const int* length, const int* slot,
                               const int* positions, int entries, int max_len, int H, int G, int D, int V, int f32, cudaStream_t stream) {
  if (entries <= 0 || entries > 65535 || H <= 0 || H > 65535 || G <= 0 || H % G || D <= 0 || V <= 0 || ldv < H * V || (!log_decay && !decay))
    return -6;
  return f32 ? run_scan<float>(q, k, v, ldv, log_decay, decay, beta, state, o, first, length, slot, positions, entries, max_len, H, G, D, V, stream)
             : run_scan<__nv_bfloat16>(q, k, v, ldv, log_decay, decay, beta, state, o, first, length, slot, positions, entries, max_len, H,
                                       G, D, V, stream);
}

// One row per entry (row first[e]).  `decay` given: retention (q, k rotated by `freq`, keys scaled); else the delta rule with
// a, b, neg_a, dt (unit q, k, queries scaled).  V % 16 == 0, at most 2048, as D; out [rows, ldo], zero behind the heads.
extern "C" int b200_decay_step(const void* q, const void* k, const void* v, int ld, const void* gate, const void* a, const void* b, int ldg,
                               const float* neg_a, const float* dt, const float* decay, const double* freq, int rot, float* state,
                               const int* first, const int* slot, const int* positions, int entries, int H, int G, int D, int V, int vdim,
                               float scale, const float* norm_w, float eps, void* out, int ldo, int f32, cudaStream_t stream) {
  if (entries <= 0 || entries > 65535 || H <= 0 || G <= 0 || H % G || D <= 0 || D > 2048 || V <= 0 || (V & 15) || V > 2048 || vdim <= 0 ||
      vdim > V || ldo < H * V || rot < 0 || (rot & 1) || rot > D || (!decay && (!a || !b || !neg_a || !dt)) || (decay && rot && !freq))
    return -6;
  return f32 ? run_step<float>(q, k, v, ld, gate, a, b, ldg, neg_a, dt, decay, freq, rot, state, first, slot, positions, entries, H, G, D, V,
                               vdim, scale, norm_w, eps, out, ldo, stream)
             : run_step<__nv_bfloat16>(q, k, v, ld, gate, a, b, ldg, neg_a, dt, decay, freq, rot, state, first, slot, positions, entries, H,
                                       G, D, V, vdim, scale, norm_w, eps, out, ldo, stream);
}
