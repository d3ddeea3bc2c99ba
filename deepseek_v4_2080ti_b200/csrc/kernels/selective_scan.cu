// Selective scan (diagonal state-space recurrence with input-dependent step sizes) over a batch of rows that belong to
// several sequences:
//
//   delta = softplus(dt + bias)          per row and channel
//   S[n]  = exp(delta A[n]) S[n] + delta x B[n],   y = sum_n S[n] C[n] + D x,   out = y silu(z)
//
// Everything in the recurrence is fp32; x, B, C, z and out are bf16 or fp32, dt is the fp32 output of its projection.
// The state lives in a slot per sequence and starts at zero when the sequence's first row of the batch has position 0.
//
// L lanes share a channel, NS states each; a block owns 128 / L channels of one sequence (or of one time slice of it) and
// walks tiles of 32 rows: step sizes and inputs are converted once per (row, channel) into shared memory, the recurrence
// runs out of it with the states in registers, and four steps' partial sums are reduced over the lanes together
// (transposing butterfly).  The next tile's rows are in flight meanwhile.  Sequences that bring a single row (decoding) take
// a kernel of their own without the tiles.
//
// A long sequence with few channels does not fill the device: its rows are then cut into slices.  A first pass runs every
// slice but the last from a zero state (the first one from the slot's state) and keeps the end state and the sum of the
// step sizes; since the decay over a slice is exp(A sum delta), the second pass composes the state at its own start from
// those and produces the outputs.
//
// The last slice also replaces the slot's convolution tail (the inputs of the convolution in front, see conv_rows.cu).
#include "launch.h"
#include "ops.h"
#include "per_device.h"
#include "vec8.cuh"

namespace {
using namespace b200;

constexpr int THREADS = 128;
constexpr int TT = 32;                   // rows per tile

template <typename T>
struct ScanParams {
  const T* x;                // [rows, ldx] convolution output
  const float* dt;           // [rows, ldd]
  const T* bc;               // [rows, ldb]: B at b_off, C at c_off
  const T* z;                // [rows, ldz]
  T* out;                    // [rows, ldo]
  const float *a, *dt_bias, *d_skip;   // [C, N] (times log2(e) for bf16 data), [C], [C]
  float* state;              // [slots, C, N]
  const int *ent_first, *ent_len, *ent_slot, *positions;
  const T* xin;              // [rows, ldin] inputs of the convolution (null: no tail to keep)
  T* tail;                   // [slots, taps - 1, C]
  float* ws_state;           // [entries, slices, C, N]: end state per slice; the last entry holds the initial state
  float* ws_sum;             // [entries, slices, C]
  int ldx, ldd, ldb, b_off, c_off, ldz, ldo, ldin, taps, C, N, slices, per;
};

template <bool FAST>
__device__ __forceinline__ float decay(float v) {
  if (!FAST) return expf(v);
  float e;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(v));
  return e;
}
// log(1 + exp(v)); the fast form sums the series of log(1 + e) where 1 + e would lose e's digits
template <bool FAST>
__device__ __forceinline__ float softplus(float v) {
  if (!FAST) return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v)));
  const float e = __expf(-fabsf(v));
  const float series = e * fmaf(e, fmaf(e, fmaf(e, fmaf(e, 0.2f, -0.25f), 1.f / 3.f), -0.5f), 1.f);
  return fmaxf(v, 0.f) + (e < 0.0625f ? series : __logf(1.f + e));
}

__device__ __forceinline__ void load4(const __nv_bfloat16* p, float (&f)[4]) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
}
__device__ __forceinline__ void load4(const float* p, float (&f)[4]) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
}
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float (&f)[4]) {
  uint2 u;
  *reinterpret_cast<__nv_bfloat162*>(&u.x) = __floats2bfloat162_rn(f[0], f[1]);
  *reinterpret_cast<__nv_bfloat162*>(&u.y) = __floats2bfloat162_rn(f[2], f[3]);
  *reinterpret_cast<uint2*>(p) = u;
}
__device__ __forceinline__ void store4(float* p, const float (&f)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
}
template <bool FAST>
__device__ __forceinline__ float silu(float z) {
  return FAST ? __fdividef(z, 1.f + __expf(-z)) : z / (1.f + expf(-z));
}

// The slot's convolution tail of channel c after `len` rows: ascending, an old entry moves down before it is overwritten.
template <typename T>
__device__ __forceinline__ void replace_tail(const ScanParams<T>& p, int slot, int first, int len, int c) {
  const int keep = p.taps - 1;
  T* tl = p.tail + (size_t)slot * keep * p.C + c;
  for (int i = 0; i < keep; ++i) {
    const int r = len - keep + i;
    tl[(size_t)i * p.C] = r >= 0 ? p.xin[(size_t)(first + r) * p.ldin + c] : tl[(size_t)(len + i) * p.C];
  }
}

template <int NS>
__device__ __forceinline__ void load_ns(const float* p, float (&f)[NS]) {
  if constexpr (NS % 4 == 0) {
#pragma unroll
    for (int i = 0; i < NS; i += 4) *reinterpret_cast<float4*>(f + i) = *reinterpret_cast<const float4*>(p + i);
  } else if constexpr (NS % 2 == 0) {
#pragma unroll
    for (int i = 0; i < NS; i += 2) *reinterpret_cast<float2*>(f + i) = *reinterpret_cast<const float2*>(p + i);
  } else {
#pragma unroll
    for (int i = 0; i < NS; ++i) f[i] = p[i];
  }
}

// PASS 0: the whole sequence or (slices > 1) the outputs of one slice; PASS 1: end state of one slice.
template <typename T, int L, int NS, int PASS>
__global__ void __launch_bounds__(THREADS) scan_kernel(ScanParams<T> p) {
  constexpr bool FAST = sizeof(T) == 2;
  constexpr int CB = THREADS / L, NP = L * NS;
  constexpr int CV = CB / 4, UNITS = TT * CV, U = (UNITS + THREADS - 1) / THREADS, UR = THREADS / CV;   // units of 4 channels
  extern __shared__ __align__(16) float sm[];
  float2* sdt = reinterpret_cast<float2*>(sm);              // [TT][CB]: (delta, delta x)
  float* sy = sm + TT * CB * 2;                             // [TT][CB]
  float* sbc = sy + TT * CB;                                // [TT][2][NP]
  pdl_grid_trigger();
  const int tid = threadIdx.x, ch = tid / L, lane = tid % L, c0 = blockIdx.x * CB, c = c0 + ch;
  const bool on = c < p.C;
  float a[NS];
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    const int n = lane * NS + i;
    a[i] = on && n < p.N ? p.a[(size_t)c * p.N + n] : 0.f;
  }
  for (int i = tid; i < TT * 2 * NP; i += THREADS) sbc[i] = 0.f;        // states past N stay zero
  // this thread's units of a tile: rows vt, vt + UR, .., channels vc..vc+3
  const int vt = tid / CV, vl = (tid % CV) * 4, vc = c0 + vl;
  const bool v_on = vc < p.C;
  float bias4[4] = {}, d4[4] = {};
  if (v_on) {
    load4(p.dt_bias + vc, bias4);
    load4(p.d_skip + vc, d4);
  }
  pdl_grid_wait();
  const int e = blockIdx.z, slice = blockIdx.y;
  const int len = p.ent_len[e], lo = slice * p.per, hi = min(len, lo + p.per);
  const bool single = len <= p.per;
  if (len == 1 || lo >= len || (PASS == 1 && (single || hi == len))) return;      // uniform per block
  const int first = p.ent_first[e], slot = p.ent_slot[e], pos = p.positions[first];
  const size_t cn = (size_t)p.C * p.N;
  float* st = p.state + (size_t)slot * cn + (size_t)c * p.N;
  float* ws = p.ws_state ? p.ws_state + (size_t)e * p.slices * cn + (size_t)c * p.N : nullptr;

  float s[NS];
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    const int n = lane * NS + i;
    s[i] = 0.f;
    if (on && n < p.N) {
      if (slice == 0) {
        if (PASS == 1 || single) s[i] = pos == 0 ? 0.f : st[n];
        else s[i] = ws[(size_t)(p.slices - 1) * cn + n];
        if (PASS == 1) ws[(size_t)(p.slices - 1) * cn + n] = s[i];
      } else if (PASS == 0) {
        s[i] = ws[n];
        for (int k = 1; k < slice; ++k)
          s[i] = decay<FAST>(p.ws_sum[((size_t)e * p.slices + k) * p.C + c] * a[i]) * s[i] + ws[k * cn + n];
      }
    }
  }

  const int nb8 = (p.c_off - p.b_off) / 8, nbc = 2 * nb8;               // vectors of B (and of C) per row
  float x4[U][4], dt4[U][4], z4[U][4], bc8[8];
  auto fetch_bc = [&](int i, int row0, float (&f)[8]) {
    const int t = i / nbc, v = i % nbc;
    if (row0 + t < hi) load8(p.bc + (size_t)(first + row0 + t) * p.ldb + p.b_off + v * 8, f);
    else {
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] = 0.f;
    }
  };
  auto put_bc = [&](int i, const float (&f)[8]) {
    const int t = i / nbc, v = i % nbc, half = v / nb8, n0 = (v % nb8) * 8;
    float* dst = sbc + (t * 2 + half) * NP + n0;
    if constexpr (NP % 8 == 0) {
      if (n0 < NP) store8(dst, f);
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (n0 + j < NP) dst[j] = f[j];
    }
  };
  auto fetch = [&](int row0) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
#pragma unroll
      for (int j = 0; j < 4; ++j) x4[u][j] = dt4[u][j] = z4[u][j] = 0.f;
      const int t = vt + u * UR, row = first + row0 + t;
      if (v_on && t < TT && row0 + t < hi) {
        load4(p.x + (size_t)row * p.ldx + vc, x4[u]);
        load4(p.dt + (size_t)row * p.ldd + vc, dt4[u]);
        if (PASS == 0) load4(p.z + (size_t)row * p.ldz + vc, z4[u]);
      }
    }
    if (tid < TT * nbc) fetch_bc(tid, row0, bc8);
  };
  fetch(lo);
  float sum = 0.f;
  for (int row0 = lo; row0 < hi; row0 += TT) {
    float xc[U][4], zc[U][4];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int t = vt + u * UR;
      const bool have = v_on && row0 + t < hi;
      float v[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        xc[u][j] = x4[u][j];
        zc[u][j] = z4[u][j];
        v[j] = have ? softplus<FAST>(dt4[u][j] + bias4[j]) : 0.f;
      }
      if (t < TT) {
        float4* dst = reinterpret_cast<float4*>(sdt + t * CB + vl);
        dst[0] = make_float4(v[0], v[0] * xc[u][0], v[1], v[1] * xc[u][1]);
        dst[1] = make_float4(v[2], v[2] * xc[u][2], v[3], v[3] * xc[u][3]);
      }
    }
    if (tid < TT * nbc) put_bc(tid, bc8);
    for (int i = tid + THREADS; i < TT * nbc; i += THREADS) {
      float f[8];
      fetch_bc(i, row0, f);
      put_bc(i, f);
    }
    __syncthreads();
    if (row0 + TT < hi) fetch(row0 + TT);
    const int n_rows = min(TT, hi - row0);
    for (int t = 0; t < n_rows; t += 4) {
      float y[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const float2 dd = sdt[(t + u) * CB + ch];
        const float* bcr = sbc + (t + u) * 2 * NP + lane * NS;
        float b[NS];
        load_ns(bcr, b);
#pragma unroll
        for (int i = 0; i < NS; ++i) s[i] = fmaf(decay<FAST>(dd.x * a[i]), s[i], dd.y * b[i]);
        if (PASS == 0) {
          float cc[NS];
          load_ns(bcr + NP, cc);
          y[u] = 0.f;
#pragma unroll
          for (int i = 0; i < NS; ++i) y[u] = fmaf(s[i], cc[i], y[u]);
        } else {
          sum += dd.x;
        }
      }
      if (PASS == 0) {
        // lane l (mod 4) ends up with the sum of step l
        const bool up2 = lane & 2, up1 = lane & 1;
        float q0 = up2 ? y[2] : y[0], q1 = up2 ? y[3] : y[1];
        q0 += __shfl_xor_sync(0xffffffffu, up2 ? y[0] : y[2], 2);
        q1 += __shfl_xor_sync(0xffffffffu, up2 ? y[1] : y[3], 2);
        float q = (up1 ? q1 : q0) + __shfl_xor_sync(0xffffffffu, up1 ? q0 : q1, 1);
#pragma unroll
        for (int o = 4; o < L; o <<= 1) q += __shfl_xor_sync(0xffffffffu, q, o);
        if (lane < 4) sy[(t + lane) * CB + ch] = q;
      }
    }
    __syncthreads();
    if (PASS == 0) {
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int t = vt + u * UR;
        if (v_on && t < TT && row0 + t < hi) {
          float o[4];
          load4(sy + t * CB + vl, o);
#pragma unroll
          for (int j = 0; j < 4; ++j) o[j] = fmaf(d4[j], xc[u][j], o[j]) * silu<FAST>(zc[u][j]);
          store4(p.out + (size_t)(first + row0 + t) * p.ldo + vc, o);
        }
      }
    }
  }

  if (PASS == 1) {
    if (on) {
#pragma unroll
      for (int i = 0; i < NS; ++i) {
        const int n = lane * NS + i;
        if (n < p.N) ws[slice * cn + n] = s[i];
      }
      if (lane == 0) p.ws_sum[((size_t)e * p.slices + slice) * p.C + c] = sum;
    }
    return;
  }
  if (hi < len) return;
  if (on) {
#pragma unroll
    for (int i = 0; i < NS; ++i) {
      const int n = lane * NS + i;
      if (n < p.N) st[n] = s[i];
    }
  }
  if (p.xin && tid < CB && c0 + tid < p.C) replace_tail(p, slot, first, len, c0 + tid);
}

// Sequences with a single row: L lanes share a channel, NS states each, straight from and to memory.
template <typename T, int L, int NS>
__global__ void __launch_bounds__(THREADS) scan_step_kernel(ScanParams<T> p) {
  constexpr bool FAST = sizeof(T) == 2;
  constexpr int CB = THREADS / L;
  pdl_grid_trigger();
  const int ch = threadIdx.x / L, lane = threadIdx.x % L, c = blockIdx.x * CB + ch, e = blockIdx.y;
  const bool on = c < p.C;
  const bool vec = NS % 4 == 0 && p.N == L * NS;              // rows of whole 16-byte vectors
  float a[NS], s[NS], b[NS], cc[NS];
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    const int n = lane * NS + i;
    a[i] = on && n < p.N ? p.a[(size_t)c * p.N + n] : 0.f;
  }
  const float bias = on ? p.dt_bias[c] : 0.f, dskip = on ? p.d_skip[c] : 0.f;
  pdl_grid_wait();
  if (p.ent_len[e] != 1) return;                              // uniform per block
  const int row = p.ent_first[e], slot = p.ent_slot[e], pos = p.positions[row];
  float* st = p.state + ((size_t)slot * p.C + c) * p.N;
  const T* bcr = p.bc + (size_t)row * p.ldb;
  if (vec && on) {
    load_ns<NS>(st + lane * NS, s);
  } else {
#pragma unroll
    for (int i = 0; i < NS; ++i) s[i] = on && lane * NS + i < p.N ? st[lane * NS + i] : 0.f;
  }
  const float dt = on ? p.dt[(size_t)row * p.ldd + c] : 0.f;
  const float x = on ? (float)p.x[(size_t)row * p.ldx + c] : 0.f, z = on ? (float)p.z[(size_t)row * p.ldz + c] : 0.f;
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    const int n = lane * NS + i;
    b[i] = n < p.N ? (float)bcr[p.b_off + n] : 0.f;
    cc[i] = n < p.N ? (float)bcr[p.c_off + n] : 0.f;
    if (pos == 0) s[i] = 0.f;
  }
  const float delta = softplus<FAST>(dt + bias), dx = delta * x;
  float y = 0.f;
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    s[i] = fmaf(decay<FAST>(delta * a[i]), s[i], dx * b[i]);
    y = fmaf(s[i], cc[i], y);
  }
#pragma unroll
  for (int o = 1; o < L; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
  if (!on) return;
  if (vec) {
#pragma unroll
    for (int i = 0; i < NS; i += 4) *reinterpret_cast<float4*>(st + lane * NS + i) = make_float4(s[i], s[i + 1 < NS ? i + 1 : 0], s[i + 2 < NS ? i + 2 : 0], s[i + 3 < NS ? i + 3 : 0]);
  } else {
#pragma unroll
    for (int i = 0; i < NS; ++i)
      if (lane * NS + i < p.N) st[lane * NS + i] = s[i];
  }
  if (lane == 0) {
    p.out[(size_t)row * p.ldo + c] = (T)(fmaf(dskip, x, y) * silu<FAST>(z));
    if (p.xin) replace_tail(p, slot, row, 1, c);
  }
}

template <typename T, int L, int NS>
int launch_scan(const ScanParams<T>& p, int entries, int max_len, int singles, cudaStream_t stream) {
  constexpr int CB = THREADS / L;
  const size_t smem = (size_t)(TT * CB * 3 + TT * 2 * L * NS) * 4;
  static PerDeviceOnce once_;
  bool& configured = once_.slot();
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(scan_kernel<T, L, NS, 0>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(scan_kernel<T, L, NS, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const int blocks = (p.C + CB - 1) / CB;
  cudaError_t e = cudaSuccess;
  if (singles) e = launch_pdl(scan_step_kernel<T, L, NS>, dim3(blocks, entries), dim3(THREADS), 0, stream, p);
  if (e == cudaSuccess && max_len > 1 && p.slices > 1)
    e = launch_pdl(scan_kernel<T, L, NS, 1>, dim3(blocks, p.slices - 1, entries), dim3(THREADS), smem, stream, p);
  if (e == cudaSuccess && max_len > 1)
    e = launch_pdl(scan_kernel<T, L, NS, 0>, dim3(blocks, p.slices, entries), dim3(THREADS), smem, stream, p);
  return (int)e;
}

template <typename T>
int run_scan(ScanParams<T> p, int entries, int max_len, int singles, cudaStream_t stream) {
  const int per_lane = (p.N + 3) / 4;
  if (per_lane <= 1) return launch_scan<T, 4, 1>(p, entries, max_len, singles, stream);
  if (per_lane <= 2) return launch_scan<T, 4, 2>(p, entries, max_len, singles, stream);
  if (per_lane <= 4) return launch_scan<T, 4, 4>(p, entries, max_len, singles, stream);
  if (per_lane <= 6) return launch_scan<T, 4, 6>(p, entries, max_len, singles, stream);
  if (per_lane <= 8) return launch_scan<T, 4, 8>(p, entries, max_len, singles, stream);
  if (per_lane <= 16) return launch_scan<T, 8, 8>(p, entries, max_len, singles, stream);
  if (per_lane <= 32) return launch_scan<T, 16, 8>(p, entries, max_len, singles, stream);
  if (per_lane <= 64) return launch_scan<T, 32, 8>(p, entries, max_len, singles, stream);
  return -6;
}

}  // namespace

// Channels per block of the kernel that serves N states (the caller chooses the slices from it); 0: not supported.
extern "C" int b200_selective_scan_channels(int N) {
  if (N <= 0 || N > 256) return 0;
  return THREADS / (N <= 32 ? 4 : N <= 64 ? 8 : N <= 128 ? 16 : 32);
}

// rows of `entries` sequences (ent_first / ent_len / ent_slot; positions per row), the longest with max_len rows; singles != 0:
// some have one row.  slices > 1: slice i of a sequence
// starts at row i * per (per a multiple of 32, slices * per >= the longest sequence); ws_state / ws_sum are given.
extern "C" int b200_selective_scan(const void* x, int ldx, const float* dt, int ldd, const void* bc, int ldb, int b_off,
                                   int c_off, const void* z, int ldz, void* out, int ldo, const float* a, const float* dt_bias,
                                   const float* d_skip, float* state, const int* ent_first, const int* ent_len,
                                   const int* ent_slot, const int* positions, const void* xin, int ldin, void* tail, int taps,
                                   int C, int N, int entries, int max_len, int singles, int slices, int per, float* ws_state,
                                   float* ws_sum, int f32, cudaStream_t stream) {
  if (C <= 0 || (C & 7) || N <= 0 || N > 256 || entries <= 0 || entries > 65535 || slices < 1 || slices > 65535 || per < 1 ||
      taps < 1 || max_len < 1 || (ldx & 7) || (ldd & 7) || (ldb & 7) || (b_off & 7) || (c_off & 7) || c_off - b_off < N || (ldz & 7) ||
      (ldo & 7) || (slices > 1 && (per % TT || !ws_state || !ws_sum)))
    return -6;
#define B200_FILL(TT_)                                                                                                     \
  ScanParams<TT_> p;                                                                                                       \
  p.x = reinterpret_cast<const TT_*>(x); p.dt = dt; p.bc = reinterpret_cast<const TT_*>(bc);                               \
  p.z = reinterpret_cast<const TT_*>(z); p.out = reinterpret_cast<TT_*>(out); p.a = a; p.dt_bias = dt_bias;                \
  p.d_skip = d_skip; p.state = state; p.ent_first = ent_first; p.ent_len = ent_len; p.ent_slot = ent_slot;                 \
  p.positions = positions; p.xin = taps > 1 ? reinterpret_cast<const TT_*>(xin) : nullptr;                                 \
  p.tail = reinterpret_cast<TT_*>(tail); p.ws_state = ws_state; p.ws_sum = ws_sum; p.ldx = ldx; p.ldd = ldd; p.ldb = ldb;  \
  p.b_off = b_off; p.c_off = c_off; p.ldz = ldz; p.ldo = ldo; p.ldin = ldin; p.taps = taps; p.C = C; p.N = N;              \
  p.slices = slices; p.per = per;                                                                                          \
  return run_scan(p, entries, max_len, singles, stream);
  if (f32) {
    B200_FILL(float)
  } else {
    B200_FILL(__nv_bfloat16)
  }
#undef B200_FILL
}
