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
// walks tiles of 32 rows: step sizes and inputs are converted once per (row, channel) into shared memory (as pairs, for the
// two-wide fp32 instructions), the recurrence runs out of it with the states in registers, and four steps' partial sums are
// reduced over the lanes together (transposing butterfly).  The next tile's rows are in flight meanwhile, unconverted: a
// conversion would wait for them.  Narrow models take more lanes per channel.  Sequences that bring a single row (decoding)
// take a kernel of their own without the tiles.
//
// A long sequence with few channels does not fill the device: its rows are then cut into slices.  A first pass runs every
// slice but the last from a zero state (the first one from the slot's state) and keeps the end state and the sum of the
// step sizes; since the decay over a slice is exp(A sum delta), the second pass composes the state at its own start from
// those and produces the outputs.
//
// The last slice also replaces the slot's convolution tail (the inputs of the convolution in front); for a single row the
// convolution has done so already (conv_rows.cu).
#include "launch.h"
#include "ops.h"
#include "per_device.h"
#include "vec8.cuh"

namespace {
using namespace b200;

constexpr int THREADS = 128;
constexpr int TT = 32;                   // rows per tile
constexpr int STEP_THREADS = 128, STEP_CHANNELS = 1;      // single-row kernel

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

// Two neighbouring channels of a row as they lie in memory, converted when they are used.
__device__ __forceinline__ float2 widen(uint32_t v) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v)); }
__device__ __forceinline__ float2 widen(float2 v) { return v; }
template <typename T> struct Pair;
template <> struct Pair<__nv_bfloat16> { using type = uint32_t; };
template <> struct Pair<float> { using type = float2; };
__device__ __forceinline__ void store_pair(__nv_bfloat16* p, float a, float b) {
  *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b);
}
__device__ __forceinline__ void store_pair(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }

template <int NS>
__device__ __forceinline__ void load_quad(const __nv_bfloat16* p, float (&f)[NS]) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = widen(u.x), b = widen(u.y);
  f[0] = a.x; f[1 % NS] = a.y; f[2 % NS] = b.x; f[3 % NS] = b.y;
}
template <int NS>
__device__ __forceinline__ void load_quad(const float* p, float (&f)[NS]) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  f[0] = a.x; f[1 % NS] = a.y; f[2 % NS] = a.z; f[3 % NS] = a.w;
}

// fp32 pairs in 64-bit registers
__device__ __forceinline__ uint64_t pair_of(float a, float b) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float2 halves_of(uint64_t v) {
  float2 f;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(v));
  return f;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
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

// States of one lane, in pairs where their number is even.
template <int NS, bool FAST>
struct Lane {
  static constexpr int P = (NS + 1) / 2;
  uint64_t s[P], a[P];

  // S <- exp(delta a) S + dx b; returns this lane's part of sum_n S c.  dd: (delta, delta, dx, dx)
  template <bool OUT>
  __device__ __forceinline__ float step(const float4& dd, const float* b, const float* c) {
    if constexpr (NS == 1) {
      const float2 v = halves_of(s[0]);
      const float t = fmaf(decay<FAST>(dd.x * halves_of(a[0]).x), v.x, dd.z * b[0]);
      s[0] = pair_of(t, 0.f);
      return OUT ? t * c[0] : 0.f;
    } else {
      const uint64_t d2 = pair_of(dd.x, dd.y), x2 = pair_of(dd.z, dd.w);
      uint64_t bb[P], cc[P], y = 0;
      load(b, bb);
      if (OUT) load(c, cc);
#pragma unroll
      for (int i = 0; i < P; ++i) {
        const float2 e = halves_of(mul2(d2, a[i]));
        s[i] = fma2(pair_of(decay<FAST>(e.x), decay<FAST>(e.y)), s[i], mul2(x2, bb[i]));
        if (OUT) y = i ? fma2(s[i], cc[i], y) : mul2(s[i], cc[i]);
      }
      const float2 f = halves_of(y);
      return f.x + f.y;
    }
  }
  __device__ __forceinline__ static void load(const float* p, uint64_t (&v)[P]) {
    if constexpr (NS % 4 == 0) {
#pragma unroll
      for (int i = 0; i < P; i += 2) {
        const ulonglong2 t = *reinterpret_cast<const ulonglong2*>(p + 2 * i);
        v[i] = t.x;
        v[i + 1] = t.y;
      }
    } else {
#pragma unroll
      for (int i = 0; i < P; ++i) v[i] = *reinterpret_cast<const uint64_t*>(p + 2 * i);
    }
  }
  // f(n): value of the lane's n-th state
  template <typename F>
  __device__ __forceinline__ static void fill(uint64_t (&v)[P], F f) {
#pragma unroll
    for (int i = 0; i < P; ++i) v[i] = pair_of(f(2 * i), 2 * i + 1 < NS ? f(2 * i + 1) : 0.f);
  }
  template <typename F>
  __device__ __forceinline__ void each(F f) const {
#pragma unroll
    for (int i = 0; i < P; ++i) {
      const float2 v = halves_of(s[i]);
      f(2 * i, v.x);
      if (2 * i + 1 < NS) f(2 * i + 1, v.y);
    }
  }
};

// PASS 0: the whole sequence or (slices > 1) the outputs of one slice; PASS 1: end state of one slice.
template <typename T, int L, int NS, int PASS>
__global__ void __launch_bounds__(THREADS) scan_kernel(ScanParams<T> p) {
  constexpr bool FAST = sizeof(T) == 2;
  constexpr int CB = THREADS / L, NP = L * NS, YP = CB + 8;
  constexpr int CV = CB / 2, UR = THREADS / CV, U = (TT + UR - 1) / UR;         // units of two channels; rows UR apart
  using pair_t = typename Pair<T>::type;
  extern __shared__ __align__(16) float sm[];
  float4* sdt = reinterpret_cast<float4*>(sm);              // [TT][CB]: (delta, delta, delta x, delta x)
  float* sbc = sm + TT * CB * 4;                            // [TT][2][NP]
  float* sy = sbc + TT * 2 * NP;                            // [TT][YP]
  pdl_grid_trigger();
  const int tid = threadIdx.x, ch = tid / L, lane = tid % L, c0 = blockIdx.x * CB, c = c0 + ch;
  const bool on = c < p.C;
  using LaneT = Lane<NS, FAST>;
  LaneT st;
  LaneT::fill(st.a, [&](int i) { return on && lane * NS + i < p.N ? p.a[(size_t)c * p.N + lane * NS + i] : 0.f; });
  for (int i = tid; i < TT * 2 * NP; i += THREADS) sbc[i] = 0.f;        // states past N stay zero
  // this thread's units of a tile: rows vt, vt + UR, .., channels vc, vc + 1
  const int vt = tid / CV, vl = (tid % CV) * 2, vc = c0 + vl;
  const bool v_on = vc < p.C && vt < TT;
  float2 bias = make_float2(0.f, 0.f), dskip = bias;
  if (v_on) {
    bias = *reinterpret_cast<const float2*>(p.dt_bias + vc);
    dskip = *reinterpret_cast<const float2*>(p.d_skip + vc);
  }
  pdl_grid_wait();
  const int e = blockIdx.z, slice = blockIdx.y;
  const int len = p.ent_len[e], lo = slice * p.per, hi = min(len, lo + p.per);
  const bool single = len <= p.per;
  if (len == 1 || lo >= len || (PASS == 1 && (single || hi == len))) return;      // uniform per block
  const int first = p.ent_first[e], slot = p.ent_slot[e], pos = p.positions[first];
  const size_t cn = (size_t)p.C * p.N;
  float* state = p.state + (size_t)slot * cn + (size_t)c * p.N;
  float* ws = p.ws_state ? p.ws_state + (size_t)e * p.slices * cn + (size_t)c * p.N : nullptr;

  LaneT::fill(st.s, [&](int i) {
    const int n = lane * NS + i;
    if (!on || n >= p.N) return 0.f;
    float v;
    if (slice == 0) {
      v = PASS == 1 || single ? (pos == 0 ? 0.f : state[n]) : ws[(size_t)(p.slices - 1) * cn + n];
      if (PASS == 1) ws[(size_t)(p.slices - 1) * cn + n] = v;
      return v;
    }
    if (PASS == 1) return 0.f;
    v = ws[n];
    const float an = p.a[(size_t)c * p.N + n];
    for (int k = 1; k < slice; ++k) v = fmaf(decay<FAST>(p.ws_sum[((size_t)e * p.slices + k) * p.C + c] * an), v, ws[k * cn + n]);
    return v;
  });

  const int nb8 = (p.c_off - p.b_off) / 8, nbc = 2 * nb8;               // vectors of B (and of C) per row
  pair_t xr[U], zr[U];
  float2 dtr[U];
  constexpr int BW = 8 * (int)sizeof(T) / 16;                           // 16-byte words of eight values
  uint4 bcr[BW];
  const int bt = tid / nbc, bv = tid % nbc;                             // first B | C vector of this thread
  float* const bdst = sbc + (bt * 2 + bv / nb8) * NP + (bv % nb8) * 8;
  const int bn0 = (bv % nb8) * 8;
  auto put_bc = [&](float* dst, int n0, const uint4 (&raw)[BW]) {
    float f[8];
    load8(reinterpret_cast<const T*>(raw), f);
    if constexpr (NP % 8 == 0) {
      if (n0 < NP) store8(dst, f);
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (n0 + j < NP) dst[j] = f[j];
    }
  };
  auto fetch_bc = [&](int t, int v, int row0, uint4 (&raw)[BW]) {
#pragma unroll
    for (int j = 0; j < BW; ++j)
      raw[j] = row0 + t < hi ? reinterpret_cast<const uint4*>(p.bc + (size_t)(first + row0 + t) * p.ldb + p.b_off + v * 8)[j]
                             : make_uint4(0, 0, 0, 0);
  };
  auto fetch = [&](int row0) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int t = vt + u * UR, row = first + row0 + t;
      if (v_on && row0 + t < hi) {
        xr[u] = *reinterpret_cast<const pair_t*>(p.x + (size_t)row * p.ldx + vc);
        dtr[u] = *reinterpret_cast<const float2*>(p.dt + (size_t)row * p.ldd + vc);
        if (PASS == 0) zr[u] = *reinterpret_cast<const pair_t*>(p.z + (size_t)row * p.ldz + vc);
      }
    }
    if (bt < TT) fetch_bc(bt, bv, row0, bcr);
  };
  fetch(lo);
  float sum = 0.f;
  for (int row0 = lo; row0 < hi; row0 += TT) {
    pair_t xc[U], zc[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int t = vt + u * UR;
      if (U * UR > TT && t >= TT) continue;
      float4 q0 = make_float4(0.f, 0.f, 0.f, 0.f), q1 = q0;
      if (v_on && row0 + t < hi) {
        const float2 x = widen(xr[u]);
        const float d0 = softplus<FAST>(dtr[u].x + bias.x), d1 = softplus<FAST>(dtr[u].y + bias.y);
        q0 = make_float4(d0, d0, d0 * x.x, d0 * x.x);
        q1 = make_float4(d1, d1, d1 * x.y, d1 * x.y);
        xc[u] = xr[u];
        if (PASS == 0) zc[u] = zr[u];
      }
      sdt[t * CB + vl] = q0;
      sdt[t * CB + vl + 1] = q1;
    }
    if (bt < TT) put_bc(bdst, bn0, bcr);
    for (int i = tid + THREADS; i < TT * nbc; i += THREADS) {
      const int t = i / nbc, v = i % nbc, n0 = (v % nb8) * 8;
      uint4 raw[BW];
      fetch_bc(t, v, row0, raw);
      put_bc(sbc + (t * 2 + v / nb8) * NP + n0, n0, raw);
    }
    __syncthreads();
    if (row0 + TT < hi) fetch(row0 + TT);
    const int n_rows = min(TT, hi - row0);
    const float4* dp = sdt + ch;
    const float* bp = sbc + lane * NS;
    float* yp = sy + lane * YP + ch;
#pragma unroll 2
    for (int t = 0; t < n_rows; t += 4, dp += 4 * CB, bp += 8 * NP, yp += 4 * YP) {
      float y[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const float4 dd = dp[u * CB];
        y[u] = st.template step<PASS == 0>(dd, bp + u * 2 * NP, bp + u * 2 * NP + NP);
        if (PASS == 1) sum += dd.x;
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
        if (lane < 4) *yp = q;
      }
    }
    __syncthreads();
    if (PASS == 0) {
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int t = vt + u * UR;
        if (v_on && t < TT && row0 + t < hi) {
          const float2 y = *reinterpret_cast<const float2*>(sy + t * YP + vl), x = widen(xc[u]), z = widen(zc[u]);
          store_pair(p.out + (size_t)(first + row0 + t) * p.ldo + vc, fmaf(dskip.x, x.x, y.x) * silu<FAST>(z.x),
                     fmaf(dskip.y, x.y, y.y) * silu<FAST>(z.y));
        }
      }
    }
  }

  if (PASS == 1) {
    if (on) {
      st.each([&](int i, float v) {
        if (lane * NS + i < p.N) ws[slice * cn + lane * NS + i] = v;
      });
      if (lane == 0) p.ws_sum[((size_t)e * p.slices + slice) * p.C + c] = sum;
    }
    return;
  }
  if (hi < len) return;
  if (on)
    st.each([&](int i, float v) {
      if (lane * NS + i < p.N) state[lane * NS + i] = v;
    });
  if (p.xin && tid < CB && c0 + tid < p.C) replace_tail(p, slot, first, len, c0 + tid);
}

// Sequences with a single row, straight from and to memory: L lanes share a channel, NS states each, KC channels per thread.
template <typename T, int L, int NS, int KC>
__global__ void __launch_bounds__(STEP_THREADS) scan_step_kernel(ScanParams<T> p) {
  constexpr bool FAST = sizeof(T) == 2;
  constexpr int CB = STEP_THREADS / L;
  using LaneT = Lane<NS, FAST>;
  pdl_grid_trigger();
  const int lane = threadIdx.x % L, c0 = blockIdx.x * CB * KC + threadIdx.x / L, e = blockIdx.y;
  const bool vec = NS % 4 == 0 && p.N == L * NS;              // rows of whole 16-byte vectors
  LaneT st[KC];
  float bias[KC], dskip[KC];
#pragma unroll
  for (int k = 0; k < KC; ++k) {
    const int c = c0 + k * CB;
    const float* src = p.a + (size_t)c * p.N + lane * NS;
    if (vec && c < p.C) LaneT::load(src, st[k].a);
    else LaneT::fill(st[k].a, [&](int i) { return c < p.C && lane * NS + i < p.N ? src[i] : 0.f; });
    bias[k] = c < p.C ? p.dt_bias[c] : 0.f;
    dskip[k] = c < p.C ? p.d_skip[c] : 0.f;
  }
  pdl_grid_wait();
  const int row = p.ent_first[e], slot = p.ent_slot[e];
  if (p.ent_len[e] != 1) return;                              // uniform per block
  float dt[KC], x[KC], z[KC], b[NS], cc[NS];
#pragma unroll
  for (int k = 0; k < KC; ++k) {
    const int c = c0 + k * CB;
    const bool on = c < p.C;
    const float* s = p.state + ((size_t)slot * p.C + c) * p.N + lane * NS;
    if (vec && on) LaneT::load(s, st[k].s);
    else LaneT::fill(st[k].s, [&](int i) { return on && lane * NS + i < p.N ? s[i] : 0.f; });
    dt[k] = on ? p.dt[(size_t)row * p.ldd + c] : 0.f;
    x[k] = on ? (float)p.x[(size_t)row * p.ldx + c] : 0.f;
    z[k] = on ? (float)p.z[(size_t)row * p.ldz + c] : 0.f;
  }
  const T* bcr = p.bc + (size_t)row * p.ldb + lane * NS;
  if (NS == 4 && lane * NS < p.N) {                           // B and C are padded to whole vectors of eight
    load_quad(bcr + p.b_off, b);
    load_quad(bcr + p.c_off, cc);
  } else {
#pragma unroll
    for (int i = 0; i < NS; ++i) {
      b[i] = lane * NS + i < p.N ? (float)bcr[p.b_off + i] : 0.f;
      cc[i] = lane * NS + i < p.N ? (float)bcr[p.c_off + i] : 0.f;
    }
  }
  const bool fresh = p.positions[row] == 0;
#pragma unroll
  for (int k = 0; k < KC; ++k) {
    const int c = c0 + k * CB;
    const float delta = softplus<FAST>(dt[k] + bias[k]), dx = delta * x[k];
    if (fresh) LaneT::fill(st[k].s, [](int) { return 0.f; });
    float y = 0.f;
#pragma unroll
    for (int i = 0; i < LaneT::P; ++i) {
      const float2 av = halves_of(st[k].a[i]), sv = halves_of(st[k].s[i]);
      float out[2] = {0.f, 0.f};
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        if (2 * i + h < NS) {
          out[h] = fmaf(decay<FAST>(delta * (h ? av.y : av.x)), h ? sv.y : sv.x, dx * b[2 * i + h < NS ? 2 * i + h : 0]);
          y = fmaf(out[h], cc[2 * i + h < NS ? 2 * i + h : 0], y);
        }
      }
      st[k].s[i] = pair_of(out[0], out[1]);
    }
#pragma unroll
    for (int o = 1; o < L; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (c >= p.C) continue;
    float* s = p.state + ((size_t)slot * p.C + c) * p.N + lane * NS;
    if (vec) {
      if constexpr (NS % 4 == 0) {
#pragma unroll
        for (int i = 0; i < NS / 2; i += 2) *reinterpret_cast<ulonglong2*>(s + 2 * i) = make_ulonglong2(st[k].s[i], st[k].s[i + 1]);
      }
    } else {
      st[k].each([&](int i, float v) {
        if (lane * NS + i < p.N) s[i] = v;
      });
    }
    if (lane == 0) p.out[(size_t)row * p.ldo + c] = (T)(fmaf(dskip[k], x[k], y) * silu<FAST>(z[k]));
  }
}

template <typename T, int L, int NS>
int launch_tiles(const ScanParams<T>& p, int entries, cudaStream_t stream) {
  constexpr int CB = THREADS / L;
  const size_t smem = (size_t)(TT * CB * 4 + TT * 2 * L * NS + TT * (CB + 8)) * 4;
  static PerDeviceOnce once_;
  bool& configured = once_.slot();
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(scan_kernel<T, L, NS, 0>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(scan_kernel<T, L, NS, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const int blocks = (p.C + CB - 1) / CB;
  // ordinary launches: a grid of one long wave that starts while its predecessor still holds some of the SMs is crowded
  // onto the others for its whole run
  if (p.slices > 1) scan_kernel<T, L, NS, 1><<<dim3(blocks, p.slices - 1, entries), THREADS, smem, stream>>>(p);
  scan_kernel<T, L, NS, 0><<<dim3(blocks, p.slices, entries), THREADS, smem, stream>>>(p);
  return (int)cudaGetLastError();
}

template <typename T, int L, int NS>
int launch_step(const ScanParams<T>& p, int entries, cudaStream_t stream) {
  constexpr int PER = STEP_THREADS / L * STEP_CHANNELS;
  return (int)launch_pdl(scan_step_kernel<T, L, NS, STEP_CHANNELS>, dim3((p.C + PER - 1) / PER, entries), dim3(STEP_THREADS), 0,
                         stream, p);
}

// Lanes per channel of the tile kernel: as few as hold the states, more for batches whose channels alone would leave the
// schedulers with less than three warps.
int pick_lanes(int C, int N, int entries) {
  int lanes = N <= 32 ? 4 : N <= 64 ? 8 : N <= 128 ? 16 : 32;
  if (lanes == 4 && N > 8 && (N <= 16 || N > 24) && (long long)C * entries * 4 < 148LL * 12 * 32) lanes = 8;
  return lanes;
}

template <typename T>
int run_scan(const ScanParams<T>& p, int entries, int max_len, int singles, cudaStream_t stream) {
  const int per_lane = (p.N + 3) / 4;
  int e = 0;
  if (singles) {
    e = per_lane <= 1    ? launch_step<T, 4, 1>(p, entries, stream)
        : per_lane <= 2  ? launch_step<T, 4, 2>(p, entries, stream)
        : per_lane <= 4  ? launch_step<T, 4, 4>(p, entries, stream)
        : per_lane <= 8  ? launch_step<T, 8, 4>(p, entries, stream)
        : per_lane <= 16 ? launch_step<T, 16, 4>(p, entries, stream)
        : per_lane <= 32 ? launch_step<T, 32, 4>(p, entries, stream)
                         : launch_step<T, 32, 8>(p, entries, stream);
    if (e || max_len == 1) return e;
  }
  const int lanes = pick_lanes(p.C, p.N, entries);
  if (lanes == 4) {
    if (per_lane <= 1) return launch_tiles<T, 4, 1>(p, entries, stream);
    if (per_lane <= 2) return launch_tiles<T, 4, 2>(p, entries, stream);
    if (per_lane <= 4) return launch_tiles<T, 4, 4>(p, entries, stream);
    if (per_lane <= 6) return launch_tiles<T, 4, 6>(p, entries, stream);
    return launch_tiles<T, 4, 8>(p, entries, stream);
  }
  if (lanes == 8) {
    if (per_lane <= 4) return launch_tiles<T, 8, 2>(p, entries, stream);
    if (per_lane <= 8) return launch_tiles<T, 8, 4>(p, entries, stream);
    return launch_tiles<T, 8, 8>(p, entries, stream);
  }
  return lanes == 16 ? launch_tiles<T, 16, 8>(p, entries, stream) : launch_tiles<T, 32, 8>(p, entries, stream);
}

}  // namespace

// Time slices per sequence of at most max_len rows: cutting doubles the recurrence's work, so only where whole sequences
// occupy less than half of the SMs.  0: a state count the kernel does not serve.
extern "C" int b200_selective_scan_slices(int C, int N, int entries, int max_len) {
  if (C <= 0 || N <= 0 || N > 256 || entries <= 0) return 0;
  const int cb = THREADS / pick_lanes(C, N, entries);
  const long long blocks = (long long)((C + cb - 1) / cb) * entries;
  if (blocks * 2 > 148) return 1;
  long long s = 4 * 148 / blocks;
  if (s > max_len / 256) s = max_len / 256;
  return s < 1 ? 1 : (int)s;
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
