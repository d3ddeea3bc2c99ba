// Attention of single query rows over a paged KV cache with a sliding window and a bias per head and distance:
//
//   s(j) = scale q . k(j) + bias[h, p - j],   p - size < j <= p,       o = softmax(s) v
//
// Two kernels, both for one row and one slice of its window per block:
//
// bf16 (window_rows_mma_kernel): up to sixteen query heads of one key/value head.  Every warp streams its own tiles of 16 keys
// from the cache into registers, which ARE the tensor-core fragments: the order of the dimensions inside a dot product is free,
// so a lane takes 16 contiguous bytes of a key as its share of two k-steps; value columns are assigned to the lanes eight at a
// time for the same reason and two keys' words are interleaved by byte permutes.  Tiles are aligned to the cache rows, so a
// tile never leaves its page; keys in front of the window are masked.
//
// fp32 and sizes outside the first (window_rows_kernel): one head per block, the warps share the keys, the lanes share the
// dimensions of a key and the columns of a value.
//
// Slices leave (maximum, sum, weighted values); a second kernel merges them.  With one slice the result is written directly.
#include "launch.h"
#include "ops.h"
#include "per_device.h"
#include "vec8.cuh"

namespace {
using namespace b200;

template <typename T>
struct WindowRowsParams {
  const T* q;                // [rows, H, D]
  const T *k_cache, *v_cache;// [pages * bs, G * D], [pages * bs, G * V]
  const float* bias;         // [H, size], in units of the exponent's base 2
  const int* block_table;    // [sequences, max_blocks]
  const int* seq;            // [rows] table row of each query row (null: row i)
  const int* positions;      // [rows]
  float* partial;            // [rows, splits, H, V + 8]
  T* out;                    // [rows, ldo]
  int max_blocks, bs, H, G, D, V, splits, size, heads, ldo;      // heads: query heads per block
  float scale_log2;
};

__device__ __forceinline__ void mma_bf16(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  const __nv_bfloat162 t = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&t);
}
__device__ __forceinline__ float pow2(float v) {
  float e;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(v));
  return e;
}

constexpr int WARPS = 4;

// KC: 32-dim chunks of a query / key, VB: 64-column blocks of a value.  heads <= 16, page size a multiple of 16.
template <int KC, int VB>
__global__ void __launch_bounds__(WARPS * 32) window_rows_mma_kernel(WindowRowsParams<__nv_bfloat16> p) {
  extern __shared__ __align__(16) float so[];               // [warps][16][64 VB] values, then [warps][16] maxima and sums
  pdl_grid_trigger();
  const int D = p.D, V = p.V, per_g = p.H / p.G, sub = per_g / p.heads;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gr = lane >> 2, kk = lane & 3;
  const int split = blockIdx.x, b = blockIdx.z, g = blockIdx.y / sub, h0 = g * per_g + (blockIdx.y % sub) * p.heads;
  float* s_m = so + WARPS * 16 * 64 * VB;
  float* s_l = s_m + WARPS * 16;
  pdl_grid_wait();
  const uint4 zero = make_uint4(0, 0, 0, 0);
  uint4 q[2][KC];                                            // head rows gr and gr + 8
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int c = 0; c < KC; ++c) {
      const int d = c * 32 + kk * 8, head = gr + 8 * m;
      q[m][c] = head < p.heads && d < D ? *reinterpret_cast<const uint4*>(p.q + ((size_t)b * p.H + h0 + head) * D + d) : zero;
    }
  const int pos = p.positions[b], lo = max(0, pos - p.size + 1), start = lo & ~15, n_keys = pos + 1 - start;
  const int per = ((n_keys + p.splits - 1) / p.splits + 16 * WARPS - 1) / (16 * WARPS) * (16 * WARPS);
  const int k0 = start + split * per, k1 = min(pos + 1, k0 + per);
  const int* bt = p.block_table + (size_t)(p.seq ? p.seq[b] : b) * p.max_blocks;
  const float* bias[2] = {p.bias + (size_t)(h0 + min(gr, p.heads - 1)) * p.size, p.bias + (size_t)(h0 + min(gr + 8, p.heads - 1)) * p.size};

  float o[VB][8][4];
#pragma unroll
  for (int v = 0; v < VB; ++v)
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) o[v][j][i] = 0.f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};

  int key0 = k0 + warp * 16;
  int page = key0 < k1 ? bt[key0 / p.bs] : 0;
  for (; key0 < k1; key0 += 16 * WARPS) {
    // a tile never leaves its page, and a page that holds a visible key is readable to its end
    const size_t row0 = (size_t)page * p.bs + key0 % p.bs;
    const int next = key0 + 16 * WARPS;
    page = next < k1 ? bt[next / p.bs] : 0;
    uint4 kf[2][KC], vf[4][VB];
    float bf[2][4];
#pragma unroll
    for (int nb = 0; nb < 2; ++nb) {
      const __nv_bfloat16* kr = p.k_cache + ((row0 + nb * 8 + gr) * p.G + g) * D + kk * 8;
#pragma unroll
      for (int c = 0; c < KC; ++c) kf[nb][c] = c * 32 + kk * 8 < D ? *reinterpret_cast<const uint4*>(kr + c * 32) : zero;
    }
#pragma unroll
    for (int nb = 0; nb < 2; ++nb)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int key = key0 + nb * 8 + kk * 2 + (i & 1);
        bf[nb][i] = key >= lo && key < k1 ? bias[i >> 1][pos - key] : -INFINITY;
      }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const __nv_bfloat16* vr = p.v_cache + ((row0 + (i >> 1) * 8 + kk * 2 + (i & 1)) * p.G + g) * V + gr * 8;
#pragma unroll
      for (int v = 0; v < VB; ++v) vf[i][v] = v * 64 + gr * 8 < V ? *reinterpret_cast<const uint4*>(vr + v * 64) : zero;
    }
    float s[2][4] = {};
#pragma unroll
    for (int nb = 0; nb < 2; ++nb)
#pragma unroll
      for (int c = 0; c < KC; ++c) {
        mma_bf16(s[nb], q[0][c].x, q[1][c].x, q[0][c].y, q[1][c].y, kf[nb][c].x, kf[nb][c].y);
        mma_bf16(s[nb], q[0][c].z, q[1][c].z, q[0][c].w, q[1][c].w, kf[nb][c].z, kf[nb][c].w);
      }
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int nb = 0; nb < 2; ++nb)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        s[nb][i] = fmaf(s[nb][i], p.scale_log2, bf[nb][i]);
        mx[i >> 1] = fmaxf(mx[i >> 1], s[nb][i]);
      }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
      mx[r] = fmaxf(mx[r], m_run[r]);                       // finite: a tile has a visible key
    }
    if (__any_sync(0xffffffffu, mx[0] > m_run[0] || mx[1] > m_run[1])) {
      const float a0 = pow2(m_run[0] - mx[0]), a1 = pow2(m_run[1] - mx[1]);
      l_run[0] *= a0;
      l_run[1] *= a1;
#pragma unroll
      for (int v = 0; v < VB; ++v)
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          o[v][j][0] *= a0; o[v][j][1] *= a0;
          o[v][j][2] *= a1; o[v][j][3] *= a1;
        }
      m_run[0] = mx[0];
      m_run[1] = mx[1];
    }
#pragma unroll
    for (int nb = 0; nb < 2; ++nb)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        s[nb][i] = pow2(s[nb][i] - m_run[i >> 1]);
        l_run[i >> 1] += s[nb][i];
      }
    const uint32_t a0 = pack_bf16(s[0][0], s[0][1]), a1 = pack_bf16(s[0][2], s[0][3]);
    const uint32_t a2 = pack_bf16(s[1][0], s[1][1]), a3 = pack_bf16(s[1][2], s[1][3]);
#pragma unroll
    for (int v = 0; v < VB; ++v) {
      const uint32_t* w0 = reinterpret_cast<const uint32_t*>(&vf[0][v]);
      const uint32_t* w1 = reinterpret_cast<const uint32_t*>(&vf[1][v]);
      const uint32_t* w2 = reinterpret_cast<const uint32_t*>(&vf[2][v]);
      const uint32_t* w3 = reinterpret_cast<const uint32_t*>(&vf[3][v]);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        mma_bf16(o[v][2 * i], a0, a1, a2, a3, __byte_perm(w0[i], w1[i], 0x5410), __byte_perm(w2[i], w3[i], 0x5410));
        mma_bf16(o[v][2 * i + 1], a0, a1, a2, a3, __byte_perm(w0[i], w1[i], 0x7632), __byte_perm(w2[i], w3[i], 0x7632));
      }
    }
  }

#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 1);
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 2);
    if (kk == 0) {
      s_m[warp * 16 + r * 8 + gr] = m_run[r];
      s_l[warp * 16 + r * 8 + gr] = l_run[r];
    }
  }
#pragma unroll
  for (int v = 0; v < VB; ++v)
#pragma unroll
    for (int h = 0; h < 4; ++h) {                           // (row half, column half) of the fragments
      float* dst = so + ((size_t)(warp * 16 + (h >> 1) * 8 + gr)) * 64 * VB + v * 64 + kk * 16 + (h & 1) * 8;
      float f[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] = o[v][j][h];
      store8(dst, f);
    }
  __syncthreads();
  const int nv = V / 4;
  for (int i = threadIdx.x; i < p.heads * nv; i += WARPS * 32) {
    const int row = i / nv, v = (i % nv) * 4;
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) M = fmaxf(M, s_m[w * 16 + row]);
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    float L = 0.f;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) {
      const float mw = s_m[w * 16 + row], f = mw == -INFINITY ? 0.f : pow2(mw - M);
      const float4 t = *reinterpret_cast<const float4*>(so + ((size_t)(w * 16 + row)) * 64 * VB + v);
      L = fmaf(f, s_l[w * 16 + row], L);
      acc.x = fmaf(f, t.x, acc.x); acc.y = fmaf(f, t.y, acc.y); acc.z = fmaf(f, t.z, acc.z); acc.w = fmaf(f, t.w, acc.w);
    }
    if (p.splits == 1) {
      const float inv = 1.f / L;
      uint2 u;
      u.x = pack_bf16(acc.x * inv, acc.y * inv);
      u.y = pack_bf16(acc.z * inv, acc.w * inv);
      *reinterpret_cast<uint2*>(p.out + (size_t)b * p.ldo + (size_t)(h0 + row) * V + v) = u;
    } else {
      float* dst = p.partial + (((size_t)b * p.splits + split) * p.H + h0 + row) * (V + 8);
      *reinterpret_cast<float4*>(dst + v) = acc;
      if (v == 0) { dst[V] = M; dst[V + 1] = L; }
    }
  }
}

constexpr int UK = 4;            // keys of a warp in flight

// grid (splits, H, rows).  DL, VL: dimensions and value columns per lane (a lane owns x, x + 32, ...).
template <typename T, int DL, int VL>
__global__ void __launch_bounds__(WARPS * 32) window_rows_kernel(WindowRowsParams<T> p) {
  extern __shared__ __align__(16) float so[];               // [warps][V], then maxima and sums
  pdl_grid_trigger();
  const int D = p.D, V = p.V, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int split = blockIdx.x, h = blockIdx.y, b = blockIdx.z, g = h / (p.H / p.G);
  float *s_m = so + WARPS * V, *s_l = s_m + WARPS;
  pdl_grid_wait();
  float q[DL], o[VL];
#pragma unroll
  for (int i = 0; i < DL; ++i) q[i] = lane + 32 * i < D ? (float)p.q[((size_t)b * p.H + h) * D + lane + 32 * i] : 0.f;
#pragma unroll
  for (int i = 0; i < VL; ++i) o[i] = 0.f;
  const int pos = p.positions[b], lo = max(0, pos - p.size + 1), n_keys = pos + 1 - lo, per = (n_keys + p.splits - 1) / p.splits;
  const int k0 = lo + split * per, k1 = min(pos + 1, k0 + per);
  const int* bt = p.block_table + (size_t)(p.seq ? p.seq[b] : b) * p.max_blocks;
  const float* bias = p.bias + (size_t)h * p.size;
  float m = -INFINITY, l = 0.f;
  for (int key0 = k0 + warp * UK; key0 < k1; key0 += WARPS * UK) {
    size_t row[UK];
    float s[UK], mx = m;
#pragma unroll
    for (int u = 0; u < UK; ++u) {
      const int key = min(key0 + u, k1 - 1);
      row[u] = ((size_t)bt[key / p.bs] * p.bs + key % p.bs) * p.G + g;
      s[u] = 0.f;
    }
#pragma unroll
    for (int u = 0; u < UK; ++u)
#pragma unroll
      for (int i = 0; i < DL; ++i)
        if (lane + 32 * i < D) s[u] = fmaf(q[i], (float)p.k_cache[row[u] * D + lane + 32 * i], s[u]);
#pragma unroll
    for (int u = 0; u < UK; ++u) {
      s[u] = warp_sum_all(s[u]);
      s[u] = key0 + u < k1 ? fmaf(s[u], p.scale_log2, bias[pos - key0 - u]) : -INFINITY;
      mx = fmaxf(mx, s[u]);
    }
    const float a = exp2f(m - mx);                           // the first key of a round is visible
    l *= a;
#pragma unroll
    for (int i = 0; i < VL; ++i) o[i] *= a;
    m = mx;
#pragma unroll
    for (int u = 0; u < UK; ++u) {
      const float e = exp2f(s[u] - m);
      l += e;
#pragma unroll
      for (int i = 0; i < VL; ++i)
        if (lane + 32 * i < V) o[i] = fmaf(e, (float)p.v_cache[row[u] * V + lane + 32 * i], o[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < VL; ++i)
    if (lane + 32 * i < V) so[warp * V + lane + 32 * i] = o[i];
  if (lane == 0) { s_m[warp] = m; s_l[warp] = l; }
  __syncthreads();
  float M = -INFINITY, L = 0.f, f[WARPS];
#pragma unroll
  for (int w = 0; w < WARPS; ++w) M = fmaxf(M, s_m[w]);
#pragma unroll
  for (int w = 0; w < WARPS; ++w) {
    f[w] = s_m[w] == -INFINITY ? 0.f : exp2f(s_m[w] - M);
    L = fmaf(f[w], s_l[w], L);
  }
  float* dst = p.partial + (((size_t)b * p.splits + split) * p.H + h) * (V + 8);
  for (int v = threadIdx.x; v < V; v += WARPS * 32) {
    float t = 0.f;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) t = fmaf(f[w], so[w * V + v], t);
    if (p.splits == 1) p.out[(size_t)b * p.ldo + (size_t)h * V + v] = (T)(t / L);
    else dst[v] = t;
  }
  if (p.splits > 1 && threadIdx.x == 0) { dst[V] = M; dst[V + 1] = L; }
}

// One block per (head, row).
template <typename T>
__global__ void window_merge_kernel(const float* __restrict__ partial, T* __restrict__ out, int splits, int H, int V, int ldo) {
  extern __shared__ float s_w[];                            // [splits]
  pdl_grid_trigger();
  pdl_grid_wait();
  const int h = blockIdx.x, b = blockIdx.y, lane = threadIdx.x & 31;
  const size_t stride = (size_t)H * (V + 8);
  const float* base = partial + ((size_t)b * splits * H + h) * (V + 8);
  if (threadIdx.x < 32) {
    float M = -INFINITY, L = 0.f;
    for (int s = lane; s < splits; s += 32) M = fmaxf(M, base[s * stride + V]);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, o));
    for (int s = lane; s < splits; s += 32) {
      const float m = base[s * stride + V], w = m == -INFINITY ? 0.f : exp2f(m - M);         // an empty slice has no maximum
      L += w * base[s * stride + V + 1];
      s_w[s] = w;
    }
    L = warp_sum_all(L);
    for (int s = lane; s < splits; s += 32) s_w[s] /= L;
  }
  __syncthreads();
  for (int d = threadIdx.x; d < V; d += blockDim.x) {
    float v = 0.f;
#pragma unroll 4
    for (int s = 0; s < splits; ++s) {
      const float w = s_w[s];
      if (w != 0.f) v = fmaf(w, base[s * stride + d], v);
    }
    out[(size_t)b * ldo + (size_t)h * V + d] = (T)v;
  }
}

template <int KC, int VB>
int launch_mma(const WindowRowsParams<__nv_bfloat16>& p, int rows, cudaStream_t stream) {
  const size_t smem = (size_t)WARPS * 16 * (64 * VB + 2) * 4;
  static PerDeviceOnce once_;
  bool& configured = once_.slot();
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(window_rows_mma_kernel<KC, VB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  return (int)launch_pdl(window_rows_mma_kernel<KC, VB>, dim3(p.splits, p.H / p.heads, rows), dim3(WARPS * 32), smem, stream, p);
}

// -1: sizes the tensor-core kernel does not cover
int run_mma(WindowRowsParams<__nv_bfloat16> p, int rows, cudaStream_t stream) {
  if (p.bs % 16 || (p.D & 7) || p.D > 128 || (p.V & 7) || p.V > 256) return -1;
  for (int r = 1; r <= 16; ++r)
    if ((p.H / p.G) % r == 0) p.heads = r;
  const int kc = (p.D + 31) / 32, vb = (p.V + 63) / 64;
#define B200_MMA(K)                                                                                  \
  case K:                                                                                            \
    return vb == 1 ? launch_mma<K, 1>(p, rows, stream) : vb == 2 ? launch_mma<K, 2>(p, rows, stream) \
                                                                 : launch_mma<K, 4>(p, rows, stream);
  switch (kc) {
    B200_MMA(1) B200_MMA(2) B200_MMA(3) B200_MMA(4)
  }
#undef B200_MMA
  return -1;
}
int run_mma(const WindowRowsParams<float>&, int, cudaStream_t) { return -1; }

template <typename T, int DL>
int launch_rows(const WindowRowsParams<T>& p, int rows, cudaStream_t stream) {
  const dim3 grid(p.splits, p.H, rows), block(WARPS * 32);
  const size_t smem = (size_t)WARPS * (p.V + 2) * 4;
  if (p.V <= 64) return (int)launch_pdl(window_rows_kernel<T, DL, 2>, grid, block, smem, stream, p);
  if (p.V <= 128) return (int)launch_pdl(window_rows_kernel<T, DL, 4>, grid, block, smem, stream, p);
  if (p.V <= 256) return (int)launch_pdl(window_rows_kernel<T, DL, 8>, grid, block, smem, stream, p);
  return (int)launch_pdl(window_rows_kernel<T, DL, 32>, grid, block, smem, stream, p);
}

template <typename T>
int run_rows(const void* q, const void* k_cache, const void* v_cache, const float* bias, void* out, const int* block_table, const int* seq,
             const int* positions, float* partial, int rows, int max_blocks, int bs, int H, int G, int D, int V, int size, int splits,
             int ldo, float scale, cudaStream_t stream) {
  WindowRowsParams<T> p;
  p.q = reinterpret_cast<const T*>(q); p.k_cache = reinterpret_cast<const T*>(k_cache); p.v_cache = reinterpret_cast<const T*>(v_cache);
  p.bias = bias; p.block_table = block_table; p.seq = seq; p.positions = positions; p.partial = partial; p.out = reinterpret_cast<T*>(out);
  p.max_blocks = max_blocks; p.bs = bs; p.H = H; p.G = G; p.D = D; p.V = V; p.splits = splits; p.size = size; p.heads = 1; p.ldo = ldo;
  p.scale_log2 = scale * 1.4426950408889634f;
  int e = run_mma(p, rows, stream);
  if (e == -1)
    e = D <= 64 ? launch_rows<T, 2>(p, rows, stream) : D <= 128 ? launch_rows<T, 4>(p, rows, stream)
        : D <= 256 ? launch_rows<T, 8>(p, rows, stream) : launch_rows<T, 32>(p, rows, stream);
  if (e || splits == 1) return e;
  const int threads = V <= 64 ? 64 : V < 256 ? (V + 31) / 32 * 32 : 256;
  return (int)launch_pdl(window_merge_kernel<T>, dim3(H, rows), dim3(threads), (size_t)splits * 4, stream, (const float*)partial,
                         reinterpret_cast<T*>(out), splits, H, V, ldo);
}

}  // namespace

// rows query rows; bias fp32 [H, size] (times log2 e); partial: fp32 [rows * splits * H * (V + 8)] for more than one split.  D, V,
// ldo multiples of 8, D and V at most 1024.  The pages of a row's whole window have to be in its table.
extern "C" int b200_attn_window_rows(const void* q, const void* k_cache, const void* v_cache, const float* bias, void* out,
                                     const int* block_table, const int* seq, const int* positions, float* partial, int rows,
                                     int max_blocks, int block_size, int H, int G, int D, int V, int size, int splits, int ldo,
                                     float scale, int f32, cudaStream_t stream) {
  if (rows <= 0 || rows > 65535 || H <= 0 || H > 65535 || G <= 0 || H % G || D <= 0 || (D & 7) || D > 1024 || V <= 0 || (V & 7) || V > 1024 ||
      size <= 0 || (ldo & 7) || ldo < H * V || block_size <= 0 || splits < 1 || splits > 4096 || (splits > 1 && !partial) || !bias)
    return -6;
  return f32 ? run_rows<float>(q, k_cache, v_cache, bias, out, block_table, seq, positions, partial, rows, max_blocks, block_size, H, G, D,
                               V, size, splits, ldo, scale, stream)
             : run_rows<__nv_bfloat16>(q, k_cache, v_cache, bias, out, block_table, seq, positions, partial, rows, max_blocks, block_size,
                                       H, G, D, V, size, splits, ldo, scale, stream);
}
