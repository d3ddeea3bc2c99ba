// Differential attention of single query rows over a paged KV cache.  Every head has two softmax maps with their own query
// and key vectors and a common value:
//
//   a_m = softmax_j(scale q_m . k_m(j)) v(j),   o = finish(a_1 - lambda a_2)        (attn_diff.cuh)
//
// Two kernels, both for one row, up to eight query heads of one key/value head and one slice of the row's keys per block.
//
// bf16 (diff_rows_mma_kernel): every warp streams its own tiles of 16 keys from the cache into registers, which ARE the
// tensor-core fragments.  The heads' map-1 queries are rows 0-7 of the A operand and the map-2 queries rows 8-15 (two
// products against the two maps' keys fill one score tile), so that one P V product serves both maps.  The order of the
// dimensions inside a dot product is free, so a lane takes 16 contiguous bytes of a key as its share of two k-steps; value
// columns are assigned to the lanes eight at a time for the same reason and two keys' words are interleaved by byte permutes.
//
// fp32 and sizes outside the first (diff_rows_kernel): tiles of TK tokens (both maps' keys and the values) are staged in shared memory, double-buffered, and serve all the block's heads
// and maps.  Per tile: dot products (four lanes share a key and map, every head of the block per key element read), one
// warp per (head, map) for the online softmax, and P V with RQ (head, map) accumulators of eight values per thread, the
// keys cut among the threads.  Slices leave (maximum, sum, weighted values) per head and map; a second kernel merges them,
// takes the difference, normalises and gates.  Used for decode batches and short portions in bf16 and for every row in fp32.
#include "attn_diff.cuh"
#include "launch.h"
#include "ops.h"
#include "per_device.h"
#include "vec8.cuh"

namespace {
using namespace b200;

constexpr int THREADS = 256;
constexpr int QMAX = 16;                 // (head, map) pairs of a block

template <typename T>
struct DiffRowsParams {
  const T* q;                // [rows, H, 2, D]
  const T *k_cache, *v_cache;// [pages * bs, G * 2 * D], [pages * bs, G * V]
  const int* block_table;    // [sequences, max_blocks]
  const int* seq;            // [rows] table row of each query row (null: row i)
  const int* positions;      // [rows]
  float* partial;            // [rows, splits, H, 2, V + 8]
  int max_blocks, bs, H, G, D, V, splits, heads, tk, ks;      // heads: query heads per block; ks: key slices of P V
  float scale_log2;
};

__device__ __forceinline__ void cp16(void* dst, const void* src, bool ok) {
  const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
  const int n = ok ? 16 : 0;                                     // 0 source bytes: the 16 bytes are zero-filled
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

template <typename T>
__host__ __device__ inline int key_pitch(int D) { return 2 * D * (int)sizeof(T) + 16; }

template <typename T, int RQ, int IT>
__global__ void __launch_bounds__(THREADS) diff_rows_kernel(DiffRowsParams<T> p) {
  extern __shared__ __align__(16) uint8_t smem[];
  pdl_grid_trigger();
  const int D = p.D, V = p.V, TK = p.tk, NQ = 2 * p.heads, per_g = p.H / p.G, sub = per_g / p.heads;
  const int kp = key_pitch<T>(D), vp = V * (int)sizeof(T);
  float* sq = reinterpret_cast<float*>(smem);              // [NQ][D]: (head, map)
  float* s_m = sq + NQ * D;                                // [QMAX] running maximum, sum, rescale of this tile
  float* s_l = s_m + QMAX;
  float* s_a = s_l + QMAX;
  int* srow = reinterpret_cast<int*>(s_a + QMAX);          // [2][64] cache row of every key of the tile
  float* ss = reinterpret_cast<float*>(srow + 128);        // [NQ][TK] scores
  float* sp = ss + NQ * TK;                                // [TK][QMAX] weights
  uint8_t* sk = reinterpret_cast<uint8_t*>(sp + TK * QMAX);// [2][TK][kp]
  uint8_t* sv = sk + (size_t)2 * TK * kp;                  // [2][TK][vp]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int split = blockIdx.x, b = blockIdx.z, g = blockIdx.y / sub, h0 = g * per_g + (blockIdx.y % sub) * p.heads;
  if (tid < QMAX) { s_m[tid] = -INFINITY; s_l[tid] = 0.f; s_a[tid] = 0.f; }
  pdl_grid_wait();
  {
    const T* qrow = p.q + ((size_t)b * p.H + h0) * 2 * D;
    for (int i = tid; i < NQ * D / 8; i += THREADS) {
      float f[8];
      load8(qrow + i * 8, f);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] *= p.scale_log2;
      store8(sq + i * 8, f);
    }
  }
  const int n_keys = p.positions[b] + 1, per = (n_keys + p.splits - 1) / p.splits;
  const int k0 = split * per, k1 = min(n_keys, k0 + per);
  const int* bt = p.block_table + (size_t)(p.seq ? p.seq[b] : b) * p.max_blocks;
  const int kvecs = 2 * D * (int)sizeof(T) / 16, vvecs = vp / 16;

  auto locate = [&](int key0, int buf) {
    if (tid < TK) {
      const int key = key0 + tid;
      srow[buf * 64 + tid] = key < k1 ? bt[key / p.bs] * p.bs + key % p.bs : -1;
    }
  };
  auto stage = [&](int buf) {
    for (int r = warp; r < TK; r += THREADS / 32) {
      const int slot = srow[buf * 64 + r];
      const size_t at = (size_t)max(slot, 0);
      const uint8_t* ks = reinterpret_cast<const uint8_t*>(p.k_cache + (at * p.G + g) * 2 * D);
      const uint8_t* vs = reinterpret_cast<const uint8_t*>(p.v_cache + (at * p.G + g) * V);
      uint8_t* kd = sk + (size_t)(buf * TK + r) * kp;
      uint8_t* vd = sv + (size_t)(buf * TK + r) * vp;
      for (int c = lane; c < kvecs + vvecs; c += 32) {
        if (c < kvecs) cp16(kd + c * 16, ks + c * 16, slot >= 0);
        else cp16(vd + (c - kvecs) * 16, vs + (c - kvecs) * 16, slot >= 0);
      }
    }
    cp_commit();
  };

  // P V ownership: item = (eight-value column, RQ queries), key slice
  const int NC = V / 8, NI = NC * (NQ / RQ), KS = p.ks, per_slice = TK / KS;
  const int my_slice = KS > 1 ? tid / NI : 0;
  float acc[IT][RQ][8];
#pragma unroll
  for (int it = 0; it < IT; ++it)
#pragma unroll
    for (int r = 0; r < RQ; ++r)
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[it][r][j] = 0.f;

  locate(k0, 0);
  locate(k0 + TK, 1);
  __syncthreads();
  stage(0);
  int buf = 0;
  for (int key0 = k0; key0 < k1; key0 += TK, buf ^= 1) {
    if (key0 + TK < k1) {
      stage(buf ^ 1);
      cp_wait<1>();
    } else {
      cp_wait<0>();
    }
    __syncthreads();
    // scores: item = (key, map) shared by four lanes, all heads of the block
    for (int base = 0; base < TK * 8; base += THREADS) {
      const int i = base + tid, key = (i >> 3) % TK, map = (i >> 2) & 1, part = i & 3;      // TK * 8 is a multiple of 64
      const bool on = i < TK * 8;
      float dot[QMAX / 2];
#pragma unroll
      for (int r = 0; r < QMAX / 2; ++r) dot[r] = 0.f;
      if (on) {
        const T* kr = reinterpret_cast<const T*>(sk + (size_t)(buf * TK + key) * kp) + map * D;
        for (int d = part * 8; d < D; d += 32) {
          float kf[8];
          load8(kr + d, kf);
#pragma unroll
          for (int r = 0; r < QMAX / 2; ++r) {
            if (r < p.heads) {
              float qf[8];
              load8(sq + (r * 2 + map) * D + d, qf);
#pragma unroll
              for (int j = 0; j < 8; ++j) dot[r] = fmaf(qf[j], kf[j], dot[r]);
            }
          }
        }
      }
#pragma unroll
      for (int r = 0; r < QMAX / 2; ++r) {
        if (r < p.heads) {
          float s = dot[r];
          s += __shfl_xor_sync(0xffffffffu, s, 1);
          s += __shfl_xor_sync(0xffffffffu, s, 2);
          if (on && part == 0) ss[(r * 2 + map) * TK + key] = s;
        }
      }
    }
    __syncthreads();
    if (tid < TK && key0 + 2 * TK < k1) srow[buf * 64 + tid] = [&] {       // rows of the tile after next
      const int key = key0 + 2 * TK + tid;
      return key < k1 ? bt[key / p.bs] * p.bs + key % p.bs : -1;
    }();
    for (int r = warp; r < NQ; r += THREADS / 32) {
      float v[2], mx = -INFINITY;
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int key = lane + 32 * u;
        v[u] = key < TK && key0 + key < k1 ? ss[r * TK + key] : -INFINITY;
        mx = fmaxf(mx, v[u]);
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float m_old = s_m[r], m_new = fmaxf(m_old, mx);      // a tile always has a visible key
      float l = 0.f;
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int key = lane + 32 * u;
        const float e = exp2f(v[u] - m_new);
        l += e;
        if (key < TK) sp[key * QMAX + r] = e;
      }
      l = warp_sum_all(l);
      __syncwarp();
      if (lane == 0) {
        const float a = exp2f(m_old - m_new);                    // 0 for the first tile
        s_m[r] = m_new;
        s_a[r] = a;
        s_l[r] = s_l[r] * a + l;
      }
    }
    __syncthreads();
#pragma unroll
    for (int it = 0; it < IT; ++it) {
      const int i = KS > 1 ? tid % NI : tid + it * THREADS;
      if (i < NI && my_slice < KS) {
        const int q0 = (i / NC) * RQ, col = i % NC;
        float a[RQ];
#pragma unroll
        for (int r = 0; r < RQ; ++r) a[r] = s_a[q0 + r];
#pragma unroll
        for (int r = 0; r < RQ; ++r)
#pragma unroll
          for (int j = 0; j < 8; ++j) acc[it][r][j] *= a[r];
        const uint8_t* base = sv + (size_t)buf * TK * vp + col * 8 * sizeof(T);
        for (int key = my_slice * per_slice; key < (my_slice + 1) * per_slice; ++key) {
          float vf[8];
          load8(reinterpret_cast<const T*>(base + (size_t)key * vp), vf);
#pragma unroll
          for (int r = 0; r < RQ; ++r) {
            const float w = sp[key * QMAX + q0 + r];
#pragma unroll
            for (int j = 0; j < 8; ++j) acc[it][r][j] = fmaf(w, vf[j], acc[it][r][j]);
          }
        }
      }
    }
    __syncthreads();
  }

  cp_wait<0>();
  __syncthreads();
  // sum the key slices (through the tile area, free now), then store
  float* red = reinterpret_cast<float*>(sk);
  for (int half = KS / 2; half > 0; half >>= 1) {
    if (my_slice >= half && my_slice < 2 * half && my_slice < KS) {
#pragma unroll
      for (int r = 0; r < RQ; ++r) store8(red + (((size_t)(my_slice - half) * NI + tid % NI) * RQ + r) * 8, acc[0][r]);
    }
    __syncthreads();
    if (my_slice < half) {
#pragma unroll
      for (int r = 0; r < RQ; ++r) {
        float f[8];
        load8(red + (((size_t)my_slice * NI + tid % NI) * RQ + r) * 8, f);
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[0][r][j] += f[j];
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int it = 0; it < IT; ++it) {
    const int i = tid + it * THREADS;
    if (i < NI) {
      const int q0 = (i / NC) * RQ, col = i % NC;
#pragma unroll
      for (int r = 0; r < RQ; ++r) {
        float* dst = p.partial + ((((size_t)b * p.splits + split) * p.H + h0) * 2 + q0 + r) * (V + 8);
        store8(dst + col * 8, acc[it][r]);
        if (col == 0) { dst[V] = s_m[q0 + r]; dst[V + 1] = s_l[q0 + r]; }
      }
    }
  }
}

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

constexpr int MMA_WARPS = 4;

// KC: 32-dim chunks of a query / key vector, VB: 64-column blocks of a value.  heads <= 8, page size a multiple of 16.
template <int KC, int VB>
__global__ void __launch_bounds__(MMA_WARPS * 32) diff_rows_mma_kernel(DiffRowsParams<__nv_bfloat16> p) {
  extern __shared__ __align__(16) float so[];               // [warps][16][64 VB] values, then [warps][16] maxima and sums
  pdl_grid_trigger();
  const int D = p.D, V = p.V, per_g = p.H / p.G, sub = per_g / p.heads;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gr = lane >> 2, kk = lane & 3;
  const int split = blockIdx.x, b = blockIdx.z, g = blockIdx.y / sub, h0 = g * per_g + (blockIdx.y % sub) * p.heads;
  float* s_m = so + MMA_WARPS * 16 * 64 * VB;
  float* s_l = s_m + MMA_WARPS * 16;
  pdl_grid_wait();
  const uint4 zero = make_uint4(0, 0, 0, 0);
  uint4 q[2][KC];
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int c = 0; c < KC; ++c) {
      const int d = c * 32 + kk * 8;
      q[m][c] = gr < p.heads && d < D ? *reinterpret_cast<const uint4*>(p.q + (((size_t)b * p.H + h0 + gr) * 2 + m) * D + d) : zero;
    }
  const int n_keys = p.positions[b] + 1;
  const int per = ((n_keys + p.splits - 1) / p.splits + 16 * MMA_WARPS - 1) / (16 * MMA_WARPS) * (16 * MMA_WARPS);
  const int k0 = split * per, k1 = min(n_keys, k0 + per);
  const int* bt = p.block_table + (size_t)(p.seq ? p.seq[b] : b) * p.max_blocks;

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
  for (; key0 < k1; key0 += 16 * MMA_WARPS) {
    // a tile never leaves its page, and a page that holds a visible key is readable to its end
    const size_t row0 = (size_t)page * p.bs + key0 % p.bs;
    const int next = key0 + 16 * MMA_WARPS;
    page = next < k1 ? bt[next / p.bs] : 0;
    uint4 kf[2][2][KC], vf[4][VB];
#pragma unroll
    for (int nb = 0; nb < 2; ++nb) {
      const __nv_bfloat16* kr = p.k_cache + ((row0 + nb * 8 + gr) * p.G + g) * 2 * D + kk * 8;
#pragma unroll
      for (int m = 0; m < 2; ++m)
#pragma unroll
        for (int c = 0; c < KC; ++c)
          kf[nb][m][c] = c * 32 + kk * 8 < D ? *reinterpret_cast<const uint4*>(kr + m * D + c * 32) : zero;
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
        mma_bf16(s[nb], q[0][c].x, 0, q[0][c].y, 0, kf[nb][0][c].x, kf[nb][0][c].y);
        mma_bf16(s[nb], q[0][c].z, 0, q[0][c].w, 0, kf[nb][0][c].z, kf[nb][0][c].w);
        mma_bf16(s[nb], 0, q[1][c].x, 0, q[1][c].y, kf[nb][1][c].x, kf[nb][1][c].y);
        mma_bf16(s[nb], 0, q[1][c].z, 0, q[1][c].w, kf[nb][1][c].z, kf[nb][1][c].w);
      }
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int nb = 0; nb < 2; ++nb)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        s[nb][i] = key0 + nb * 8 + kk * 2 + (i & 1) < k1 ? s[nb][i] * p.scale_log2 : -INFINITY;
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
  for (int i = threadIdx.x; i < 2 * p.heads * nv; i += MMA_WARPS * 32) {
    const int r = i / nv, v = (i % nv) * 4, head = r >> 1, row = (r & 1) * 8 + head;
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < MMA_WARPS; ++w) M = fmaxf(M, s_m[w * 16 + row]);
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    float L = 0.f;
#pragma unroll
    for (int w = 0; w < MMA_WARPS; ++w) {
      const float mw = s_m[w * 16 + row], f = mw == -INFINITY ? 0.f : pow2(mw - M);
      const float4 t = *reinterpret_cast<const float4*>(so + ((size_t)(w * 16 + row)) * 64 * VB + v);
      L = fmaf(f, s_l[w * 16 + row], L);
      acc.x = fmaf(f, t.x, acc.x); acc.y = fmaf(f, t.y, acc.y); acc.z = fmaf(f, t.z, acc.z); acc.w = fmaf(f, t.w, acc.w);
    }
    float* dst = p.partial + ((((size_t)b * p.splits + split) * p.H + h0) * 2 + r) * (V + 8);
    *reinterpret_cast<float4*>(dst + v) = acc;
    if (v == 0) { dst[V] = M; dst[V + 1] = L; }
  }
}

// One block per (head, row): merge the slices of both maps, difference, norm, gate.
template <typename T>
__global__ void diff_rows_merge_kernel(const float* __restrict__ partial, T* __restrict__ out, const T* __restrict__ gate,
                                       int ld_gate, int splits, int H, int V, int ldo, DiffFinish fin) {
  extern __shared__ float s_w[];                            // [2][splits] weight of a slice in its map, lambda included
  __shared__ float red[32];
  pdl_grid_trigger();
  pdl_grid_wait();
  const int h = blockIdx.x, b = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const size_t stride = (size_t)H * 2 * (V + 8);
  const float* base = partial + ((size_t)b * splits * H + h) * 2 * (V + 8);
  if (warp < 2) {
    const float* part = base + warp * (V + 8) + V;
    float M = -INFINITY, L = 0.f;
    for (int s = lane; s < splits; s += 32) M = fmaxf(M, part[s * stride]);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, o));
    for (int s = lane; s < splits; s += 32) {
      const float m = part[s * stride], w = m == -INFINITY ? 0.f : exp2f(m - M);       // an empty slice has no maximum
      L += w * part[s * stride + 1];
      s_w[warp * splits + s] = w;
    }
    L = warp_sum_all(L);
    const float f = (warp ? -fin.lambda : 1.f) / L;
    for (int s = lane; s < splits; s += 32) s_w[warp * splits + s] *= f;
  }
  __syncthreads();
  auto value = [&](int d) {
    float v = 0.f;
#pragma unroll 4
    for (int s = 0; s < splits; ++s) v = fmaf(s_w[s], base[s * stride + d], fmaf(s_w[splits + s], base[s * stride + V + 8 + d], v));
    return v;
  };
  float keep = 0.f, ss = 0.f;
  for (int d = threadIdx.x; d < V; d += blockDim.x) {
    keep = value(d);
    ss += keep * keep;
  }
  const float f = diff_head_scale(block_sum_all(ss, red), (float)gate[(size_t)b * ld_gate + h], fin);
  T* orow = out + (size_t)b * ldo + h * V;
  if (V <= blockDim.x) {
    if (threadIdx.x < V) orow[threadIdx.x] = (T)(keep * f);
  } else {
    for (int d = threadIdx.x; d < V; d += blockDim.x) orow[d] = (T)(value(d) * f);
  }
}

template <typename T>
size_t rows_smem(int heads, int D, int V, int tk) {
  const int nq = 2 * heads;
  const size_t tiles = (size_t)2 * tk * (key_pitch<T>(D) + V * sizeof(T)), red = (size_t)THREADS / 2 * 8 * 8 * 4;
  return (size_t)(nq * D + 3 * QMAX + 128 + nq * tk + tk * QMAX) * 4 + (tiles > red ? tiles : red);
}

template <typename T, int RQ>
int launch_rows(DiffRowsParams<T> p, int rows, cudaStream_t stream) {
  const size_t small = 74 * 1024, big = 227 * 1024 - 256;
  int tk = 64;
  while (tk > 16 && rows_smem<T>(p.heads, p.D, p.V, tk) > small) tk >>= 1;
  while (tk > 8 && rows_smem<T>(p.heads, p.D, p.V, tk) > big) tk >>= 1;
  const size_t smem = rows_smem<T>(p.heads, p.D, p.V, tk);
  if (smem > big) return -6;
  const int NI = p.V / 8 * (2 * p.heads / RQ);
  p.tk = tk;
  p.ks = 1;
  while (p.ks * 2 * NI <= THREADS && p.ks * 2 <= tk) p.ks *= 2;
  const int it = (NI + THREADS - 1) / THREADS;
  const dim3 grid(p.splits, p.H / p.heads, rows), block(THREADS);
#define B200_ROWS(IT)                                                                                                      \
  {                                                                                                                        \
    static PerDeviceOnce once_;                                                                                            \
    bool& configured = once_.slot();                                                                                       \
    if (!configured) {                                                                                                     \
      const cudaError_t e = cudaFuncSetAttribute(diff_rows_kernel<T, RQ, IT>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                                 (int)big);                                                                \
      if (e != cudaSuccess) return (int)e;                                                                                 \
      configured = true;                                                                                                   \
    }                                                                                                                      \
    return (int)launch_pdl(diff_rows_kernel<T, RQ, IT>, grid, block, smem, stream, p);                                     \
  }
  if (it == 1) B200_ROWS(1)
  if (it == 2) B200_ROWS(2)
  if (it <= 4) B200_ROWS(4)
#undef B200_ROWS
  return -6;
}

template <int KC, int VB>
int launch_mma(const DiffRowsParams<__nv_bfloat16>& p, int rows, cudaStream_t stream) {
  const size_t smem = (size_t)MMA_WARPS * 16 * (64 * VB + 2) * 4;
  static PerDeviceOnce once_;
  bool& configured = once_.slot();
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(diff_rows_mma_kernel<KC, VB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  return (int)launch_pdl(diff_rows_mma_kernel<KC, VB>, dim3(p.splits, p.H / p.heads, rows), dim3(MMA_WARPS * 32), smem, stream, p);
}

// -1: sizes the tensor-core kernel does not cover
int run_mma(const DiffRowsParams<__nv_bfloat16>& p, int rows, cudaStream_t stream) {
  if (p.bs % 16 || p.D > 128 || p.V > 256 || p.heads > 8) return -1;
  const int kc = (p.D + 31) / 32, vb = (p.V + 63) / 64;
#define B200_MMA(K)                                                                  \
  case K:                                                                            \
    return vb == 1 ? launch_mma<K, 1>(p, rows, stream) : vb == 2 ? launch_mma<K, 2>(p, rows, stream) \
                                                                 : launch_mma<K, 4>(p, rows, stream);
  switch (kc) {
    B200_MMA(1) B200_MMA(2) B200_MMA(3) B200_MMA(4)
  }
#undef B200_MMA
  return -1;
}
int run_mma(const DiffRowsParams<float>&, int, cudaStream_t) { return -1; }

template <typename T>
int run_rows(const void* q, const void* k_cache, const void* v_cache, void* out, const void* gate, int ld_gate,
             const int* block_table, const int* seq, const int* positions, float* partial, int rows, int max_blocks, int bs, int H,
             int G, int D, int V, int splits, int ldo, float scale, const DiffFinish& fin, cudaStream_t stream) {
  DiffRowsParams<T> p;
  p.q = reinterpret_cast<const T*>(q); p.k_cache = reinterpret_cast<const T*>(k_cache);
  p.v_cache = reinterpret_cast<const T*>(v_cache); p.block_table = block_table; p.seq = seq; p.positions = positions;
  p.partial = partial; p.max_blocks = max_blocks; p.bs = bs; p.H = H; p.G = G; p.D = D; p.V = V; p.splits = splits;
  p.scale_log2 = scale * 1.4426950408889634f; p.tk = 0; p.ks = 1;
  p.heads = 1;
  for (int r = 2; r <= QMAX / 2; ++r)
    if ((H / G) % r == 0) p.heads = r;
  const int nq = 2 * p.heads;
  int e = run_mma(p, rows, stream);
  if (e == -1)
    e = nq % 8 == 0 ? launch_rows<T, 8>(p, rows, stream) : nq % 4 == 0 ? launch_rows<T, 4>(p, rows, stream)
                                                                       : launch_rows<T, 2>(p, rows, stream);
  if (e) return e;
  const int threads = V <= 64 ? 64 : V < 256 ? (V + 31) / 32 * 32 : 256;
  return (int)launch_pdl(diff_rows_merge_kernel<T>, dim3(H, rows), dim3(threads), (size_t)2 * splits * 4, stream, (const float*)partial,
                         reinterpret_cast<T*>(out), reinterpret_cast<const T*>(gate), ld_gate, splits, H, V, ldo, fin);
}

// Finish of rows whose difference a1 - lambda a2 was left in fp32 by the tile kernel: norm and gate.
template <typename T>
__global__ void diff_finish_kernel(const float* __restrict__ diff, T* __restrict__ out, const T* __restrict__ gate, int ld_gate,
                                   int H, int V, int ldo, DiffFinish fin) {
  __shared__ float red[32];
  pdl_grid_trigger();
  pdl_grid_wait();
  const int h = blockIdx.x, b = blockIdx.y;
  const float* src = diff + ((size_t)b * H + h) * V;
  float ss = 0.f;
  for (int d = threadIdx.x; d < V; d += blockDim.x) ss += src[d] * src[d];
  const float f = diff_head_scale(block_sum_all(ss, red), (float)gate[(size_t)b * ld_gate + h], fin);
  for (int d = threadIdx.x; d < V; d += blockDim.x) out[(size_t)b * ldo + h * V + d] = (T)(src[d] * f);
}

}  // namespace

// rows query rows; partial: fp32 [rows * splits * H * 2 * (V + 8)].  D, V, ldo multiples of 8; gate: one logit per row and
// head, rows ld_gate apart.
extern "C" int b200_attn_diff_rows(const void* q, const void* k_cache, const void* v_cache, void* out, const void* gate,
                                   int ld_gate, const int* block_table, const int* seq, const int* positions, float* partial,
                                   int rows, int max_blocks, int block_size, int H, int G, int D, int V, int vdim, int splits,
                                   int ldo, float scale, float lambda, float keep, float eps, int f32, cudaStream_t stream) {
  if (rows <= 0 || rows > 65535 || H <= 0 || G <= 0 || H % G || D <= 0 || (D & 7) || V <= 0 || (V & 7) || V > 1024 || vdim <= 0 ||
      vdim > V || (ldo & 7) || ldo < H * V || block_size <= 0 || splits < 1 || splits > 4096 || !partial || !gate)
    return -6;
  const DiffFinish fin = {lambda, keep, eps, 1.f / (float)vdim};
  return f32 ? run_rows<float>(q, k_cache, v_cache, out, gate, ld_gate, block_table, seq, positions, partial, rows, max_blocks,
                               block_size, H, G, D, V, splits, ldo, scale, fin, stream)
             : run_rows<__nv_bfloat16>(q, k_cache, v_cache, out, gate, ld_gate, block_table, seq, positions, partial, rows,
                                       max_blocks, block_size, H, G, D, V, splits, ldo, scale, fin, stream);
}

// diff [rows, H, V] fp32 -> out [rows, ldo] bf16.
extern "C" int b200_attn_diff_finish(const float* diff, void* out, const void* gate, int ld_gate, int rows, int H, int V, int vdim,
                                     int ldo, float keep, float eps, cudaStream_t stream) {
  if (rows <= 0 || rows > 65535 || H <= 0 || V <= 0 || vdim <= 0 || vdim > V || ldo < H * V) return -6;
  const DiffFinish fin = {0.f, keep, eps, 1.f / (float)vdim};
  const int threads = V < 256 ? (V + 31) / 32 * 32 : 256;
  return (int)launch_pdl(diff_finish_kernel<__nv_bfloat16>, dim3(H, rows), dim3(threads), 0, stream, diff,
                         reinterpret_cast<__nv_bfloat16*>(out), reinterpret_cast<const __nv_bfloat16*>(gate), ld_gate, H, V, ldo,
                         fin);
}
