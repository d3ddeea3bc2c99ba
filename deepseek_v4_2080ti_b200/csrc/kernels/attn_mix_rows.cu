// Attention of single query rows over a paged KV cache, with the scores of all heads mixed before the softmax:
//
//   s_h(j)  = scale * sum_g talk[h, g] (q_g . k_{kv(g)}(j)),   softmax over the visible j,   o_h = sum_j p_h(j) v_{kv(h)}(j)
//
// A row at position p sees the keys of its own chunk, [p - p % chunk, p] (chunk 0: every key up to p).  One block owns
// one row and one slice of its keys, for ALL heads (the mixing needs them together): key and value tiles of TK tokens
// are staged in shared memory once and serve every head.  Per tile: per-head dot products (one lane per key, RT query
// heads of one key head per thread), mixing + online softmax (one lane per key, four heads per thread, shuffles over
// the keys), then P V with the accumulators in registers, one (key head, 8 values) column per thread.  Slices are
// merged by a second small kernel.  Used for decode batches in bf16 and for every row when the engine runs in fp32.
#include "launch.h"
#include "ops.h"
#include "per_device.h"
#include "vec8.cuh"

namespace {
using namespace b200;

constexpr int THREADS = 256;

template <typename T>
struct RowsParams {
  const float* q;            // [rows, H, D]
  const T *k_cache, *v_cache;// [pages * bs, G * D]
  T* out;                    // [rows out, ldo]
  const float* talk_t;       // [H (g), H4 (h)]
  const int* block_table;    // [sequences, max_blocks]
  const int* seq;            // [rows] table row of each query row (null: row i)
  const int* positions;      // [rows]
  float* partial;            // [rows, splits, H, D + 2]
  int max_blocks, bs, H, G, D, chunk, splits, ldo, tk, slices;
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

__host__ __device__ inline int pitch_bytes(int G, int D, int elem) { return G * D * elem + 16; }

template <typename T, int RT, int IT>
__global__ void __launch_bounds__(THREADS) mix_rows_kernel(RowsParams<T> p) {
  extern __shared__ __align__(16) uint8_t smem[];
  pdl_grid_trigger();
  const int H = p.H, D = p.D, KW = p.G * p.D, TK = p.tk, H4 = (H + 3) & ~3, R = H / p.G;
  const int pitch = pitch_bytes(p.G, D, sizeof(T));
  float* sq = reinterpret_cast<float*>(smem);              // [H * D]
  float* st = sq + H * D;                                  // [H, H4]
  float* s_m = st + H * H4;                                // [H4] running maximum, sum, rescale of this tile
  float* s_l = s_m + H4;
  float* s_a = s_l + H4;
  int* srow = reinterpret_cast<int*>(s_a + H4);            // [32] cache row of every key of the tile (-1: past the slice)
  float* ss = reinterpret_cast<float*>(srow + 32);         // [H4, TK] raw scores
  float* sp = ss + H4 * TK;                                // [H4, TK] weights
  uint8_t* sk = reinterpret_cast<uint8_t*>(sp + H4 * TK);  // [TK, pitch]
  uint8_t* sv = sk + (size_t)TK * pitch;
  const int tid = threadIdx.x, split = blockIdx.x, b = blockIdx.y;

  for (int i = tid; i < H * H4 / 4; i += THREADS)
    reinterpret_cast<float4*>(st)[i] = __ldg(reinterpret_cast<const float4*>(p.talk_t) + i);
  for (int i = tid; i < H4; i += THREADS) { s_m[i] = -INFINITY; s_l[i] = 0.f; s_a[i] = 0.f; }
  pdl_grid_wait();
  for (int i = tid; i < H * D / 4; i += THREADS)
    reinterpret_cast<float4*>(sq)[i] = reinterpret_cast<const float4*>(p.q + (size_t)b * H * D)[i];

  const int pos = p.positions[b];
  const int lo = p.chunk > 0 ? pos - pos % p.chunk : 0;
  const int per = (pos + 1 - lo + p.splits - 1) / p.splits;
  const int k0 = lo + split * per, k1 = min(pos + 1, k0 + per);
  const int* bt = p.block_table + (size_t)(p.seq ? p.seq[b] : b) * p.max_blocks;

  const int row_vecs = KW * (int)sizeof(T) / 16, warp = tid >> 5, lane = tid & 31;
  auto locate = [&](int key0) {
    if (tid < TK) {
      const int key = key0 + tid;
      srow[tid] = key < k1 ? bt[key / p.bs] * p.bs + key % p.bs : -1;
    }
  };
  auto stage = [&](uint8_t* dst, const T* cache) {
    for (int r = warp; r < TK; r += THREADS / 32) {
      const int slot = srow[r];
      const uint8_t* src = reinterpret_cast<const uint8_t*>(cache + (size_t)max(slot, 0) * KW);
      for (int c = lane; c < row_vecs; c += 32) cp16(dst + (size_t)r * pitch + c * 16, src + c * 16, slot >= 0);
    }
    cp_commit();
  };

  // P V ownership: column i = (head group hg, 8-value vector v of its key head), key slice ks
  const int HG = H / RT, DV = D / 8, NI = HG * DV;
  float acc[IT][RT][8];
#pragma unroll
  for (int it = 0; it < IT; ++it)
#pragma unroll
    for (int r = 0; r < RT; ++r)
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[it][r][j] = 0.f;
  const int KS = p.slices, per_slice = TK / KS;
  // with KS > 1 every column has a thread in this pass (NI * KS <= THREADS)
  const int my_slice = KS > 1 ? tid / NI : 0;

  locate(k0);
  __syncthreads();
  for (int key0 = k0; key0 < k1; key0 += TK) {
    stage(sk, p.k_cache);
    stage(sv, p.v_cache);
    cp_wait<1>();
    __syncthreads();
    for (int i = tid; i < TK * HG; i += THREADS) {
      const int key = i % TK, h0 = (i / TK) * RT, c = h0 / R;
      const T* kr = reinterpret_cast<const T*>(sk + (size_t)key * pitch) + c * D;
      float dot[RT];
#pragma unroll
      for (int r = 0; r < RT; ++r) dot[r] = 0.f;
      for (int d = 0; d < D; d += 8) {
        float kf[8];
        load8(kr + d, kf);
#pragma unroll
        for (int r = 0; r < RT; ++r) {
          float qf[8];
          load8(sq + (h0 + r) * D + d, qf);
#pragma unroll
          for (int j = 0; j < 8; ++j) dot[r] = fmaf(qf[j], kf[j], dot[r]);
        }
      }
#pragma unroll
      for (int r = 0; r < RT; ++r) ss[(h0 + r) * TK + key] = dot[r] * p.scale_log2;
    }
    __syncthreads();
    // a group of TK neighbouring lanes holds the keys of one set of four heads (TK is a power of two <= 32)
    const int n_mix = TK * (H4 / 4);
    for (int base = 0; base < n_mix; base += THREADS) {
      const int i = base + tid;
      const bool on = i < n_mix;
      const int key = i % TK, h0 = on ? (i / TK) * 4 : 0;
      float x[4] = {0.f, 0.f, 0.f, 0.f};
      if (on) {
        for (int g = 0; g < H; ++g) {
          const float s = ss[g * TK + key];
          const float4 w = *reinterpret_cast<const float4*>(st + g * H4 + h0);
          x[0] = fmaf(w.x, s, x[0]); x[1] = fmaf(w.y, s, x[1]);
          x[2] = fmaf(w.z, s, x[2]); x[3] = fmaf(w.w, s, x[3]);
        }
      }
      const bool seen = on && key0 + key < k1;
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const float s = seen ? x[u] : -INFINITY;
        float mx = s;
        for (int o = TK / 2; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        const float m_old = s_m[h0 + u], m_new = fmaxf(m_old, mx);
        const float e = seen ? exp2f(s - m_new) : 0.f;
        float l = e;
        for (int o = TK / 2; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
        __syncwarp();
        if (on) {
          sp[(h0 + u) * TK + key] = e;
          if (key == 0) {
            const float a = m_old == -INFINITY ? 0.f : exp2f(m_old - m_new);
            s_m[h0 + u] = m_new;
            s_a[h0 + u] = a;
            s_l[h0 + u] = s_l[h0 + u] * a + l;
          }
        }
      }
    }
    cp_wait<0>();
    __syncthreads();
#pragma unroll
    for (int it = 0; it < IT; ++it) {
      const int i = KS > 1 ? tid % NI : tid + it * THREADS;
      if (i < NI && my_slice < KS) {
        const int h0 = (i / DV) * RT, c = h0 / R, v = i % DV;
        float a[RT];
#pragma unroll
        for (int r = 0; r < RT; ++r) a[r] = s_a[h0 + r];
#pragma unroll
        for (int r = 0; r < RT; ++r)
#pragma unroll
          for (int j = 0; j < 8; ++j) acc[it][r][j] *= a[r];
        const uint8_t* base = sv + (size_t)(c * D + v * 8) * sizeof(T);
        const int e0 = my_slice * per_slice, e1 = e0 + per_slice;
        auto add = [&](int key, const float (&w)[RT]) {
          float vf[8];
          load8(reinterpret_cast<const T*>(base + (size_t)key * pitch), vf);
#pragma unroll
          for (int r = 0; r < RT; ++r)
#pragma unroll
            for (int j = 0; j < 8; ++j) acc[it][r][j] = fmaf(w[r], vf[j], acc[it][r][j]);
        };
        if (per_slice >= 4) {
          for (int key = e0; key < e1; key += 4) {
            float4 w4[RT];
#pragma unroll
            for (int r = 0; r < RT; ++r) w4[r] = *reinterpret_cast<const float4*>(sp + (h0 + r) * TK + key);
            float w[RT];
#pragma unroll
            for (int r = 0; r < RT; ++r) w[r] = w4[r].x;
            add(key, w);
#pragma unroll
            for (int r = 0; r < RT; ++r) w[r] = w4[r].y;
            add(key + 1, w);
#pragma unroll
            for (int r = 0; r < RT; ++r) w[r] = w4[r].z;
            add(key + 2, w);
#pragma unroll
            for (int r = 0; r < RT; ++r) w[r] = w4[r].w;
            add(key + 3, w);
          }
        } else {
          for (int key = e0; key < e1; ++key) {
            float w[RT];
#pragma unroll
            for (int r = 0; r < RT; ++r) w[r] = sp[(h0 + r) * TK + key];
            add(key, w);
          }
        }
      }
    }
    locate(key0 + TK);
    __syncthreads();
  }

  // sum the key slices (through the score and tile area, free now), then store
  float* red = ss;
  for (int s = 1; s < KS; ++s) {
    if (my_slice == s) {
#pragma unroll
      for (int r = 0; r < RT; ++r) store8(red + ((size_t)(tid % NI) * RT + r) * 8, acc[0][r]);
    }
    __syncthreads();
    if (tid < NI) {
#pragma unroll
      for (int r = 0; r < RT; ++r) {
        float f[8];
        load8(red + ((size_t)tid * RT + r) * 8, f);
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
      const int h0 = (i / DV) * RT, v = i % DV;
#pragma unroll
      for (int r = 0; r < RT; ++r) {
        const int h = h0 + r;
        if (p.splits == 1) {
          const float inv = 1.f / s_l[h];
#pragma unroll
          for (int j = 0; j < 8; ++j) acc[it][r][j] *= inv;
          store8(p.out + (size_t)b * p.ldo + h * D + v * 8, acc[it][r]);
        } else {
          float* dst = p.partial + (((size_t)b * p.splits + split) * H + h) * (D + 8);
          store8(dst + v * 8, acc[it][r]);
          if (v == 0) { dst[D] = s_m[h]; dst[D + 1] = s_l[h]; }
        }
      }
    }
  }
}

template <typename T>
__global__ void mix_rows_merge_kernel(const float* __restrict__ partial, T* __restrict__ out, int splits, int H, int D, int ldo) {
  pdl_grid_trigger();
  pdl_grid_wait();
  const int h = blockIdx.x, b = blockIdx.y;
  const size_t stride = (size_t)H * (D + 8);
  const float* base = partial + ((size_t)b * splits * H + h) * (D + 8);
  float M = -INFINITY;
  for (int s = 0; s < splits; ++s) M = fmaxf(M, base[s * stride + D]);
  for (int d = threadIdx.x; d < D; d += blockDim.x) {
    float L = 0.f, O = 0.f;
    for (int s = 0; s < splits; ++s) {
      const float m = base[s * stride + D];
      if (m == -INFINITY) continue;                       // an empty slice
      const float w = exp2f(m - M);
      L += base[s * stride + D + 1] * w;
      O += base[s * stride + d] * w;
    }
    out[(size_t)b * ldo + h * D + d] = (T)(O / L);
  }
}

template <typename T>
size_t rows_smem(int H, int G, int D, int tk, int rt) {
  const int H4 = (H + 3) & ~3;
  const size_t head = (size_t)(H * D + H * H4 + 3 * H4 + 32) * 4;
  size_t rest = (size_t)(2 * H4 * tk) * 4 + 2 * (size_t)tk * pitch_bytes(G, D, sizeof(T));
  const size_t red = (size_t)THREADS * rt * 8 * 4;                    // the slice reduction reuses everything from `ss` on
  if (rest < red) rest = red;
  return head + rest;
}

template <typename T, int RT>
int launch_rows(RowsParams<T> p, int rows, cudaStream_t stream) {
  const size_t small = 110 * 1024, big = 227 * 1024 - 256;
  int tk = 32;
  while (tk > 8 && rows_smem<T>(p.H, p.G, p.D, tk, RT) > small) tk >>= 1;
  while (tk > 1 && rows_smem<T>(p.H, p.G, p.D, tk, RT) > big) tk >>= 1;
  const size_t smem = rows_smem<T>(p.H, p.G, p.D, tk, RT);
  if (smem > big) return -6;
  const int NI = p.H / RT * (p.D / 8);
  p.tk = tk;
  p.slices = 1;
  while (p.slices * 2 * NI <= THREADS && p.slices * 2 <= tk) p.slices *= 2;
  const int it = (NI + THREADS - 1) / THREADS;
  const dim3 grid(p.splits, rows), block(THREADS);
#define B200_ROWS(IT)                                                                                                     \
  {                                                                                                                       \
    static PerDeviceOnce once_;                                                                                           \
    bool& configured = once_.slot();                                                                                      \
    if (!configured) {                                                                                                    \
      const cudaError_t e = cudaFuncSetAttribute(mix_rows_kernel<T, RT, IT>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                                 (int)big);                                                               \
      if (e != cudaSuccess) return (int)e;                                                                                \
      configured = true;                                                                                                  \
    }                                                                                                                     \
    const cudaError_t e = launch_pdl(mix_rows_kernel<T, RT, IT>, grid, block, smem, stream, p);                          \
    if (e != cudaSuccess) return (int)e;                                                                                  \
  }
  if (it == 1) B200_ROWS(1)
  else if (it == 2) B200_ROWS(2)
  else if (it <= 4) B200_ROWS(4)
  else return -6;
#undef B200_ROWS
  if (p.splits > 1)
    return (int)launch_pdl(mix_rows_merge_kernel<T>, dim3(p.H, rows), dim3(p.D < 256 ? (p.D + 31) / 32 * 32 : 256), 0, stream,
                           (const float*)p.partial, p.out, p.splits, p.H, p.D, p.ldo);
  return 0;
}

template <typename T>
int run_rows(const float* q, const void* k_cache, const void* v_cache, void* out, const float* talk_t, const int* block_table,
             const int* seq, const int* positions, float* partial, int rows, int max_blocks, int bs, int H, int G, int D,
             int chunk, int splits, int ldo, float scale, cudaStream_t stream) {
  RowsParams<T> p;
  p.q = q; p.k_cache = reinterpret_cast<const T*>(k_cache); p.v_cache = reinterpret_cast<const T*>(v_cache);
  p.out = reinterpret_cast<T*>(out); p.talk_t = talk_t; p.block_table = block_table; p.seq = seq; p.positions = positions;
  p.partial = partial; p.max_blocks = max_blocks; p.bs = bs; p.H = H; p.G = G; p.D = D; p.chunk = chunk; p.splits = splits;
  p.ldo = ldo; p.scale_log2 = scale * 1.4426950408889634f; p.tk = 0; p.slices = 1;
  const int R = H / G;
  if (R % 4 == 0) return launch_rows<T, 4>(p, rows, stream);
  if (R % 2 == 0) return launch_rows<T, 2>(p, rows, stream);
  return launch_rows<T, 1>(p, rows, stream);
}

}  // namespace

// rows query rows; partial: fp32 [rows * splits * H * (D + 8)] when splits > 1.  D % 8 == 0, ldo % 8 == 0.
extern "C" int b200_attn_mix_rows(const float* q, const void* k_cache, const void* v_cache, void* out, const float* talk_t,
                                  const int* block_table, const int* seq, const int* positions, float* partial, int rows,
                                  int max_blocks, int block_size, int H, int G, int D, int chunk, int splits, int ldo,
                                  float scale, int f32, cudaStream_t stream) {
  if (rows <= 0 || rows > 65535 || H <= 0 || G <= 0 || H % G || D <= 0 || (D & 7) || (ldo & 7) || ldo < H * D ||
      block_size <= 0 || splits < 1 || (splits > 1 && !partial) || chunk < 0)
    return -6;
  return f32 ? run_rows<float>(q, k_cache, v_cache, out, talk_t, block_table, seq, positions, partial, rows, max_blocks,
                               block_size, H, G, D, chunk, splits, ldo, scale, stream)
             : run_rows<__nv_bfloat16>(q, k_cache, v_cache, out, talk_t, block_table, seq, positions, partial, rows,
                                       max_blocks, block_size, H, G, D, chunk, splits, ldo, scale, stream);
}
