// Latent attention of single query rows over a paged cache in the absorbed form: all heads of a row attend to the same cache
// rows [latent | rotated key part] with queries of that width, and what is summed up is the latent:
//
//   o[h] = softmax_j(scale q[h] . row(j)) latent(j)
//
// Used for decode batches and short portions that attn_latent_decode.cu does not take, and for every row in fp32.  Sizes are
// run-time values.
//
// bf16 (latent_rows_mma_kernel): a block takes one row, 16 MT heads (the M side of m16n8k16 products) and one slice of the
// row's keys.  Tiles of 32 cache rows are
// copied ahead with cp.async, once for all heads of the block.  Four warps share 16 heads: each scores 8 keys of a tile, the
// probabilities travel through shared memory, and each sums its 16-column blocks of the latent.
// fp32 and wider latents (latent_rows_kernel): CUDA cores, four heads per block, a warp per key for the dot products.
//
// Slices leave their unnormalised sums, then (maximum, sum of weights) per head; latent_rows_merge_kernel combines them.
#include <cuda_bf16.h>
#include <stdint.h>
#include "launch.h"
#include "ops.h"
#include "per_device.h"
#include "vec8.cuh"

namespace {
using namespace b200;

constexpr int KT = 32;        // keys per tile

struct Rows {
  const int* block_table;     // [sequences, max_blocks]
  const int* seq;             // [rows] table row of each query row (null: row i)
  const int* positions;       // [rows]
  int max_blocks, bs, H, C, D, splits;      // C: latent columns, D: columns of a cache row
  float scale_log2;
  float* partial;             // [rows, H, splits, C], or null: one slice
  float* stats;               // [rows, H, splits, 2] maximum, sum
};

__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], const void* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], const void* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void cp16(void* dst, const void* src, bool ok) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  const int n = ok ? 16 : 0;                                     // 0 source bytes: the 16 bytes are zero-filled
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ uint32_t pack_bf16(float a, float b) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&h);
}

// Columns of a shared-memory row: whole pairs of 16-column steps, plus 8 that skew the banks.
__host__ __device__ inline int smem_ld(int D) { return (D + 31) / 32 * 32 + 8; }

template <int MT>
__host__ __device__ inline size_t mma_smem(int D) {
  const int HG = 16 * MT;
  return (size_t)(HG + 2 * KT) * smem_ld(D) * 2 + (size_t)HG * (KT + 8) * 2 + 2 * 4 * HG * 4;
}

// grid (splits, head groups, rows), 128 MT threads.  Warp w: heads 16 (w / 4), quarter w % 4.  NB: 16-column blocks of the
// latent per warp.
template <int MT, int NB>
__global__ void __launch_bounds__(128 * MT)
latent_rows_mma_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ cache, __nv_bfloat16* __restrict__ out,
                       Rows p) {
  constexpr int HG = 16 * MT, NTHR = 128 * MT, PLD = KT + 8, TPK = NTHR / KT;
  extern __shared__ __align__(16) uint8_t smem[];
  const int D = p.D, C = p.C, LD = smem_ld(D);
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(smem);
  __nv_bfloat16* sK = sQ + HG * LD;                              // [2][KT][LD]
  __nv_bfloat16* sP = sK + 2 * KT * LD;                          // [HG][PLD]
  float* sMax = reinterpret_cast<float*>(sP + HG * PLD);         // [4][HG]
  float* sSum = sMax + 4 * HG;
  pdl_grid_trigger();
  const int tid = threadIdx.x, lane = tid & 31, g = lane >> 2, tig = lane & 3;
  const int warp = (tid >> 5) & 3, mt = tid >> 7;
  const int split = blockIdx.x, h0 = blockIdx.y * HG, b = blockIdx.z;
  const uint4 zero = make_uint4(0, 0, 0, 0);
  // columns behind a row stay zero for the odd last step
  for (int i = tid; i < 2 * KT * 2; i += NTHR)
    if (D + (i & 1) * 8 < LD - 8) *reinterpret_cast<uint4*>(sK + (i >> 1) * LD + D + (i & 1) * 8) = zero;
  pdl_grid_wait();
  const int n_keys = p.positions[b] + 1;
  const int per = ((n_keys + p.splits - 1) / p.splits + KT - 1) / KT * KT;
  const int k0 = split * per, k1 = min(n_keys, k0 + per);
  const int* bt = p.block_table + (size_t)(p.seq ? p.seq[b] : b) * p.max_blocks;
  const int j_of = tid / TPK, part_of = tid % TPK;
  auto fetch = [&](int key0, int buf) {
    const int key = key0 + j_of;
    const bool ok = key < k1;
    const __nv_bfloat16* src = cache + (ok ? ((size_t)bt[key / p.bs] * p.bs + key % p.bs) * D : 0);
    __nv_bfloat16* dst = sK + (size_t)(buf * KT + j_of) * LD;
    for (int c = part_of; c < D / 8; c += TPK) cp16(dst + c * 8, src + c * 8, ok);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (k0 < k1) fetch(k0, 0);
  for (int i = tid; i < HG * ((LD - 8) / 8); i += NTHR) {
    const int r = i / ((LD - 8) / 8), c = i % ((LD - 8) / 8) * 8;
    *reinterpret_cast<uint4*>(sQ + r * LD + c) =
        h0 + r < p.H && c < D ? *reinterpret_cast<const uint4*>(q + ((size_t)b * p.H + h0 + r) * D + c) : zero;
  }

  float o[NB][2][4];
#pragma unroll
  for (int n = 0; n < NB; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) o[n][0][i] = o[n][1][i] = 0.f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};   // heads g and g + 8
  const int pairs = (LD - 8) / 32;

  int buf = 0;
  for (int key0 = k0; key0 < k1; key0 += KT, buf ^= 1) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                   // tile landed; previous tile's readers are done
    if (key0 + KT < k1) fetch(key0 + KT, buf ^ 1);
    const __nv_bfloat16* kt = sK + (size_t)buf * KT * LD;
    float s[4] = {0.f, 0.f, 0.f, 0.f};
    {
      const __nv_bfloat16* ap = sQ + (16 * mt + (lane & 15)) * LD + (lane >> 4) * 8;
      const __nv_bfloat16* bp = kt + (8 * warp + (lane & 7)) * LD + (lane >> 3) * 8;
#pragma unroll 4
      for (int ks = 0; ks < pairs; ++ks) {
        uint32_t a0[4], a1[4], bb[4];
        ldmatrix_x4(a0, ap + ks * 32);
        ldmatrix_x4(a1, ap + ks * 32 + 16);
        ldmatrix_x4(bb, bp + ks * 32);
        mma_bf16(s, a0, bb[0], bb[1]);
        mma_bf16(s, a1, bb[2], bb[3]);
      }
    }
    {
      const int kc = key0 + 8 * warp + 2 * tig;
      const bool v0 = kc < k1, v1 = kc + 1 < k1;
      s[0] = v0 ? s[0] * p.scale_log2 : -INFINITY; s[1] = v1 ? s[1] * p.scale_log2 : -INFINITY;
      s[2] = v0 ? s[2] * p.scale_log2 : -INFINITY; s[3] = v1 ? s[3] * p.scale_log2 : -INFINITY;
      float mx0 = fmaxf(s[0], s[1]), mx1 = fmaxf(s[2], s[3]);
      mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1)); mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
      mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1)); mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
      if (tig == 0) { sMax[warp * HG + 16 * mt + g] = mx0; sMax[warp * HG + 16 * mt + g + 8] = mx1; }
    }
    __syncthreads();
    float corr[2];
    {
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int r = 16 * mt + g + 8 * hf;
        const float mx = fmaxf(fmaxf(m_run[hf], fmaxf(sMax[r], sMax[HG + r])), fmaxf(sMax[2 * HG + r], sMax[3 * HG + r]));
        corr[hf] = exp2f(m_run[hf] - mx);              // 0 for the first tile; a tile has a visible key, so mx is finite
        m_run[hf] = mx;
      }
      const float e0 = exp2f(s[0] - m_run[0]), e1 = exp2f(s[1] - m_run[0]);
      const float e2 = exp2f(s[2] - m_run[1]), e3 = exp2f(s[3] - m_run[1]);
      const int kc = 8 * warp + 2 * tig;
      *reinterpret_cast<uint32_t*>(sP + (16 * mt + g) * PLD + kc) = pack_bf16(e0, e1);
      *reinterpret_cast<uint32_t*>(sP + (16 * mt + g + 8) * PLD + kc) = pack_bf16(e2, e3);
      float sm0 = e0 + e1, sm1 = e2 + e3;
      sm0 += __shfl_xor_sync(0xffffffffu, sm0, 1); sm0 += __shfl_xor_sync(0xffffffffu, sm0, 2);
      sm1 += __shfl_xor_sync(0xffffffffu, sm1, 1); sm1 += __shfl_xor_sync(0xffffffffu, sm1, 2);
      if (tig == 0) { sSum[warp * HG + 16 * mt + g] = sm0; sSum[warp * HG + 16 * mt + g + 8] = sm1; }
    }
    __syncthreads();
    uint32_t pa[2][4];                                 // P as the A operand of two k-steps (16 keys each)
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int r = 16 * mt + g + 8 * hf;
      l_run[hf] = l_run[hf] * corr[hf] + (sSum[r] + sSum[HG + r]) + (sSum[2 * HG + r] + sSum[3 * HG + r]);
    }
    ldmatrix_x4(pa[0], sP + (16 * mt + (lane & 15)) * PLD + (lane >> 4) * 8);
    ldmatrix_x4(pa[1], sP + (16 * mt + (lane & 15)) * PLD + 16 + (lane >> 4) * 8);
    if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
#pragma unroll
      for (int n = 0; n < NB; ++n)
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          o[n][j][0] *= corr[0]; o[n][j][1] *= corr[0];
          o[n][j][2] *= corr[1]; o[n][j][3] *= corr[1];
        }
    }
#pragma unroll
    for (int ks = 0; ks < 2; ++ks) {
      const int key = 16 * ks + (lane & 7) + ((lane >> 3) & 1) * 8;
#pragma unroll
      for (int n = 0; n < NB; ++n) {
        const int col = (n * 4 + warp) * 16;
        if (col < C) {
          uint32_t bb[4];
          ldmatrix_x4_trans(bb, kt + key * LD + col + (lane >> 4) * 8);
          mma_bf16(o[n][0], pa[ks], bb[0], bb[1]);
          mma_bf16(o[n][1], pa[ks], bb[2], bb[3]);
        }
      }
    }
  }
#pragma unroll
  for (int hf = 0; hf < 2; ++hf) {
    const int h = h0 + 16 * mt + g + 8 * hf;
    if (h >= p.H) continue;
    const size_t at = ((size_t)b * p.H + h) * p.splits + split;
    float* part = p.partial ? p.partial + at * C : nullptr;
    const float inv = part ? 1.f : 1.f / l_run[hf];
    __nv_bfloat16* dst = out + ((size_t)b * p.H + h) * C;
#pragma unroll
    for (int n = 0; n < NB; ++n)
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int col = (n * 4 + warp) * 16 + j * 8 + 2 * tig;
        if (col >= C) continue;
        const float v0 = o[n][j][2 * hf] * inv, v1 = o[n][j][2 * hf + 1] * inv;
        if (part) *reinterpret_cast<float2*>(part + col) = make_float2(v0, v1);
        else *reinterpret_cast<uint32_t*>(dst + col) = pack_bf16(v0, v1);
      }
    if (part && warp == 0 && tig == 0) { p.stats[2 * at] = m_run[hf]; p.stats[2 * at + 1] = l_run[hf]; }
  }
}

constexpr int SH = 4;         // heads per block of the CUDA-core kernel
constexpr int ST = 256;

// grid (splits, ceil(H / 4), rows).  CI: latent columns per thread.
template <typename T, int CI>
__global__ void __launch_bounds__(ST) latent_rows_kernel(const T* __restrict__ q, const T* __restrict__ cache, T* __restrict__ out, Rows p) {
  extern __shared__ __align__(16) float sm[];
  pdl_grid_trigger();
  const int D = p.D, C = p.C, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  float* sq = sm;                                          // [SH][D]
  float* sp = sq + SH * D;                                 // [SH][KT] scores, then weights
  float* sa = sp + SH * KT;                                // [SH] factor on what was summed before
  float* sml = sa + SH;                                    // [2][SH] running maximum and sum
  size_t* srow = reinterpret_cast<size_t*>(sml + 2 * SH);  // [KT]
  const int split = blockIdx.x, h0 = blockIdx.y * SH, b = blockIdx.z;
  if (tid < SH) { sml[tid] = -INFINITY; sml[SH + tid] = 0.f; }
  pdl_grid_wait();
  for (int i = tid; i < SH * D; i += ST) {
    const int h = h0 + i / D;
    sq[i] = h < p.H ? (float)q[((size_t)b * p.H + h) * D + i % D] * p.scale_log2 : 0.f;
  }
  const int n_keys = p.positions[b] + 1, per = (n_keys + p.splits - 1) / p.splits;
  const int k0 = split * per, k1 = min(n_keys, k0 + per);
  const int* bt = p.block_table + (size_t)(p.seq ? p.seq[b] : b) * p.max_blocks;
  float acc[SH][CI];
#pragma unroll
  for (int h = 0; h < SH; ++h)
#pragma unroll
    for (int i = 0; i < CI; ++i) acc[h][i] = 0.f;
  for (int key0 = k0; key0 < k1; key0 += KT) {
    const int n = min(KT, k1 - key0);
    __syncthreads();
    if (tid < n) srow[tid] = ((size_t)bt[(key0 + tid) / p.bs] * p.bs + (key0 + tid) % p.bs) * D;
    __syncthreads();
    for (int j = warp; j < n; j += ST / 32) {
      const T* row = cache + srow[j];
      float d[SH] = {};
      for (int i = lane * 8; i < D; i += 256) {
        float f[8];
        load8(row + i, f);
#pragma unroll
        for (int h = 0; h < SH; ++h)
#pragma unroll
          for (int e = 0; e < 8; ++e) d[h] = fmaf(sq[h * D + i + e], f[e], d[h]);
      }
#pragma unroll
      for (int h = 0; h < SH; ++h) {
        d[h] = warp_sum_all(d[h]);
        if (lane == 0) sp[h * KT + j] = d[h];
      }
    }
    __syncthreads();
    if (warp < SH) {
      const float s = lane < n ? sp[warp * KT + lane] : -INFINITY;
      float mx = s;
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      mx = fmaxf(mx, sml[warp]);
      const float e = exp2f(s - mx), l = warp_sum_all(e);
      sp[warp * KT + lane] = e;
      __syncwarp();
      if (lane == 0) {
        const float a = exp2f(sml[warp] - mx);
        sa[warp] = a;
        sml[warp] = mx;
        sml[SH + warp] = sml[SH + warp] * a + l;
      }
    }
    __syncthreads();
#pragma unroll
    for (int h = 0; h < SH; ++h)
#pragma unroll
      for (int i = 0; i < CI; ++i) acc[h][i] *= sa[h];
    for (int j = 0; j < n; ++j) {
      const T* row = cache + srow[j];
#pragma unroll
      for (int i = 0; i < CI; ++i) {
        const int c = tid + i * ST;
        const float v = c < C ? (float)row[c] : 0.f;
#pragma unroll
        for (int h = 0; h < SH; ++h) acc[h][i] = fmaf(sp[h * KT + j], v, acc[h][i]);
      }
    }
  }
  __syncthreads();
#pragma unroll
  for (int h = 0; h < SH; ++h) {
    if (h0 + h >= p.H) continue;
    const float m = sml[h], l = sml[SH + h];
    const size_t at = ((size_t)b * p.H + h0 + h) * p.splits + split;
    float* part = p.partial ? p.partial + at * C : nullptr;
#pragma unroll
    for (int i = 0; i < CI; ++i) {
      const int c = tid + i * ST;
      if (c >= C) continue;
      if (part) part[c] = acc[h][i];
      else out[((size_t)b * p.H + h0 + h) * C + c] = (T)(acc[h][i] / l);
    }
    if (part && tid == 0) { p.stats[2 * at] = m; p.stats[2 * at + 1] = l; }
  }
}

constexpr int MW = 8;         // warps of the merge kernel: each takes every eighth slice

// grid (H, rows, ceil(C / 128)): combine the slices of one head and row, 128 columns per block.
template <typename T>
__global__ void __launch_bounds__(MW * 32)
latent_rows_merge_kernel(const float* __restrict__ partial, const float* __restrict__ stats, T* __restrict__ out, int H, int C, int splits) {
  extern __shared__ float s_w[];                           // [splits] weights, then [MW][128]
  pdl_grid_trigger();
  pdl_grid_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const size_t hr = (size_t)blockIdx.y * H + blockIdx.x;
  const float* st = stats + hr * splits * 2;
  float* s_o = s_w + (splits + 3) / 4 * 4;
  if (warp == 0) {
    float M = -INFINITY, L = 0.f;
    for (int s = lane; s < splits; s += 32) M = fmaxf(M, st[2 * s]);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, o));
    for (int s = lane; s < splits; s += 32) {
      const float m = st[2 * s], w = m == -INFINITY ? 0.f : exp2f(m - M);            // an empty slice has no maximum
      L += w * st[2 * s + 1];
      s_w[s] = w;
    }
    L = warp_sum_all(L);
    __syncwarp();
    for (int s = lane; s < splits; s += 32) s_w[s] /= L;
  }
  __syncthreads();
  const int c = blockIdx.z * 128 + lane * 4;
  float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
  if (c < C) {
    const float* base = partial + hr * splits * C + c;
#pragma unroll 4
    for (int s = warp; s < splits; s += MW) {
      const float4 f = *reinterpret_cast<const float4*>(base + (size_t)s * C);       // an empty slice left zeros
      const float w = s_w[s];
      v.x = fmaf(w, f.x, v.x); v.y = fmaf(w, f.y, v.y); v.z = fmaf(w, f.z, v.z); v.w = fmaf(w, f.w, v.w);
    }
  }
  *reinterpret_cast<float4*>(s_o + warp * 128 + lane * 4) = v;
  __syncthreads();
  const int col = blockIdx.z * 128 + threadIdx.x;
  if (threadIdx.x < 128 && col < C) {
    float a = 0.f;
#pragma unroll
    for (int w = 0; w < MW; ++w) a += s_o[w * 128 + threadIdx.x];
    out[hr * C + col] = (T)a;
  }
}

template <int MT, int NB>
int launch_mma(const void* q, const void* cache, void* out, const Rows& p, int rows, cudaStream_t stream) {
  static PerDeviceOnce once_;
  bool& configured = once_.slot();
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(latent_rows_mma_kernel<MT, NB>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  return (int)launch_pdl(latent_rows_mma_kernel<MT, NB>, dim3(p.splits, (p.H + 16 * MT - 1) / (16 * MT), rows), dim3(128 * MT),
                         mma_smem<MT>(p.D), stream, reinterpret_cast<const __nv_bfloat16*>(q),
                         reinterpret_cast<const __nv_bfloat16*>(cache), reinterpret_cast<__nv_bfloat16*>(out), p);
}

template <int MT>
int pick_mma(const void* q, const void* cache, void* out, const Rows& p, int rows, cudaStream_t stream) {
  if (p.C <= 64) return launch_mma<MT, 1>(q, cache, out, p, rows, stream);
  if (p.C <= 128) return launch_mma<MT, 2>(q, cache, out, p, rows, stream);
  if (p.C <= 256) return launch_mma<MT, 4>(q, cache, out, p, rows, stream);
  return launch_mma<MT, 8>(q, cache, out, p, rows, stream);
}

template <typename T, int CI>
int launch_simt(const void* q, const void* cache, void* out, const Rows& p, int rows, cudaStream_t stream) {
  const size_t smem = (size_t)(SH * p.D + SH * KT + 4 * SH) * 4 + KT * 8;
  if (smem > 227 * 1024) return -6;
  static PerDeviceOnce once_;
  bool& configured = once_.slot();
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(latent_rows_kernel<T, CI>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  return (int)launch_pdl(latent_rows_kernel<T, CI>, dim3(p.splits, (p.H + SH - 1) / SH, rows), dim3(ST), smem, stream,
                         reinterpret_cast<const T*>(q), reinterpret_cast<const T*>(cache), reinterpret_cast<T*>(out), p);
}

template <typename T>
int run_simt(const void* q, const void* cache, void* out, const Rows& p, int rows, cudaStream_t stream) {
  if (p.C <= ST) return launch_simt<T, 1>(q, cache, out, p, rows, stream);
  if (p.C <= 2 * ST) return launch_simt<T, 2>(q, cache, out, p, rows, stream);
  if (p.C <= 4 * ST) return launch_simt<T, 4>(q, cache, out, p, rows, stream);
  if (p.C <= 8 * ST) return launch_simt<T, 8>(q, cache, out, p, rows, stream);
  return -6;
}

template <typename T>
int merge(const Rows& p, void* out, int rows, cudaStream_t stream) {
  return (int)launch_pdl(latent_rows_merge_kernel<T>, dim3(p.H, rows, (p.C + 127) / 128), dim3(MW * 32),
                         (size_t)((p.splits + 3) / 4 * 4 + MW * 128) * 4, stream, (const float*)p.partial, (const float*)p.stats,
                         reinterpret_cast<T*>(out), p.H, p.C, p.splits);
}

}  // namespace

// Heads a block shares a key tile among (the split count is chosen for it).
extern "C" int b200_attn_latent_rows_heads(int H, int C, int D, int rows, int f32) {
  if (f32 || C > 512) return SH;
  if (H > 32 && mma_smem<4>(D) <= 227 * 1024 && (long long)rows * ((H + 63) / 64) >= 148) return 64;
  if (H > 16 && mma_smem<2>(D) <= 227 * 1024 && (long long)rows * ((H + 31) / 32) >= 74) return 32;
  return 16;
}

// q [rows, H, D], cache [pages * bs, D], out [rows, H, C]; C, D multiples of 16, C <= 2048; partial: fp32
// [rows * H * splits * (C + 2)] when splits > 1.
extern "C" int b200_attn_latent_rows(const void* q, const void* cache, void* out, const int* block_table, const int* seq,
                                     const int* positions, float* partial, int rows, int max_blocks, int bs, int H, int C, int D,
                                     int splits, float scale, int f32, cudaStream_t stream) {
  if (rows <= 0 || rows > 65535 || H <= 0 || C <= 0 || D < C || (C & 15) || (D & 15) || splits <= 0 || (splits > 1 && !partial) || bs <= 0)
    return -6;
  Rows p;
  p.block_table = block_table; p.seq = seq; p.positions = positions; p.max_blocks = max_blocks; p.bs = bs; p.H = H; p.C = C; p.D = D;
  p.splits = splits; p.scale_log2 = scale * 1.4426950408889634f; p.partial = splits > 1 ? partial : nullptr;
  p.stats = partial + (size_t)rows * H * splits * C;
  int rc;
  const int heads = b200_attn_latent_rows_heads(H, C, D, rows, f32);
  if (f32) rc = run_simt<float>(q, cache, out, p, rows, stream);
  else if (heads == SH || mma_smem<1>(D) > 227 * 1024) rc = run_simt<__nv_bfloat16>(q, cache, out, p, rows, stream);
  else if (heads == 64) rc = pick_mma<4>(q, cache, out, p, rows, stream);
  else if (heads == 32) rc = pick_mma<2>(q, cache, out, p, rows, stream);
  else rc = pick_mma<1>(q, cache, out, p, rows, stream);
  if (rc || splits == 1) return rc;
  return f32 ? merge<float>(p, out, rows, stream) : merge<__nv_bfloat16>(p, out, rows, stream);
}

// The merge on its own: partial as above (sums, then maxima and weights), out [rows, H, C].
extern "C" int b200_attn_latent_merge(const float* partial, void* out, int rows, int H, int C, int splits, int f32, cudaStream_t stream) {
  if (rows <= 0 || rows > 65535 || H <= 0 || C <= 0 || (C & 15) || splits <= 1 || !partial) return -6;
  Rows p = {};
  p.H = H; p.C = C; p.splits = splits;
  p.partial = const_cast<float*>(partial);
  p.stats = p.partial + (size_t)rows * H * splits * C;
  return f32 ? merge<float>(p, out, rows, stream) : merge<__nv_bfloat16>(p, out, rows, stream);
}
