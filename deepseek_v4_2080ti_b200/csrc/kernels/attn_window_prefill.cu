// Flash-attention prefill over a paged KV cache with a sliding window and a bias per head and distance, sm_100a:
//
//   s(p, j) = scale q(p) . k(j) + bias[h, p - j],   p - size < j <= p
//
// One CTA = 256 query rows of one head as two streams of 128 that share the key and value slabs both of them see; the streams
// keep the tensor core and the exponential units busy in turn.  Each stream visits only the key tiles its own rows see.  Warp
// roles:
//   warps 0-3, 4-7: softmax of stream 0 and 1 - one query row per thread, online maximum / sum in the exp2 domain, P as bf16
//             back into the tensor memory its scores came from, lazy rescale of the stream's O;
//   warp 8  : TMA producer.  Keys and values travel as slabs of [128 tokens x 64 columns] through one ring, page by page
//             through the sequence's block table (pages outside the context or in front of the window read page 0, which holds
//             zeros);
//   warp 9  : tcgen05.mma issuer - per tile P0 V, S0 of the next tile, P1 V, S1 of the next tile.
// The biases of a tile depend on the distance only: every warp lays out the 159 its rows need in shared memory, -infinity where
// a distance is outside the window, so that the addition is the mask as well.  Four copies, each shifted by one value, let every
// lane read its row's run of 128 in aligned vectors.
// Tensor memory: S0 | S1 (128 columns each) and O0 | O1 (up to 128 columns each).  Wider values are cut into column slices,
// one CTA each.  A slab reads on past its head's columns; the products stop at them.  The two value slabs of a tile have to be
// neighbours in the ring: where they would wrap, a stage is left out (handed through empty).
// All mbarrier waits are bounded and unwind through the common exit.
#include <cuda_bf16.h>
#include "per_device.h"
#include "../ptx/sm100.cuh"
#include "tma_host.h"
#include "ops.h"

namespace b200 {
namespace windowattn {

constexpr int BQ = 128;         // query rows per stream
constexpr int BKV = 128;        // keys per tile
constexpr int ATOM = 16384;     // bytes of one [128 x 64] bf16 swizzled slab
constexpr int NTHREADS = 384;   // three warpgroups; the third has the two issuing roles and gives its registers up
constexpr int MAX_STAGES = 12;
constexpr int BIAS_COPY = 168;  // floats between the shifted copies of a warp's biases: 8 banks apart
constexpr int BIAS_BYTES = 8 * 4 * BIAS_COPY * 4;
constexpr int BUDGET = 232448 - 1024 /* alignment */ - 512 /* barriers */ - BIAS_BYTES;

struct Params {
  const int* block_table;  // [sequences, max_blocks]
  const int* seq;          // [B] table row of each entry, or null (entry i -> row i)
  const int* q_start;      // [B] first query row of the entry
  const int* q_len;        // [B]
  const int* kv_len;       // [B] context length including the entry's own tokens
  const float* bias;       // [H, size], in units of the exponent's base 2
  int max_blocks, block_size;
  int H, G, D, V;          // columns per key and value head (multiples of 16)
  int size;
  int slabs, stages, slice, v_slices;
  float scale_log2;
  __nv_bfloat16* out;      // [rows, ldo], head h at columns h * V
  int ldo;
  int* status;
};

// MN-major operand, 128-byte swizzle: 64-element MN atoms LBO bytes apart, 8-row K groups SBO bytes apart.
__device__ __forceinline__ uint64_t desc_mn_sw128(const void* p, uint32_t lbo, uint32_t sbo) {
  uint64_t d = 0;
  d |= (uint64_t)((smem_u32(p) & 0x3FFFF) >> 4);
  d |= (uint64_t)(lbo >> 4) << 16;
  d |= (uint64_t)(sbo >> 4) << 32;
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;
  return d;
}

struct Ring {
  int st;
  uint32_t ph;
  __device__ __forceinline__ void next(int stages) {
    if (++st == stages) { st = 0; ph ^= 1; }
  }
};

// VN: columns of a value slice rounded up to 32 (the accumulator's width in tensor memory and of the products).  SL: key slabs
// where the last has no ragged end (loops the issuer has unrolled), or 0.
template <int VN, int SL>
__global__ void __launch_bounds__(NTHREADS, 1)
window_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                      const __grid_constant__ CUtensorMap tmV, Params p) {
  constexpr uint32_t idesc_qk = umma_idesc_bf16(128, 128);
  constexpr uint32_t idesc_pv = umma_idesc_bf16(128, VN) | (1u << 16);   // B is MN-major
  constexpr int VS = (VN + 63) / 64;                                     // slabs of the value slice
  extern __shared__ uint8_t smem_base[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_base) + 1023) & ~uintptr_t(1023));
  const int slabs = SL ? SL : p.slabs, stages = p.stages;
  uint8_t* sQ = smem;                                   // [2 streams][slabs] atoms
  uint8_t* sR = sQ + 2 * slabs * ATOM;                  // ring of slabs
  float* sB = reinterpret_cast<float*>(sR + stages * ATOM);              // [8 warps][4 copies] biases
  uint64_t* bars = reinterpret_cast<uint64_t*>(sB + BIAS_BYTES / 4);
  uint64_t* r_full = bars;                   // MAX_STAGES
  uint64_t* r_empty = bars + MAX_STAGES;     // MAX_STAGES
  uint64_t* q_full = bars + 2 * MAX_STAGES;
  uint64_t* s_full = q_full + 1;             // per stream
  uint64_t* p_full = q_full + 3;
  uint64_t* pv_done = q_full + 5;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(q_full + 7);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0), lane = threadIdx.x & 31;   // uniform: the issuer depends on it
  const int b = blockIdx.z, h = blockIdx.y / p.v_slices, v0 = (blockIdx.y % p.v_slices) * p.slice;
  const int q_len = p.q_len[b], kv_len = p.kv_len[b];
  const int q0 = blockIdx.x * 2 * BQ;
  if (q0 >= q_len) return;                   // uniform per CTA, before any barrier / TMEM use
  const int q_row0 = p.q_start[b] + q0, g = h / (p.H / p.G);
  const int pos0 = kv_len - q_len + q0;      // position of the first query row
  const bool two = q0 + BQ < q_len;          // the second stream has rows
  // tiles [first, end) a stream's rows see; the second stream's begin and end no earlier, and there is none between them
  const int first0 = __shfl_sync(0xffffffffu, max(0, pos0 - p.size + 1) / BKV, 0);
  const int end0 = __shfl_sync(0xffffffffu, (min(kv_len, pos0 + BQ) + BKV - 1) / BKV, 0);
  const int first1 = __shfl_sync(0xffffffffu, two ? max(0, pos0 + BQ - p.size + 1) / BKV : end0, 0);
  const int end1 = __shfl_sync(0xffffffffu, two ? (min(kv_len, pos0 + 2 * BQ) + BKV - 1) / BKV : end0, 0);

  if (threadIdx.x == 0) {
    for (int i = 0; i < stages; ++i) {
      mbar_init(&r_full[i], 1);
      mbar_init(&r_empty[i], 1);
    }
    mbar_init(q_full, 1);
    for (int m = 0; m < 2; ++m) {
      mbar_init(&s_full[m], 1);
      mbar_init(&p_full[m], 128);
      mbar_init(&pv_done[m], 1);
    }
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 9) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = __shfl_sync(0xffffffffu, *tmem_slot, 0);

  // registers per thread at launch: 168 (3 x 168 = 2 x 216 + 72)
  if (warp >= 8) {
    asm volatile("setmaxnreg.dec.sync.aligned.u32 72;");
    if (warp == 8 && lane == 0) {
      tma_prefetch_desc(&tmQ);
      tma_prefetch_desc(&tmK);
      tma_prefetch_desc(&tmV);
      const int streams = two ? 2 : 1;
      mbar_expect_tx(q_full, streams * slabs * ATOM);
      for (int m = 0; m < streams; ++m)
        for (int s = 0; s < slabs; ++s) tma_load_2d(sQ + (m * slabs + s) * ATOM, &tmQ, q_full, h * p.D + s * 64, q_row0 + m * BQ);
      const int* bt = p.block_table + (size_t)(p.seq ? p.seq[b] : b) * p.max_blocks;
      const int bs = p.block_size, pages = BKV / bs, last_page = (kv_len - 1) / bs;
      const uint32_t sub_bytes = bs * 128;   // 64 columns of one page
      Ring r = {0, 1};
      bool ok = true;
      for (int j = first0; ok && j < end1 && !*abort_flag; ++j) {
        int rows[BKV / 16];
#pragma unroll
        for (int i = 0; i < BKV / 16; ++i) {
          const int page = j * pages + i;
          rows[i] = i < pages && page <= last_page ? bt[page] * bs : 0;
        }
        auto slab = [&](const CUtensorMap* tm, int x) {
          if (!mbar_wait(&r_empty[r.st], r.ph)) return false;
          uint8_t* dst = sR + r.st * ATOM;
          mbar_expect_tx(&r_full[r.st], ATOM);
#pragma unroll
          for (int i = 0; i < BKV / 16; ++i)
            if (i < pages) tma_load_2d(dst + i * sub_bytes, tm, &r_full[r.st], x, rows[i]);
          r.next(stages);
          return true;
        };
        for (int s = 0; ok && s < slabs; ++s) ok = slab(&tmK, g * p.D + s * 64);
        if (ok && VS == 2 && r.st == stages - 1) {
          ok = mbar_wait(&r_empty[r.st], r.ph);
          if (ok) mbar_arrive(&r_full[r.st]);
          r.next(stages);
        }
#pragma unroll
        for (int s = 0; s < VS; ++s)
          if (ok) ok = slab(&tmV, g * p.V + v0 + s * 64);
      }
      if (!ok) { atomicExch(p.status, ERR_WAIT_STAGE); *abort_flag = 1; }
    } else if (warp == 9) {
      // The whole warp walks the loop, so that addresses and descriptors stay warp-uniform, and one elected lane issues.
      bool ok = true;
      const uint32_t on = elect_one();
      auto wait = [&](uint64_t* bar, uint32_t parity) {
        ok = __all_sync(0xffffffffu, mbar_wait(bar, parity));
        return ok;
      };
      auto sees = [&](int m, int j) { return m ? j >= first1 && j < end1 : j >= first0 && j < end0; };
      wait(q_full, 0);
      const uint64_t ring = umma_desc_sw128(sR), dq0 = umma_desc_sw128(sQ);
      const int last_steps = (p.D - (slabs - 1) * 64) / 16;
      // scores of a tile whose key slabs begin at ring position r (by value: both streams walk the same slabs); the tile's
      // last stream gives them back
      auto issue_s = [&](const int m, Ring r, bool last) {
#pragma unroll
        for (int s = 0; s < (SL ? SL : slabs); ++s) {
          if (!wait(&r_full[r.st], r.ph)) return;
          tc_fence_after();
          const uint64_t dk = ring + r.st * (ATOM >> 4), dq = dq0 + (m * slabs + s) * (ATOM >> 4);
          const int steps = SL || s + 1 < slabs ? 4 : last_steps;
          umma_bf16_ss_warp(on, tmem + m * 128, dq, dk, idesc_qk, s ? 1u : 0u);
#pragma unroll
          for (int kk = 1; kk < 4; ++kk)
            if (kk < steps) umma_bf16_ss_warp(on, tmem + m * 128, dq + 2 * kk, dk + 2 * kk, idesc_qk, 1u);
          if (last) umma_commit_warp(on, &r_empty[r.st]);
          if (s + 1 == slabs) umma_commit_warp(on, &s_full[m]);
          r.next(stages);
        }
      };
      Ring k = {0, 0};                       // key slabs of the tile whose scores come next
      if (ok) issue_s(0, k, !sees(1, first0));
      if (ok && sees(1, first0)) issue_s(1, k, true);
      for (int j = first0; ok && j < end1 && !*abort_flag; ++j) {
        Ring v = k;                          // value slabs of tile j lie behind its keys
        for (int s = 0; s < slabs; ++s) v.next(stages);
        if (VS == 2 && v.st == stages - 1) { // the stage that was left out
          if (!wait(&r_full[v.st], v.ph)) break;
          if (on) mbar_arrive(&r_empty[v.st]);
          v.next(stages);
        }
        k = v;
        for (int s = 0; s < VS; ++s) k.next(stages);
#pragma unroll
        for (int m = 0; m < 2; ++m) {
          if (sees(m, j)) {
            const int n = j - (m ? first1 : first0);           // the stream's tile
            if (!ok || !wait(&p_full[m], n & 1)) break;
            Ring w = v;
#pragma unroll
            for (int s = 0; s < VS; ++s) {
              if (ok) wait(&r_full[w.st], w.ph);
              w.next(stages);
            }
            if (!ok) break;
            tc_fence_after();
            const uint64_t dv = desc_mn_sw128(sR, ATOM, 1024) + v.st * (ATOM >> 4);
            umma_bf16_ts_warp(on, tmem + 256 + m * 128, tmem + m * 128, dv, idesc_pv, n ? 1u : 0u);
#pragma unroll
            for (int kk = 1; kk < 8; ++kk)
              umma_bf16_ts_warp(on, tmem + 256 + m * 128, tmem + m * 128 + kk * 8, dv + kk * 128, idesc_pv, 1u);
            umma_commit_warp(on, &pv_done[m]);
            if (m == 1 || !sees(1, j)) {
#pragma unroll
              for (int s = 0; s < VS; ++s) umma_commit_warp(on, &r_empty[v.st + s]);
            }
          }
          if (ok && j + 1 < end1 && sees(m, j + 1)) issue_s(m, k, m == 1 || !sees(1, j + 1));
        }
      }
      if (!ok && lane == 0) { atomicExch(p.status, ERR_WAIT_TMA); *abort_flag = 1; }
    }
  } else {
    asm volatile("setmaxnreg.inc.sync.aligned.u32 216;");
    const int m = warp >> 2;                 // stream
    const int r = (warp & 3) * 32 + lane;    // query row in the tile == TMEM lane
    const int first = m ? first1 : first0, my_tiles = (m ? end1 : end0) - first;
    const uint32_t lane_off = uint32_t((warp & 3) * 32) << 16;
    const uint32_t tS = tmem + m * 128 + lane_off, tO = tmem + 256 + m * 128 + lane_off;
    // value x of a warp's biases: distance base - x; a row reads x = 31 - lane + key of the tile
    float* wb = sB + warp * 4 * BIAS_COPY;
    const float4* run = reinterpret_cast<const float4*>(wb + ((31 - lane) & 3) * BIAS_COPY + ((31 - lane) & ~3));
    const float* bias = p.bias + (size_t)h * p.size;
    int base = pos0 + m * BQ + (warp & 3) * 32 + 31 - first * BKV;
    float nb[5];
    auto fetch = [&]() {
#pragma unroll
      for (int i = 0; i < 5; ++i) {
        const int dist = base - (i * 32 + lane);
        nb[i] = dist >= 0 && dist < p.size ? bias[dist] : -INFINITY;
      }
      base -= BKV;
    };
    fetch();
    float m_run = -INFINITY, l_run = 0.f;
    bool alive = true;
    for (int j = 0; j < my_tiles; ++j) {
      __syncwarp();                          // the last tile's biases have been read
#pragma unroll
      for (int i = 0; i < 5; ++i)
#pragma unroll
        for (int c = 0; c < 4; ++c)
          if (i * 32 + lane >= c) wb[c * BIAS_COPY + i * 32 + lane - c] = nb[i];
      __syncwarp();
      if (j + 1 < my_tiles) fetch();
      bool ok = mbar_wait(&s_full[m], j & 1);
      ok = __all_sync(0xffffffffu, ok) && !*abort_flag;
      if (!ok) { alive = false; break; }
      tc_fence_after();
      uint32_t sv[4][32];                    // the row's 128 scores
#pragma unroll
      for (int c = 0; c < 4; ++c) tmem_ld_32x32(tS + c * 32, sv[c]);
      tmem_ld_wait();
      float mx[8];                           // independent chains
#pragma unroll
      for (int i = 0; i < 8; ++i) mx[i] = -INFINITY;
#pragma unroll
      for (int i = 0; i < 128; i += 4) {
        const float4 f = run[i >> 2];
        const float add[4] = {f.x, f.y, f.z, f.w};
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const float s = fmaf(__uint_as_float(sv[i >> 5][(i & 31) + u]), p.scale_log2, add[u]);
          sv[i >> 5][(i & 31) + u] = __float_as_uint(s);
          mx[(i + u) & 7] = fmaxf(mx[(i + u) & 7], s);
        }
      }
      const float m_tile = fmaxf(fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])), fmaxf(fmaxf(mx[4], mx[5]), fmaxf(mx[6], mx[7])));
      // a row may see nothing of its stream's first tiles: its maximum is then still -infinity, and its P zero
      const float m_new = fmaxf(m_run, m_tile);
      const bool grow = m_new > m_run + 8.f;
      if (j == 0) {
        m_run = m_new;
      } else if (__any_sync(0xffffffffu, grow)) {
        // O is about to be rescaled: the product that last added to it must have finished
        bool ok2 = mbar_wait(&pv_done[m], (j - 1) & 1);
        ok2 = __all_sync(0xffffffffu, ok2);
        if (!ok2) { alive = false; break; }
        tc_fence_after();
        const float m_next = grow ? m_new : m_run;
        const float alpha = m_run == -INFINITY ? 0.f : exp2f(m_run - m_next);
        l_run *= alpha;
#pragma unroll
        for (int c = 0; c < VN / 32; ++c) {
          uint32_t v[32];
          tmem_ld_32x32(tO + c * 32, v);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * alpha);
          tmem_st_32x32(tO + c * 32, v);
        }
        tmem_st_wait();
        m_run = m_next;
      }
      const float m_sub = m_run == -INFINITY ? 0.f : m_run;
      float lsum[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t w[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          const int kx = half * 64 + 2 * i;
          const float e0 = exp2f(__uint_as_float(sv[kx >> 5][kx & 31]) - m_sub);
          const float e1 = exp2f(__uint_as_float(sv[kx >> 5][(kx & 31) + 1]) - m_sub);
          lsum[i & 3] += e0 + e1;
          __nv_bfloat162 t = __floats2bfloat162_rn(e0, e1);
          w[i] = *reinterpret_cast<uint32_t*>(&t);
        }
        // 64 keys = 32 columns of packed pairs over this tile's own scores, which are all in registers by now
        tmem_st_32x32(tS + half * 32, w);
      }
      tmem_st_wait();
      l_run += (lsum[0] + lsum[1]) + (lsum[2] + lsum[3]);
      tc_fence_before();
      mbar_arrive(&p_full[m]);
    }
    if (alive && my_tiles > 0) {
      bool ok = mbar_wait(&pv_done[m], (my_tiles - 1) & 1);
      ok = __all_sync(0xffffffffu, ok);
      alive = ok;
      if (ok) {
        tc_fence_after();
        const float inv = 1.f / l_run;
        const bool row_ok = q0 + m * BQ + r < q_len;
        const int cols = min(p.slice, p.V - v0);
        __nv_bfloat16* orow = p.out + (size_t)(q_row0 + m * BQ + r) * p.ldo + h * p.V + v0;
#pragma unroll
        for (int c = 0; c < VN / 32; ++c) {
          uint32_t u[32];
          tmem_ld_32x32(tO + c * 32, u);
          tmem_ld_wait();
          if (row_ok) {
#pragma unroll
            for (int i = 0; i < 32; i += 8) {
              if (c * 32 + i < cols) {
                uint4 o;
                uint32_t* w = reinterpret_cast<uint32_t*>(&o);
#pragma unroll
                for (int x = 0; x < 4; ++x) {
                  __nv_bfloat162 t = __floats2bfloat162_rn(__uint_as_float(u[i + 2 * x]) * inv, __uint_as_float(u[i + 2 * x + 1]) * inv);
                  w[x] = *reinterpret_cast<uint32_t*>(&t);
                }
                *reinterpret_cast<uint4*>(orow + c * 32 + i) = o;
              }
            }
          }
        }
      }
    }
    if (!alive) {
      if (lane == 0) atomicExch(p.status, ERR_WAIT_ACC);
      *abort_flag = 1;
    }
  }

  tc_fence_before();
  __syncthreads();
  if (*abort_flag) {
    uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 9) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

template <int VN, int SL>
int launch_as(const CUtensorMap& q, const CUtensorMap& k, const CUtensorMap& v, const Params& p, dim3 grid, size_t smem,
              cudaStream_t stream) {
  static PerDeviceOnce once_;
  bool& configured = once_.slot();
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(window_prefill_kernel<VN, SL>, cudaFuncAttributeMaxDynamicSharedMemorySize, 232448);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  window_prefill_kernel<VN, SL><<<grid, NTHREADS, smem, stream>>>(q, k, v, p);
  return (int)cudaGetLastError();
}

template <int VN>
int launch(const CUtensorMap& q, const CUtensorMap& k, const CUtensorMap& v, const Params& p, dim3 grid, size_t smem, cudaStream_t stream) {
  if (p.D == 64) return launch_as<VN, 1>(q, k, v, p, grid, smem, stream);
  if (p.D == 128) return launch_as<VN, 2>(q, k, v, p, grid, smem, stream);
  return launch_as<VN, 0>(q, k, v, p, grid, smem, stream);
}

}  // namespace windowattn
}  // namespace b200

using namespace b200;

// Sizes the kernel covers: D, V multiples of 16, at most three 64-column slabs of keys, pages of 16 to 128 tokens.
extern "C" int b200_attn_window_prefill_supported(int H, int G, int D, int V, int block_size) {
  return H > 0 && G > 0 && !(H % G) && D > 0 && V > 0 && !(D % 16) && !(V % 16) && D <= 192 &&
         (block_size == 16 || block_size == 32 || block_size == 64 || block_size == 128);
}

// q [q_rows, H, D] bf16; caches [num_blocks * block_size, G * D], [.., G * V] bf16; bias fp32 [H, size] (times log2 e); entry b:
// query rows [q_start, q_start + q_len), table row seq[b] (or b).  The pages of a row's whole window have to be in its table, and
// page 0 finite.
extern "C" int b200_attn_window_prefill(const void* q, const void* k_cache, const void* v_cache, const float* bias, void* out, int ldo,
                                        const int* block_table, const int* seq, const int* q_start, const int* q_len, const int* kv_len,
                                        int batch, int max_q_len, int q_rows, int max_blocks, int num_blocks, int block_size, int H, int G,
                                        int D, int V, int size, float scale, int* status, cudaStream_t stream) {
  using namespace b200::windowattn;
  if (!b200_attn_window_prefill_supported(H, G, D, V, block_size) || batch <= 0 || batch > 65535 || max_q_len <= 0 || q_rows <= 0 ||
      size <= 0 || !bias || (ldo & 7) || ldo < H * V)
    return -ERR_BAD_ARG;
  Params p;
  p.slabs = (D + 63) / 64;
  p.slice = p.slabs >= 3 ? 64 : 128;         // wide keys leave room for one value slab per tile
  const int VN = V >= p.slice ? p.slice : (V + 31) / 32 * 32, VS = (VN + 63) / 64;
  p.v_slices = (V + p.slice - 1) / p.slice;
  p.stages = (BUDGET - 2 * p.slabs * ATOM) / ATOM;
  if (p.stages > MAX_STAGES) p.stages = MAX_STAGES;
  if (p.stages < p.slabs + VS + (VS == 2) || (long long)H * p.v_slices > 65535) return -ERR_BAD_ARG;
  const size_t smem = (size_t)(2 * p.slabs + p.stages) * ATOM + 1024 + 512 + BIAS_BYTES;
  CUtensorMap tmQ, tmK, tmV;
  const uint64_t QW = (uint64_t)H * D, KW = (uint64_t)G * D, VW = (uint64_t)G * V, kv_rows = (uint64_t)num_blocks * block_size;
  bool ok = make_tmap_2d(&tmQ, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, q, q_rows, QW, QW * 2, BQ, 64, CU_TENSOR_MAP_SWIZZLE_128B);
  ok = ok && make_tmap_2d(&tmK, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, k_cache, kv_rows, KW, KW * 2, block_size, 64,
                          CU_TENSOR_MAP_SWIZZLE_128B);
  ok = ok && make_tmap_2d(&tmV, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, v_cache, kv_rows, VW, VW * 2, block_size, 64,
                          CU_TENSOR_MAP_SWIZZLE_128B);
  if (!ok) return -ERR_BAD_ARG;
  p.block_table = block_table; p.seq = seq; p.q_start = q_start; p.q_len = q_len; p.kv_len = kv_len; p.bias = bias;
  p.max_blocks = max_blocks; p.block_size = block_size; p.H = H; p.G = G; p.D = D; p.V = V; p.size = size;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.out = reinterpret_cast<__nv_bfloat16*>(out); p.ldo = ldo; p.status = status;
  const dim3 grid((max_q_len + 2 * BQ - 1) / (2 * BQ), H * p.v_slices, batch);
  switch (VN) {
    case 32: return launch<32>(tmQ, tmK, tmV, p, grid, smem, stream);
    case 64: return launch<64>(tmQ, tmK, tmV, p, grid, smem, stream);
    case 96: return launch<96>(tmQ, tmK, tmV, p, grid, smem, stream);
    default: return launch<128>(tmQ, tmK, tmV, p, grid, smem, stream);
  }
}
