// Flash-attention prefill over a paged KV cache for heads whose scores are mixed before the softmax, sm_100a.
//
// The mixing s_h = sum_g talk[h, g] (q_g . k_kv(g)) is linear, so it is folded into the queries (qk_row_prep.cu):
// head h becomes ONE dot product of q_mix[h] with all key heads of a token side by side.  Every head then reads the same
// [keys, G * D] key matrix, and the score GEMM accumulates the mixed scores in fp32 in tensor memory: no pass over raw
// scores, no H x H arithmetic per key.
//
// One CTA = one 128-row query tile of one head.  Warp roles:
//   warp 4  : TMA producer of the key tile of 128 tokens, in slabs of 64 columns through a ring (with the query slab of the
//             same columns beside it when the query tile does not fit in shared memory as a whole), page by page through
//             the sequence's block table;
//   warp 6  : TMA producer of the value tile of the head's key/value group, on its own so that neither kind of tile waits
//             for the other's buffers;
//   warp 5  : tcgen05.mma issuer - S(j+1) into the other of two TMEM score buffers before P(j) V(j), so that the softmax
//             of one tile overlaps the score GEMM of the next; O accumulates in TMEM, V consumed MN-major;
//   warps 0-3: softmax - one query row per thread, online maximum / sum in the exp2 domain, P as bf16 back into the tensor
//             memory its scores came from (the P V product reads it there), lazy rescale of O.
// Masks: causal, and (chunk > 0) only keys of the query's own chunk of `chunk` positions; key tiles below the first
// row's chunk are skipped.  All mbarrier waits are bounded and unwind through the common exit.
#include <cuda_bf16.h>
#include "per_device.h"
#include "../ptx/sm100.cuh"
#include "tma_host.h"
#include "ops.h"

namespace b200 {
namespace mixattn {

constexpr int BQ = 128;         // query rows per CTA
constexpr int BKV = 128;        // keys per tile
constexpr int ATOM = 16384;     // bytes of one [128 x 64] bf16 swizzled atom
constexpr int NTHREADS = 224;
constexpr int MAX_STAGES = 8;
constexpr int BUDGET = 232448 - 1024 /* alignment */ - 512 /* barriers */;

struct Params {
  const int* block_table;  // [B, max_blocks]
  const int* seq;          // [B] table row of each entry, or null (entry i -> row i)
  const int* q_start;      // [B] first query row of the entry
  const int* q_len;        // [B]
  const int* kv_len;       // [B] context length including the entry's own tokens
  int max_blocks, block_size;
  int H, G, D;
  int slabs, stages, chunk;
  float scale_log2;
  __nv_bfloat16* out;      // [rows, ldo]
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

// VA: 64-column atoms of the value tile (head width up to 64 * VA).  QRES: the query tile stays in shared memory.
template <int VA, bool QRES>
__global__ void __launch_bounds__(NTHREADS, 1)
mix_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                   const __grid_constant__ CUtensorMap tmV, Params p) {
  constexpr int VN = 64 * VA;
  constexpr uint32_t idesc_qk = umma_idesc_bf16(128, 128);
  constexpr uint32_t idesc_pv = umma_idesc_bf16(128, VN) | (1u << 16);   // B is MN-major
  constexpr int STAGE = QRES ? ATOM : 2 * ATOM;
  extern __shared__ uint8_t smem_base[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_base) + 1023) & ~uintptr_t(1023));
  uint8_t* sV = smem;                                   // VA atoms
  uint8_t* sQ = sV + VA * ATOM;                         // slabs atoms when resident
  uint8_t* sR = sQ + (QRES ? p.slabs * ATOM : 0);       // ring: K slab (+ Q slab)
  uint64_t* bars = reinterpret_cast<uint64_t*>(sR + p.stages * STAGE);
  uint64_t* r_full = bars;                   // MAX_STAGES
  uint64_t* r_empty = bars + MAX_STAGES;     // MAX_STAGES
  uint64_t* q_full = bars + 2 * MAX_STAGES;
  uint64_t* v_full = q_full + 1;
  uint64_t* v_empty = q_full + 2;
  uint64_t* s_full = q_full + 3;             // 2
  uint64_t* p_full = q_full + 5;
  uint64_t* pv_done = q_full + 6;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(q_full + 7);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0), lane = threadIdx.x & 31;   // uniform: the issuer depends on it
  const int b = blockIdx.z, h = blockIdx.y, qt = (int)gridDim.x - 1 - (int)blockIdx.x;   // long tiles first
  const int q_len = p.q_len[b], kv_len = p.kv_len[b];
  const int q0 = qt * BQ;
  if (q0 >= q_len) return;                   // uniform per CTA, before any barrier / TMEM use
  const int q_row0 = p.q_start[b] + q0;
  const int kvh = h / (p.H / p.G);
  const int pos0 = kv_len - q_len + q0;      // position of the tile's first query row
  const int tile_end = (min(kv_len, pos0 + BQ) + BKV - 1) / BKV;
  const int tile0 = p.chunk > 0 ? (pos0 - pos0 % p.chunk) / BKV : 0;
  const int n_tiles = tile_end - tile0;      // >= 1: the tile holding pos0 itself

  if (threadIdx.x == 0) {
    for (int i = 0; i < p.stages; ++i) {
      mbar_init(&r_full[i], 1);
      mbar_init(&r_empty[i], 1);
    }
    mbar_init(q_full, 1);
    mbar_init(v_full, 1);
    mbar_init(v_empty, 1);
    mbar_init(&s_full[0], 1);
    mbar_init(&s_full[1], 1);
    mbar_init(p_full, 128);
    mbar_init(pv_done, 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 5) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  // V starts finite: rows of keys past the context are never loaded but still multiply P = 0
  for (int i = threadIdx.x; i < VA * ATOM / 16; i += NTHREADS) reinterpret_cast<uint4*>(sV)[i] = make_uint4(0, 0, 0, 0);
  fence_proxy_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  const uint32_t tO = tmem + 256;

  if (warp == 4) {
    if (lane == 0) {
      tma_prefetch_desc(&tmQ);
      tma_prefetch_desc(&tmK);
      tma_prefetch_desc(&tmV);
      // the query tile: rows (token, head) -> the map is [tokens, H * G * D], head h starts at column h * G * D
      const int qx = h * p.G * p.D;
      if (QRES) {
        mbar_expect_tx(q_full, p.slabs * ATOM);
        for (int s = 0; s < p.slabs; ++s) tma_load_2d(sQ + s * ATOM, &tmQ, q_full, qx + s * 64, q_row0);
      }
      const int* bt = p.block_table + (size_t)(p.seq ? p.seq[b] : b) * p.max_blocks;
      const int bs = p.block_size;
      const uint32_t sub_bytes = bs * 128;   // 64 columns of one page
      bool ok = true;
      int st = 0;
      uint32_t ph = 1;
      auto load_k = [&](int j) {
        const int key0 = (tile0 + j) * BKV, page0 = key0 / bs, nblk = (min(BKV, kv_len - key0) + bs - 1) / bs;
        // pages of 64 tokens and more: the table is read once per tile, and a slab is two copies at most (this thread's
        // instruction count per slab is what paces the whole pipeline)
        const int row0 = bt[page0] * bs, row1 = nblk > 1 ? bt[page0 + 1] * bs : 0;
        for (int s = 0; s < p.slabs; ++s) {
          if (!mbar_wait(&r_empty[st], ph)) return false;
          uint8_t* dst = sR + st * STAGE;
          mbar_expect_tx(&r_full[st], nblk * sub_bytes + (QRES ? 0 : ATOM));
          if (!QRES) tma_load_2d(dst + ATOM, &tmQ, &r_full[st], qx + s * 64, q_row0);
          tma_load_2d(dst, &tmK, &r_full[st], s * 64, row0);
          if (nblk > 1) tma_load_2d(dst + sub_bytes, &tmK, &r_full[st], s * 64, row1);
          for (int i = 2; i < nblk; ++i) tma_load_2d(dst + i * sub_bytes, &tmK, &r_full[st], s * 64, bt[page0 + i] * bs);
          if (++st == p.stages) { st = 0; ph ^= 1; }
        }
        return true;
      };
      for (int j = 0; ok && j < n_tiles && !*abort_flag; ++j) ok = load_k(j);
      if (!ok) { atomicExch(p.status, ERR_WAIT_STAGE); *abort_flag = 1; }
    }
  } else if (warp == 6) {
    if (lane == 0) {
      const int* bt = p.block_table + (size_t)(p.seq ? p.seq[b] : b) * p.max_blocks;
      const int bs = p.block_size;
      const uint32_t sub_bytes = bs * 128;
      bool ok = true;
      for (int j = 0; ok && j < n_tiles && !*abort_flag; ++j) {
        const int key0 = (tile0 + j) * BKV, page0 = key0 / bs, nblk = (min(BKV, kv_len - key0) + bs - 1) / bs;
        if (!mbar_wait(v_empty, (j & 1) ^ 1)) { ok = false; break; }
        mbar_expect_tx(v_full, nblk * sub_bytes * VA);
        for (int i = 0; i < nblk; ++i) {
          const int row = bt[page0 + i] * bs;
#pragma unroll
          for (int a = 0; a < VA; ++a) tma_load_2d(sV + a * ATOM + i * sub_bytes, &tmV, v_full, kvh * p.D + a * 64, row);
        }
      }
      if (!ok) { atomicExch(p.status, ERR_WAIT_STAGE); *abort_flag = 1; }
    }
  } else if (warp == 5) {
    if (lane == 0) {
      bool ok = !QRES || mbar_wait(q_full, 0);
      int st = 0;
      uint32_t ph = 0;
      auto issue_s = [&](int j) -> bool {
        const uint32_t tS = tmem + (j & 1) * 128;
        for (int s = 0; s < p.slabs; ++s) {
          if (!mbar_wait(&r_full[st], ph)) return false;
          tc_fence_after();
          const uint8_t* k = sR + st * STAGE;
          const uint8_t* q = QRES ? sQ + s * ATOM : k + ATOM;
#pragma unroll
          for (int kk = 0; kk < 4; ++kk)
            umma_bf16_ss(tS, umma_desc_sw128(q) + 2 * kk, umma_desc_sw128(k) + 2 * kk, idesc_qk, (s | kk) ? 1u : 0u);
          umma_commit(&r_empty[st]);
          if (++st == p.stages) { st = 0; ph ^= 1; }
        }
        umma_commit(&s_full[j & 1]);
        return true;
      };
      if (ok) ok = issue_s(0);
      for (int j = 0; ok && j < n_tiles && !*abort_flag; ++j) {
        if (j + 1 < n_tiles) {
          ok = issue_s(j + 1);
          if (!ok) break;
        }
        if (!mbar_wait(p_full, j & 1) || !mbar_wait(v_full, j & 1)) { ok = false; break; }
        tc_fence_after();
#pragma unroll
        for (int kk = 0; kk < 8; ++kk) {
          const uint64_t db = desc_mn_sw128(sV + kk * 2048, ATOM, 1024);
          umma_bf16_ts(tO, tmem + (j & 1) * 128 + kk * 8, db, idesc_pv, (j | kk) ? 1u : 0u);
        }
        umma_commit(v_empty);
        umma_commit(pv_done);
      }
      if (!ok) { atomicExch(p.status, ERR_WAIT_TMA); *abort_flag = 1; }
    }
  } else {
    const int r = warp * 32 + lane;          // query row in the tile == TMEM lane
    const int limit = pos0 + r;              // last visible key of this row
    const int first = p.chunk > 0 ? limit - limit % p.chunk : 0;
    const uint32_t lane_off = uint32_t(warp * 32) << 16;
    float m_run = -INFINITY, l_run = 0.f;
    bool alive = true;
    for (int j = 0; j < n_tiles; ++j) {
      const int sb = j & 1;
      bool ok = mbar_wait(&s_full[sb], (j >> 1) & 1);
      ok = __all_sync(0xffffffffu, ok) && !*abort_flag;
      if (!ok) { alive = false; break; }
      tc_fence_after();
      float s[128];
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        uint32_t v[32];
        tmem_ld_32x32(tmem + sb * 128 + lane_off + c * 32, v);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) s[c * 32 + i] = __uint_as_float(v[i]) * p.scale_log2;
      }
      const int key0 = (tile0 + j) * BKV;
      const int kmax = min(limit, kv_len - 1) - key0, kmin = first - key0;
      float m_tile = -INFINITY;
      if (kmax < 127 || kmin > 0) {
#pragma unroll
        for (int i = 0; i < 128; ++i) {
          if (i > kmax || i < kmin) s[i] = -INFINITY;
          m_tile = fmaxf(m_tile, s[i]);
        }
      } else {
#pragma unroll
        for (int i = 0; i < 128; ++i) m_tile = fmaxf(m_tile, s[i]);
      }
      // a row whose keys were all masked so far has m_run = -inf, l_run = 0 and an O of zeros
      const float m_new = fmaxf(m_run, m_tile);
      const bool grow = m_new > m_run + 8.f || (m_run == -INFINITY && m_new > -INFINITY);
      if (j == 0) {
        m_run = m_new;
      } else if (__any_sync(0xffffffffu, grow)) {
        // O is about to be rescaled: the product that last added to it must have finished
        bool ok2 = mbar_wait(pv_done, (j - 1) & 1);
        ok2 = __all_sync(0xffffffffu, ok2);
        if (!ok2) { alive = false; break; }
        tc_fence_after();
        const float m_next = grow ? m_new : m_run;
        const float alpha = (m_run == -INFINITY) ? 0.f : exp2f(m_run - m_next);
        l_run *= alpha;
#pragma unroll
        for (int c = 0; c < VN / 32; ++c) {
          uint32_t v[32];
          tmem_ld_32x32(tO + lane_off + c * 32, v);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * alpha);
          tmem_st_32x32(tO + lane_off + c * 32, v);
        }
        tmem_st_wait();
        m_run = m_next;
      }
      const float m_use = m_run == -INFINITY ? 0.f : m_run;
      float lsum = 0.f;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t w[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          const float e0 = exp2f(s[half * 64 + 2 * i] - m_use), e1 = exp2f(s[half * 64 + 2 * i + 1] - m_use);
          lsum += e0 + e1;
          __nv_bfloat162 t = __floats2bfloat162_rn(e0, e1);
          w[i] = *reinterpret_cast<uint32_t*>(&t);
        }
        // 64 keys = 32 columns of packed pairs over this tile's own scores, which are all in registers by now
        tmem_st_32x32(tmem + sb * 128 + lane_off + half * 32, w);
      }
      tmem_st_wait();
      l_run += lsum;
      // the issuer handles one P at a time: hand this one over only after the previous product is through
      if (j > 0) {
        bool ok2 = mbar_wait(pv_done, (j - 1) & 1);
        ok2 = __all_sync(0xffffffffu, ok2);
        if (!ok2) { alive = false; break; }
      }
      tc_fence_before();
      mbar_arrive(p_full);
    }
    if (alive) {
      bool ok = mbar_wait(pv_done, (n_tiles - 1) & 1);
      ok = __all_sync(0xffffffffu, ok);
      if (ok) {
        tc_fence_after();
        const float inv = l_run > 0.f ? 1.f / l_run : 0.f;
        const bool row_ok = (q0 + r) < q_len;
        __nv_bfloat16* orow = p.out + (size_t)(q_row0 + r) * p.ldo + h * p.D;
#pragma unroll
        for (int c = 0; c < VN / 32; ++c) {
          uint32_t v[32];
          tmem_ld_32x32(tO + lane_off + c * 32, v);
          tmem_ld_wait();
#pragma unroll
          for (int g8 = 0; g8 < 4; ++g8) {
            if (row_ok && c * 32 + g8 * 8 < p.D) {
              uint4 u;
              uint32_t* w = reinterpret_cast<uint32_t*>(&u);
#pragma unroll
              for (int i = 0; i < 4; ++i) {
                __nv_bfloat162 t = __floats2bfloat162_rn(__uint_as_float(v[g8 * 8 + 2 * i]) * inv,
                                                         __uint_as_float(v[g8 * 8 + 2 * i + 1]) * inv);
                w[i] = *reinterpret_cast<uint32_t*>(&t);
              }
              *reinterpret_cast<uint4*>(orow + c * 32 + g8 * 8) = u;
            }
          }
        }
      } else {
        alive = false;
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
  if (warp == 5) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

template <int VA, bool QRES>
int launch(const CUtensorMap& q, const CUtensorMap& k, const CUtensorMap& v, const Params& p, dim3 grid, size_t smem,
           cudaStream_t stream) {
  static PerDeviceOnce once_;
  bool& configured = once_.slot();
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(mix_prefill_kernel<VA, QRES>, cudaFuncAttributeMaxDynamicSharedMemorySize, 232448);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  mix_prefill_kernel<VA, QRES><<<grid, NTHREADS, smem, stream>>>(q, k, v, p);
  return (int)cudaGetLastError();
}

}  // namespace mixattn
}  // namespace b200

using namespace b200;

// 1 when the tensor-core kernel covers these sizes (one head's values fit the accumulator).
extern "C" int b200_attn_mix_prefill_supported(int H, int G, int D, int block_size) {
  return H > 0 && G > 0 && H % G == 0 && D > 0 && D % 8 == 0 && D <= 256 &&
         (block_size == 16 || block_size == 32 || block_size == 64 || block_size == 128);
}

// q_mix: [q_rows, H, G * D] bf16; caches [num_blocks * block_size, G * D] bf16; entries of B sequences, rows
// [q_start, q_start + q_len) each; out [q_rows, ldo] bf16 (head h at columns h * D).
extern "C" int b200_attn_mix_prefill(const void* q_mix, const void* k_cache, const void* v_cache, void* out,
                                     const int* block_table, const int* seq, const int* q_start, const int* q_len,
                                     const int* kv_len, int batch, int max_q_len, int q_rows, int max_blocks, int num_blocks,
                                     int block_size, int H, int G, int D, int chunk, int ldo, float scale, int* status,
                                     cudaStream_t stream) {
  using namespace b200::mixattn;
  if (!b200_attn_mix_prefill_supported(H, G, D, block_size) || batch <= 0 || max_q_len <= 0 || q_rows <= 0 || chunk < 0 ||
      (ldo & 7) || ldo < H * D)
    return -ERR_BAD_ARG;
  const int KW = G * D, VA = (D + 63) / 64;
  Params p;
  p.slabs = (KW + 63) / 64;
  const int fixed = VA * ATOM;
  const bool qres = fixed + p.slabs * ATOM + 3 * ATOM <= BUDGET;
  const int stage = qres ? ATOM : 2 * ATOM;
  p.stages = (BUDGET - fixed - (qres ? p.slabs * ATOM : 0)) / stage;
  if (p.stages > MAX_STAGES) p.stages = MAX_STAGES;
  if (p.stages < 2) return -ERR_BAD_ARG;
  const size_t smem = fixed + (qres ? p.slabs * ATOM : 0) + (size_t)p.stages * stage + 1024 + 512;
  // a query slab may run past its head into the next one: the key map ends at G * D, so those columns multiply zeros
  CUtensorMap tmQ, tmK, tmV;
  bool ok = make_tmap_2d(&tmQ, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, q_mix, q_rows, (uint64_t)H * KW, (uint64_t)H * KW * 2, BQ, 64,
                         CU_TENSOR_MAP_SWIZZLE_128B);
  const uint64_t kv_rows = (uint64_t)num_blocks * block_size;
  ok = ok && make_tmap_2d(&tmK, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, k_cache, kv_rows, KW, (uint64_t)KW * 2, block_size, 64,
                          CU_TENSOR_MAP_SWIZZLE_128B);
  ok = ok && make_tmap_2d(&tmV, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, v_cache, kv_rows, KW, (uint64_t)KW * 2, block_size, 64,
                          CU_TENSOR_MAP_SWIZZLE_128B);
  if (!ok) return -ERR_BAD_ARG;
  p.block_table = block_table; p.seq = seq; p.q_start = q_start; p.q_len = q_len; p.kv_len = kv_len;
  p.max_blocks = max_blocks; p.block_size = block_size; p.H = H; p.G = G; p.D = D; p.chunk = chunk;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.out = reinterpret_cast<__nv_bfloat16*>(out);
  p.ldo = ldo;
  p.status = status;
  const dim3 grid((max_q_len + BQ - 1) / BQ, H, batch);
#define B200_MIX_CASE(va)                                                        \
  case va:                                                                       \
    return qres ? launch<va, true>(tmQ, tmK, tmV, p, grid, smem, stream)         \
                : launch<va, false>(tmQ, tmK, tmV, p, grid, smem, stream);
  switch (VA) {
    B200_MIX_CASE(1) B200_MIX_CASE(2) B200_MIX_CASE(3) B200_MIX_CASE(4)
  }
#undef B200_MIX_CASE
  return -ERR_BAD_ARG;
}
