// Differential flash-attention prefill over a paged KV cache, sm_100a.  Every head has two softmax maps with their own
// query and key vectors and a common value; the output is a_1 - lambda a_2, normalised per head and gated (attn_diff.cuh).
//
// One CTA = one 128-row query tile of one head, BOTH maps: the value tile is loaded once for the two products, and the two
// maps are the two streams that keep the tensor core and the exponential units busy in turn.  Warp roles:
//   warps 0-3, 4-7: softmax of map 1 and of map 2 - one query row per thread, online maximum / sum in the exp2 domain, P as
//             bf16 back into the tensor memory its scores came from, lazy rescale of the map's O;
//   warp 8  : TMA producer.  Keys and values travel as slabs of [128 tokens x 64 columns] through one ring, page by page
//             through the sequence's block table (pages past the context read page 0, which holds zeros);
//   warp 9  : tcgen05.mma issuer - per tile P1 V, S1 of the next tile, P2 V, S2 of the next tile: each map's score GEMM runs
//             while the other map's softmax does.
// Tensor memory: S1 | S2 (128 columns each) and O1 | O2 (up to 128 columns each).  Values wider than 128 are cut into
// column slices, one CTA each; the difference then goes out in fp32 and a row kernel finishes it (attn_diff_rows.cu).
// Vectors narrower than 64 columns leave the rest of their slab unused: a slab reads on into the next vector, the products
// stop at D.  All mbarrier waits are bounded and unwind through the common exit.
#include <cuda_bf16.h>
#include "attn_diff.cuh"
#include "per_device.h"
#include "../ptx/sm100.cuh"
#include "tma_host.h"
#include "ops.h"

namespace b200 {
namespace diffattn {

constexpr int BQ = 128;         // query rows per CTA
constexpr int BKV = 128;        // keys per tile
constexpr int ATOM = 16384;     // bytes of one [128 x 64] bf16 swizzled slab
constexpr int NTHREADS = 384;   // three warpgroups; the third has the two single-thread roles and gives its registers up
constexpr int MAX_STAGES = 12;
constexpr int BUDGET = 232448 - 1024 /* alignment */ - 512 /* barriers */ - 1024 /* row sums */;

struct Params {
  const int* block_table;  // [B, max_blocks]
  const int* seq;          // [B] table row of each entry, or null (entry i -> row i)
  const int* q_start;      // [B] first query row of the entry
  const int* q_len;        // [B]
  const int* kv_len;       // [B] context length including the entry's own tokens
  int max_blocks, block_size;
  int H, G, D, V;
  int slabs, stages, v_slices;
  float scale_log2;
  __nv_bfloat16* out;      // [rows, ldo], or null
  float* diff;             // [rows, H, V] (out null)
  const __nv_bfloat16* gate;   // [rows, ld_gate]
  int ldo, ld_gate;
  DiffFinish fin;
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

// VN: columns of a value slice rounded up to 32 (the accumulator's width in tensor memory and of the products).
template <int VN>
__global__ void __launch_bounds__(NTHREADS, 1)
diff_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                    const __grid_constant__ CUtensorMap tmV, Params p) {
  constexpr uint32_t idesc_qk = umma_idesc_bf16(128, 128);
  constexpr uint32_t idesc_pv = umma_idesc_bf16(128, VN) | (1u << 16);   // B is MN-major
  constexpr int VS = (VN + 63) / 64;                                     // slabs of the value slice
  extern __shared__ uint8_t smem_base[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_base) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;                                   // [2 maps][slabs] atoms
  uint8_t* sR = sQ + 2 * p.slabs * ATOM;                // ring of slabs
  float* s_sum = reinterpret_cast<float*>(sR + p.stages * ATOM);         // [2][128] reciprocal sums
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_sum + 256);
  uint64_t* r_full = bars;                   // MAX_STAGES
  uint64_t* r_empty = bars + MAX_STAGES;     // MAX_STAGES
  uint64_t* q_full = bars + 2 * MAX_STAGES;
  uint64_t* s_full = q_full + 1;             // per map
  uint64_t* p_full = q_full + 3;
  uint64_t* pv_done = q_full + 5;
  uint64_t* o_ready = q_full + 7;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(q_full + 8);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0), lane = threadIdx.x & 31;   // uniform: the issuer depends on it
  const int b = blockIdx.z, qt = (int)gridDim.x - 1 - (int)blockIdx.x;   // long tiles first
  const int h = blockIdx.y / p.v_slices, v0 = (blockIdx.y % p.v_slices) * 128;
  const int q_len = p.q_len[b], kv_len = p.kv_len[b];
  const int q0 = qt * BQ;
  if (q0 >= q_len) return;                   // uniform per CTA, before any barrier / TMEM use
  const int q_row0 = p.q_start[b] + q0;
  const int g = h / (p.H / p.G);
  const int pos0 = kv_len - q_len + q0;      // position of the tile's first query row
  const int n_tiles = (min(kv_len, pos0 + BQ) + BKV - 1) / BKV;

  if (threadIdx.x == 0) {
    for (int i = 0; i < p.stages; ++i) {
      mbar_init(&r_full[i], 1);
      mbar_init(&r_empty[i], 1);
    }
    mbar_init(q_full, 1);
    for (int m = 0; m < 2; ++m) {
      mbar_init(&s_full[m], 1);
      mbar_init(&p_full[m], 128);
      mbar_init(&pv_done[m], 1);
    }
    mbar_init(o_ready, 128);
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
  const uint32_t tmem = *tmem_slot;

  // registers per thread at launch: 168 (3 x 168 = 2 x 216 + 72)
  if (warp >= 8) {
    asm volatile("setmaxnreg.dec.sync.aligned.u32 72;");
    if (warp == 8 && lane == 0) {
      tma_prefetch_desc(&tmQ);
      tma_prefetch_desc(&tmK);
      tma_prefetch_desc(&tmV);
      mbar_expect_tx(q_full, 2 * p.slabs * ATOM);
      for (int m = 0; m < 2; ++m)
        for (int s = 0; s < p.slabs; ++s)
          tma_load_2d(sQ + (m * p.slabs + s) * ATOM, &tmQ, q_full, (h * 2 + m) * p.D + s * 64, q_row0);
      const int* bt = p.block_table + (size_t)(p.seq ? p.seq[b] : b) * p.max_blocks;
      const int bs = p.block_size, pages = BKV / bs, last_page = (kv_len - 1) / bs;
      const uint32_t sub_bytes = bs * 128;   // 64 columns of one page
      int st = 0;
      uint32_t ph = 1;
      bool ok = true;
      for (int j = 0; ok && j < n_tiles && !*abort_flag; ++j) {
        int rows[BKV / 16];
#pragma unroll
        for (int i = 0; i < BKV / 16; ++i) {
          const int page = j * pages + i;
          rows[i] = i < pages && page <= last_page ? bt[page] * bs : 0;
        }
        auto slab = [&](const CUtensorMap* tm, int x) {
          if (!mbar_wait(&r_empty[st], ph)) return false;
          uint8_t* dst = sR + st * ATOM;
          mbar_expect_tx(&r_full[st], ATOM);
#pragma unroll
          for (int i = 0; i < BKV / 16; ++i)
            if (i < pages) tma_load_2d(dst + i * sub_bytes, tm, &r_full[st], x, rows[i]);
          if (++st == p.stages) { st = 0; ph ^= 1; }
          return true;
        };
        for (int m = 0; ok && m < 2; ++m)
          for (int s = 0; ok && s < p.slabs; ++s) ok = slab(&tmK, (g * 2 + m) * p.D + s * 64);
#pragma unroll
        for (int s = 0; s < VS; ++s)
          if (ok) ok = slab(&tmV, g * p.V + v0 + s * 64);
      }
      if (!ok) { atomicExch(p.status, ERR_WAIT_STAGE); *abort_flag = 1; }
    } else if (warp == 9) {
      // The whole warp walks the loop, so that addresses and descriptors stay warp-uniform, and one elected lane issues.
      bool ok = true;
      auto wait = [&](uint64_t* bar, uint32_t parity) {
        ok = __all_sync(0xffffffffu, mbar_wait(bar, parity));
        return ok;
      };
      wait(q_full, 0);
      // slabs are waited for in the order they were filled; only a tile's value slabs are given back later (after the next
      // tile's first-map keys, which lie behind them)
      int st = 0;
      uint32_t ph = 0;
      const uint64_t ring = umma_desc_sw128(sR), dq0 = umma_desc_sw128(sQ);
      const int stages = p.stages, slabs = p.slabs, last_steps = (p.D - (slabs - 1) * 64) / 16;
      auto issue_s = [&](const int m) {
        for (int s = 0; s < slabs; ++s) {
          if (!wait(&r_full[st], ph)) return;
          tc_fence_after();
          const uint64_t dk = ring + st * (ATOM >> 4), dq = dq0 + (m * slabs + s) * (ATOM >> 4);
          const int steps = s + 1 < slabs ? 4 : last_steps;
          if (elect_one()) {
            umma_bf16_ss(tmem + m * 128, dq, dk, idesc_qk, s ? 1u : 0u);
#pragma unroll
            for (int kk = 1; kk < 4; ++kk)
              if (kk < steps) umma_bf16_ss(tmem + m * 128, dq + 2 * kk, dk + 2 * kk, idesc_qk, 1u);
            umma_commit(&r_empty[st]);
            if (s + 1 == slabs) umma_commit(&s_full[m]);
          }
          if (++st == stages) { st = 0; ph ^= 1; }
        }
      };
      if (ok) issue_s(0);
      if (ok) issue_s(1);
      for (int j = 0; ok && j < n_tiles && !*abort_flag; ++j) {
        int sv = 0;
#pragma unroll
        for (int m = 0; m < 2; ++m) {
          if (!ok || !wait(&p_full[m], j & 1)) break;
          if (m == 0) {
            // two slabs of a tile are neighbours: the ring has an even number of stages and a tile an even number of slabs
            sv = st;
#pragma unroll
            for (int s = 0; s < VS; ++s)
              if (ok && wait(&r_full[st], ph) && ++st == stages) { st = 0; ph ^= 1; }
            if (!ok) break;
          }
          tc_fence_after();
          const uint64_t dv = desc_mn_sw128(sR, ATOM, 1024) + sv * (ATOM >> 4);
          if (elect_one()) {
            umma_bf16_ts(tmem + 256 + m * 128, tmem + m * 128, dv, idesc_pv, j ? 1u : 0u);
#pragma unroll
            for (int kk = 1; kk < 8; ++kk) umma_bf16_ts(tmem + 256 + m * 128, tmem + m * 128 + kk * 8, dv + kk * 128, idesc_pv, 1u);
            umma_commit(&pv_done[m]);
            if (m == 1) {
#pragma unroll
              for (int s = 0; s < VS; ++s) umma_commit(&r_empty[sv + s]);
            }
          }
          if (j + 1 < n_tiles) issue_s(m);
        }
      }
      if (!ok && lane == 0) { atomicExch(p.status, ERR_WAIT_TMA); *abort_flag = 1; }
    }
  } else {
    asm volatile("setmaxnreg.inc.sync.aligned.u32 216;");
    const int m = warp >> 2;                 // map
    const int r = (warp & 3) * 32 + lane;    // query row in the tile == TMEM lane
    const int limit = pos0 + r;              // last visible key of this row
    const uint32_t lane_off = uint32_t((warp & 3) * 32) << 16;
    const uint32_t tS = tmem + m * 128 + lane_off, tO = tmem + 256 + m * 128 + lane_off;
    float m_run = -INFINITY, l_run = 0.f;
    bool alive = true;
    for (int j = 0; j < n_tiles; ++j) {
      bool ok = mbar_wait(&s_full[m], j & 1);
      ok = __all_sync(0xffffffffu, ok) && !*abort_flag;
      if (!ok) { alive = false; break; }
      tc_fence_after();
      uint32_t sv[4][32];                    // the row's 128 scores
#pragma unroll
      for (int c = 0; c < 4; ++c) tmem_ld_32x32(tS + c * 32, sv[c]);
      tmem_ld_wait();
      const int kmax = min(limit, kv_len - 1) - j * BKV;
      if (kmax < 127) {
#pragma unroll
        for (int i = 0; i < 128; ++i)
          if (i > kmax) sv[i >> 5][i & 31] = 0xff800000u;      // -inf
      }
      float mx[8];                           // independent chains
#pragma unroll
      for (int i = 0; i < 8; ++i) mx[i] = __uint_as_float(sv[0][i]);
#pragma unroll
      for (int i = 8; i < 128; ++i) mx[i & 7] = fmaxf(mx[i & 7], __uint_as_float(sv[i >> 5][i & 31]));
      const float m_tile = p.scale_log2 * fmaxf(fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])), fmaxf(fmaxf(mx[4], mx[5]), fmaxf(mx[6], mx[7])));
      // every row sees key 0, so the first tile gives a finite maximum
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
        const float alpha = exp2f(m_run - m_next);
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
      float lsum[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t w[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          const int k = half * 64 + 2 * i;
          const float e0 = exp2f(fmaf(__uint_as_float(sv[k >> 5][k & 31]), p.scale_log2, -m_run));
          const float e1 = exp2f(fmaf(__uint_as_float(sv[k >> 5][(k & 31) + 1]), p.scale_log2, -m_run));
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
    if (alive) {
      // the second map's rows hand over their sums; the first map's threads read both accumulators of their row
      if (m == 1) {
        s_sum[r] = l_run;
        mbar_arrive(o_ready);
      } else {
        // o_ready first: it says that the second map has reached its last tile, whose phase is then the one waited for
        bool ok = mbar_wait(o_ready, 0) && mbar_wait(&pv_done[0], (n_tiles - 1) & 1) && mbar_wait(&pv_done[1], (n_tiles - 1) & 1);
        ok = __all_sync(0xffffffffu, ok);
        alive = ok;
        if (ok) {
          tc_fence_after();
          const float inv1 = 1.f / l_run, inv2 = p.fin.lambda / s_sum[r];
          const bool row_ok = (q0 + r) < q_len;
          const size_t row = (size_t)(q_row0 + r);
          const int cols = min(128, p.V - v0);
          // 32 columns of the difference; columns past the slice come from the next group's values
          auto load_diff = [&](int c, float (&d)[32]) {
            uint32_t u[32], v[32];
            tmem_ld_32x32(tO + c * 32, u);
            tmem_ld_32x32(tO + 128 + c * 32, v);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i)
              d[i] = c * 32 + i < cols ? __uint_as_float(u[i]) * inv1 - __uint_as_float(v[i]) * inv2 : 0.f;
          };
          float f = 0.f;
          if (!p.diff) {
            float ss = 0.f;
#pragma unroll
            for (int c = 0; c < VN / 32; ++c) {
              float d[32];
              load_diff(c, d);
#pragma unroll
              for (int i = 0; i < 32; ++i) ss = fmaf(d[i], d[i], ss);
            }
            f = diff_head_scale(ss, row_ok ? __bfloat162float(p.gate[row * p.ld_gate + h]) : 0.f, p.fin);
          }
#pragma unroll
          for (int c = 0; c < VN / 32; ++c) {
            float d[32];
            load_diff(c, d);
            if (row_ok && p.diff) {
              float* dst = p.diff + (row * p.H + h) * p.V + v0 + c * 32;
#pragma unroll
              for (int i = 0; i < 32; i += 4)
                if (c * 32 + i < cols) *reinterpret_cast<float4*>(dst + i) = make_float4(d[i], d[i + 1], d[i + 2], d[i + 3]);
            } else if (row_ok) {
              __nv_bfloat16* dst = p.out + row * p.ldo + h * p.V + c * 32;
#pragma unroll
              for (int i = 0; i < 32; i += 8) {
                if (c * 32 + i < cols) {
                  uint4 u;
                  uint32_t* w = reinterpret_cast<uint32_t*>(&u);
#pragma unroll
                  for (int k = 0; k < 4; ++k) {
                    __nv_bfloat162 t = __floats2bfloat162_rn(d[i + 2 * k] * f, d[i + 2 * k + 1] * f);
                    w[k] = *reinterpret_cast<uint32_t*>(&t);
                  }
                  *reinterpret_cast<uint4*>(dst + i) = u;
                }
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

template <int VN>
int launch(const CUtensorMap& q, const CUtensorMap& k, const CUtensorMap& v, const Params& p, dim3 grid, size_t smem,
           cudaStream_t stream) {
  static PerDeviceOnce once_;
  bool& configured = once_.slot();
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(diff_prefill_kernel<VN>, cudaFuncAttributeMaxDynamicSharedMemorySize, 232448);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  diff_prefill_kernel<VN><<<grid, NTHREADS, smem, stream>>>(q, k, v, p);
  return (int)cudaGetLastError();
}

}  // namespace diffattn
}  // namespace b200

using namespace b200;

// Column slices of the value head the tile kernel uses (more than one: it needs the fp32 difference buffer); 0: sizes it
// does not cover.  D: query / key vector, V: value head, both multiples of 16.
extern "C" int b200_attn_diff_prefill_slices(int H, int G, int D, int V, int block_size) {
  if (H <= 0 || G <= 0 || H % G || D <= 0 || D % 16 || D > 256 || V <= 0 || V % 16 || V > 1024) return 0;
  if (block_size != 16 && block_size != 32 && block_size != 64 && block_size != 128) return 0;
  return (V + 127) / 128;
}

// q: [q_rows, H, 2, D] bf16; caches [num_blocks * block_size, G * 2 * D], [.., G * V] bf16; entries of B sequences, rows
// [q_start, q_start + q_len) each; out [q_rows, ldo] bf16 (head h at columns h * V), or diff [q_rows, H, V] fp32 when the
// value head is sliced.
extern "C" int b200_attn_diff_prefill(const void* q, const void* k_cache, const void* v_cache, void* out, float* diff,
                                      const void* gate, int ld_gate, const int* block_table, const int* seq, const int* q_start,
                                      const int* q_len, const int* kv_len, int batch, int max_q_len, int q_rows, int max_blocks,
                                      int num_blocks, int block_size, int H, int G, int D, int V, int vdim, int ldo, float scale,
                                      float lambda, float keep, float eps, int* status, cudaStream_t stream) {
  using namespace b200::diffattn;
  const int slices = b200_attn_diff_prefill_slices(H, G, D, V, block_size);
  if (slices < 1 || batch <= 0 || batch > 65535 || max_q_len <= 0 || q_rows <= 0 || (slices > 1) != (diff != nullptr) ||
      (!diff && (!out || !gate || (ldo & 7) || ldo < H * V)) || vdim <= 0 || vdim > V || (long long)H * slices > 65535)
    return -ERR_BAD_ARG;
  Params p;
  p.slabs = (D + 63) / 64;
  p.stages = (BUDGET - 2 * p.slabs * ATOM) / ATOM;
  if (p.stages > MAX_STAGES) p.stages = MAX_STAGES;
  const int VN = V >= 128 ? 128 : (V + 31) / 32 * 32, VS = (VN + 63) / 64;
  p.stages &= ~1;
  if (p.stages < VS + 2) return -ERR_BAD_ARG;
  const size_t smem = (size_t)(2 * p.slabs + p.stages) * ATOM + 1024 + 512 + 1024;
  CUtensorMap tmQ, tmK, tmV;
  const uint64_t QW = (uint64_t)H * 2 * D, KW = (uint64_t)G * 2 * D, VW = (uint64_t)G * V, kv_rows = (uint64_t)num_blocks * block_size;
  bool ok = make_tmap_2d(&tmQ, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, q, q_rows, QW, QW * 2, BQ, 64, CU_TENSOR_MAP_SWIZZLE_128B);
  ok = ok && make_tmap_2d(&tmK, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, k_cache, kv_rows, KW, KW * 2, block_size, 64,
                          CU_TENSOR_MAP_SWIZZLE_128B);
  ok = ok && make_tmap_2d(&tmV, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, v_cache, kv_rows, VW, VW * 2, block_size, 64,
                          CU_TENSOR_MAP_SWIZZLE_128B);
  if (!ok) return -ERR_BAD_ARG;
  p.block_table = block_table; p.seq = seq; p.q_start = q_start; p.q_len = q_len; p.kv_len = kv_len;
  p.max_blocks = max_blocks; p.block_size = block_size; p.H = H; p.G = G; p.D = D; p.V = V; p.v_slices = slices;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.out = reinterpret_cast<__nv_bfloat16*>(out); p.diff = diff; p.gate = reinterpret_cast<const __nv_bfloat16*>(gate);
  p.ldo = ldo; p.ld_gate = ld_gate; p.status = status;
  p.fin = DiffFinish{lambda, keep, eps, 1.f / (float)vdim};
  const dim3 grid((max_q_len + BQ - 1) / BQ, H * slices, batch);
  switch (VN) {
    case 32: return launch<32>(tmQ, tmK, tmV, p, grid, smem, stream);
    case 64: return launch<64>(tmQ, tmK, tmV, p, grid, smem, stream);
    case 96: return launch<96>(tmQ, tmK, tmV, p, grid, smem, stream);
    default: return launch<128>(tmQ, tmK, tmV, p, grid, smem, stream);
  }
}
