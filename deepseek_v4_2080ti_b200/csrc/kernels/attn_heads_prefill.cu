// Causal flash-attention prefill over contiguous keys and values, every head with keys of its own made of two parts, sm_100a:
// D columns per head and R columns shared by all heads (the prompt form of latent attention: the latents of a context are
// expanded into keys and values by one GEMM, the rotated key part stays as it is cached).
//
// One CTA = 256 query rows of one head as two streams of 128 that share every key and value slab; the streams keep the tensor
// core and the exponential units busy in turn.  Warp roles:
//   warps 0-3, 4-7: softmax of stream 0 and 1 - one query row per thread, online maximum / sum in the exp2 domain, P as bf16
//             back into the tensor memory its scores came from, lazy rescale of the stream's O;
//   warp 8  : TMA producer.  Keys, shared key part and values travel as slabs of [128 tokens x 64 columns] through one ring;
//   warp 9  : tcgen05.mma issuer - per tile P0 V, S0 of the next tile, P1 V, S1 of the next tile.
// Tensor memory: S0 | S1 (128 columns each) and O0 | O1 (up to 128 columns each).  Wider values are cut into column slices,
// one CTA each.  A slab reads on past its part's columns; the products stop at them.  The two value slabs of a tile have to be
// neighbours in the ring: where they would wrap, a stage is left out (handed through empty).
// All mbarrier waits are bounded and unwind through the common exit.
#include <cuda_bf16.h>
#include "per_device.h"
#include "../ptx/sm100.cuh"
#include "tma_host.h"
#include "ops.h"

namespace b200 {
namespace headsattn {

constexpr int BQ = 128;         // query rows per stream
constexpr int BKV = 128;        // keys per tile
constexpr int ATOM = 16384;     // bytes of one [128 x 64] bf16 swizzled slab
constexpr int NTHREADS = 384;   // three warpgroups; the third has the two issuing roles and gives its registers up
constexpr int MAX_STAGES = 12;
constexpr int BUDGET = 232448 - 1024 /* alignment */ - 512 /* barriers */;

struct Params {
  const int* q_start;      // [B] first query row of the entry
  const int* q_len;        // [B]
  const int* kv_len;       // [B] context length including the entry's own tokens
  const int* kv_start;     // [B] first row of the entry's context in the expanded buffers
  int D, R, V;             // columns per head: keys, shared key part, values (multiples of 16)
  int head0;               // first head of this launch (queries and output; keys and values start at column 0)
  int slabs_d, slabs_r, stages, slice, v_slices;
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
// where none has a ragged end (loops the issuer has unrolled), or 0.
template <int VN, int SL>
__global__ void __launch_bounds__(NTHREADS, 1)
heads_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmKV,
                     const __grid_constant__ CUtensorMap tmR, Params p) {
  constexpr uint32_t idesc_qk = umma_idesc_bf16(128, 128);
  constexpr uint32_t idesc_pv = umma_idesc_bf16(128, VN) | (1u << 16);   // B is MN-major
  constexpr int VS = (VN + 63) / 64;                                     // slabs of the value slice
  extern __shared__ uint8_t smem_base[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_base) + 1023) & ~uintptr_t(1023));
  const int slabs = SL ? SL : p.slabs_d + p.slabs_r, stages = p.stages;
  uint8_t* sQ = smem;                                   // [2 streams][slabs] atoms
  uint8_t* sR = sQ + 2 * slabs * ATOM;                  // ring of slabs
  uint64_t* bars = reinterpret_cast<uint64_t*>(sR + stages * ATOM);
  uint64_t* r_full = bars;                   // MAX_STAGES
  uint64_t* r_empty = bars + MAX_STAGES;     // MAX_STAGES
  uint64_t* q_full = bars + 2 * MAX_STAGES;
  uint64_t* s_full = q_full + 1;             // per stream
  uint64_t* p_full = q_full + 3;
  uint64_t* pv_done = q_full + 5;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(q_full + 7);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0), lane = threadIdx.x & 31;   // uniform: the issuer depends on it
  const int b = blockIdx.z, qt = (int)gridDim.x - 1 - (int)blockIdx.x;   // long tiles first
  const int hl = blockIdx.y / p.v_slices, v0 = (blockIdx.y % p.v_slices) * p.slice;
  const int h = p.head0 + hl;
  const int q_len = p.q_len[b], kv_len = p.kv_len[b];
  const int q0 = qt * 2 * BQ;
  if (q0 >= q_len) return;                   // uniform per CTA, before any barrier / TMEM use
  const int q_row0 = p.q_start[b] + q0;
  const int pos0 = kv_len - q_len + q0;      // position of the first query row
  const bool two = q0 + BQ < q_len;          // the second stream has rows
  const int n_tiles0 = __shfl_sync(0xffffffffu, (min(kv_len, pos0 + BQ) + BKV - 1) / BKV, 0);
  const int n_tiles1 = __shfl_sync(0xffffffffu, two ? (min(kv_len, pos0 + 2 * BQ) + BKV - 1) / BKV : 0, 0);
  const int n_tiles = max(n_tiles0, n_tiles1);

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
      tma_prefetch_desc(&tmKV);
      tma_prefetch_desc(&tmR);
      const int streams = two ? 2 : 1, q_col = h * (p.D + p.R);
      mbar_expect_tx(q_full, streams * slabs * ATOM);
      for (int m = 0; m < streams; ++m)
        for (int s = 0; s < slabs; ++s)
          tma_load_2d(sQ + (m * slabs + s) * ATOM, &tmQ, q_full, s < p.slabs_d ? q_col + s * 64 : q_col + p.D + (s - p.slabs_d) * 64,
                      q_row0 + m * BQ);
      const int row0 = p.kv_start[b], kv_col = hl * (p.D + p.V);
      Ring r = {0, 1};
      bool ok = true;
      for (int j = 0; ok && j < n_tiles && !*abort_flag; ++j) {
        auto slab = [&](const CUtensorMap* tm, int x) {
          if (!mbar_wait(&r_empty[r.st], r.ph)) return false;
          mbar_expect_tx(&r_full[r.st], ATOM);
          tma_load_2d(sR + r.st * ATOM, tm, &r_full[r.st], x, row0 + j * BKV);
          r.next(stages);
          return true;
        };
        for (int s = 0; ok && s < p.slabs_d; ++s) ok = slab(&tmKV, kv_col + s * 64);
        for (int s = 0; ok && s < p.slabs_r; ++s) ok = slab(&tmR, s * 64);
        if (ok && VS == 2 && r.st == stages - 1) {
          ok = mbar_wait(&r_empty[r.st], r.ph);
          if (ok) mbar_arrive(&r_full[r.st]);
          r.next(stages);
        }
#pragma unroll
        for (int s = 0; s < VS; ++s)
          if (ok) ok = slab(&tmKV, kv_col + p.D + v0 + s * 64);
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
      wait(q_full, 0);
      const uint64_t ring = umma_desc_sw128(sR), dq0 = umma_desc_sw128(sQ);
      const int steps_d = (p.D - (p.slabs_d - 1) * 64) / 16, steps_r = (p.R - (p.slabs_r - 1) * 64) / 16;
      // scores of a tile whose key slabs begin at ring position r (by value: both streams walk the same slabs); the tile's
      // last stream gives them back
      auto issue_s = [&](const int m, Ring r, bool last) {
#pragma unroll
        for (int s = 0; s < (SL ? SL : slabs); ++s) {
          if (!wait(&r_full[r.st], r.ph)) return;
          tc_fence_after();
          const uint64_t dk = ring + r.st * (ATOM >> 4), dq = dq0 + (m * slabs + s) * (ATOM >> 4);
          const int steps = SL ? 4 : s == p.slabs_d - 1 ? steps_d : s == slabs - 1 ? steps_r : 4;
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
      if (ok) issue_s(0, k, !two);
      if (ok && two) issue_s(1, k, true);
      for (int j = 0; ok && j < n_tiles && !*abort_flag; ++j) {
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
          const int mine = m ? n_tiles1 : n_tiles0;
          if (j < mine) {
            if (!ok || !wait(&p_full[m], j & 1)) break;
            Ring w = v;
#pragma unroll
            for (int s = 0; s < VS; ++s) {
              if (ok) wait(&r_full[w.st], w.ph);
              w.next(stages);
            }
            if (!ok) break;
            tc_fence_after();
            const uint64_t dv = desc_mn_sw128(sR, ATOM, 1024) + v.st * (ATOM >> 4);
            umma_bf16_ts_warp(on, tmem + 256 + m * 128, tmem + m * 128, dv, idesc_pv, j ? 1u : 0u);
#pragma unroll
            for (int kk = 1; kk < 8; ++kk)
              umma_bf16_ts_warp(on, tmem + 256 + m * 128, tmem + m * 128 + kk * 8, dv + kk * 128, idesc_pv, 1u);
            umma_commit_warp(on, &pv_done[m]);
            if (m == (two ? 1 : 0)) {
#pragma unroll
              for (int s = 0; s < VS; ++s) umma_commit_warp(on, &r_empty[v.st + s]);
            }
          }
          // the second stream sees at least as many tiles as the first, so it is the one that gives slabs back
          if (j + 1 < mine) issue_s(m, k, m == (two ? 1 : 0));
        }
      }
      if (!ok && lane == 0) { atomicExch(p.status, ERR_WAIT_TMA); *abort_flag = 1; }
    }
  } else {
    asm volatile("setmaxnreg.inc.sync.aligned.u32 216;");
    const int m = warp >> 2;                 // stream
    const int r = (warp & 3) * 32 + lane;    // query row in the tile == TMEM lane
    const int limit = pos0 + m * BQ + r;     // last visible key of this row
    const int my_tiles = m ? n_tiles1 : n_tiles0;
    const uint32_t lane_off = uint32_t((warp & 3) * 32) << 16;
    const uint32_t tS = tmem + m * 128 + lane_off, tO = tmem + 256 + m * 128 + lane_off;
    float m_run = -INFINITY, l_run = 0.f;
    bool alive = true;
    for (int j = 0; j < my_tiles; ++j) {
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
          const int kx = half * 64 + 2 * i;
          const float e0 = exp2f(fmaf(__uint_as_float(sv[kx >> 5][kx & 31]), p.scale_log2, -m_run));
          const float e1 = exp2f(fmaf(__uint_as_float(sv[kx >> 5][(kx & 31) + 1]), p.scale_log2, -m_run));
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
int launch_as(const CUtensorMap& q, const CUtensorMap& kv, const CUtensorMap& r, const Params& p, dim3 grid, size_t smem,
              cudaStream_t stream) {
  static PerDeviceOnce once_;
  bool& configured = once_.slot();
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(heads_prefill_kernel<VN, SL>, cudaFuncAttributeMaxDynamicSharedMemorySize, 232448);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  heads_prefill_kernel<VN, SL><<<grid, NTHREADS, smem, stream>>>(q, kv, r, p);
  return (int)cudaGetLastError();
}

template <int VN>
int launch(const CUtensorMap& q, const CUtensorMap& kv, const CUtensorMap& r, const Params& p, dim3 grid, size_t smem,
           cudaStream_t stream) {
  if (p.D % 64 == 0 && p.R % 64 == 0) {
    if (p.slabs_d + p.slabs_r == 2) return launch_as<VN, 2>(q, kv, r, p, grid, smem, stream);
    if (p.slabs_d + p.slabs_r == 3) return launch_as<VN, 3>(q, kv, r, p, grid, smem, stream);
  }
  return launch_as<VN, 0>(q, kv, r, p, grid, smem, stream);
}

}  // namespace headsattn
}  // namespace b200

using namespace b200;

// Sizes the kernel covers: D, R, V multiples of 16 (R may be 0), at most four 64-column slabs of keys.
extern "C" int b200_attn_heads_prefill_supported(int H, int D, int R, int V) {
  return H > 0 && D > 0 && R >= 0 && V > 0 && !(D % 16) && !(R % 16) && !(V % 16) && (D + 63) / 64 + (R + 63) / 64 <= 4;
}

// q [q_rows, ldq] bf16 (head h: D + R columns at h * (D + R)); kv [kv_rows, H * (D + V)] bf16 of the `H` heads from head0 on;
// key [kv_rows, ld_key] the shared part (ld_key >= 64 ceil(R / 64)); entry b: query rows [q_start, q_start + q_len), context rows
// [kv_start, kv_start + kv_len).  Rows of kv behind a context must be finite.
extern "C" int b200_attn_heads_prefill(const void* q, int ldq, const void* kv, const void* key, int ld_key, void* out, int ldo,
                                       const int* q_start, const int* q_len, const int* kv_len, const int* kv_start, int batch,
                                       int max_q_len, int q_rows, int kv_rows, int head0, int H, int D, int R, int V, float scale,
                                       int* status, cudaStream_t stream) {
  using namespace b200::headsattn;
  if (!b200_attn_heads_prefill_supported(H, D, R, V) || batch <= 0 || batch > 65535 || max_q_len <= 0 || q_rows <= 0 || kv_rows <= 0 ||
      head0 < 0 || (ldq & 7) || ldq < (head0 + H) * (D + R) || (ldo & 7) || ldo < (head0 + H) * V ||
      (R && (!key || (ld_key & 7) || ld_key < (R + 63) / 64 * 64)))
    return -ERR_BAD_ARG;
  Params p;
  p.slabs_d = (D + 63) / 64;
  p.slabs_r = (R + 63) / 64;
  const int slabs = p.slabs_d + p.slabs_r;
  p.slice = slabs == 4 ? 64 : 128;           // four key slabs leave room for one value slab in flight
  const int VN = V >= p.slice ? p.slice : (V + 31) / 32 * 32, VS = (VN + 63) / 64;
  p.v_slices = (V + p.slice - 1) / p.slice;
  p.stages = (BUDGET - 2 * slabs * ATOM) / ATOM;
  if (p.stages > MAX_STAGES) p.stages = MAX_STAGES;
  if (p.stages < slabs + VS + (VS == 2) || (long long)H * p.v_slices > 65535) return -ERR_BAD_ARG;
  const size_t smem = (size_t)(2 * slabs + p.stages) * ATOM + 1024 + 512;
  CUtensorMap tmQ, tmKV, tmR;
  const uint64_t KW = (uint64_t)H * (D + V);
  bool ok = make_tmap_2d(&tmQ, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, q, q_rows, ldq, (uint64_t)ldq * 2, BQ, 64, CU_TENSOR_MAP_SWIZZLE_128B);
  ok = ok && make_tmap_2d(&tmKV, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, kv, kv_rows, KW, KW * 2, BKV, 64, CU_TENSOR_MAP_SWIZZLE_128B);
  if (R)
    ok = ok && make_tmap_2d(&tmR, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, key, kv_rows, ld_key, (uint64_t)ld_key * 2, BKV, 64,
                            CU_TENSOR_MAP_SWIZZLE_128B);
  else
    tmR = tmKV;
  if (!ok) return -ERR_BAD_ARG;
  p.q_start = q_start; p.q_len = q_len; p.kv_len = kv_len; p.kv_start = kv_start;
  p.D = D; p.R = R; p.V = V; p.head0 = head0;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.out = reinterpret_cast<__nv_bfloat16*>(out); p.ldo = ldo; p.status = status;
  const dim3 grid((max_q_len + 2 * BQ - 1) / (2 * BQ), H * p.v_slices, batch);
  switch (VN) {
    case 32: return launch<32>(tmQ, tmKV, tmR, p, grid, smem, stream);
    case 64: return launch<64>(tmQ, tmKV, tmR, p, grid, smem, stream);
    case 96: return launch<96>(tmQ, tmKV, tmR, p, grid, smem, stream);
    default: return launch<128>(tmQ, tmKV, tmR, p, grid, smem, stream);
  }
}
