// Latent attention of single query rows (attn_latent_rows.cu) on the 5th-generation tensor cores, sm_100a: bf16, latents up to
// 512 wide.  One CTA = one row, N heads and one slice of the row's keys; it streams the cache rows once, in tiles of 64 keys by
// TMA, and both products read them from there:
//
//   S   [heads x 64 keys]  = Q K^T        the queries stay in tensor memory as the 128-lane operand, of which N lanes are real
//                                         (what the others hold ends in lanes nobody reads): only the keys are fetched
//   O^T [latent x heads]  += V^T P^T      the tile itself, read with its columns as rows, is the 128-row operand; so the sums
//                                         of 512 latent columns and N heads fit tensor memory
//
// The products cost the tensor core the same for N heads as for one, and less time than the tile takes to arrive.  A tile
// travels as units of 128 columns through one ring; a unit is given back by the last product that reads it.
// Warp roles: 0 softmax (a thread per head); 0-3 rescaling of O^T (a thread per latent column) and epilogue; 4 TMA producer;
// 5 issuer: scores of the next tile before the sums of this one.
// Tensor memory: queries (32 columns per 64 of a cache row), scores (64), N columns per 128 columns of the latent.
// All mbarrier waits are bounded and unwind through the common exit.
#include <cuda_bf16.h>
#include "launch.h"
#include "per_device.h"
#include "../ptx/sm100.cuh"
#include "tma_host.h"
#include "ops.h"

namespace b200 {
namespace latdec {

constexpr int KT = 64;           // keys per tile
constexpr int SLAB = KT * 128;   // bytes of one [64 keys x 64 columns] bf16 swizzled slab
constexpr int NTHREADS = 192;
constexpr int UNIT = 2 * SLAB;   // 128 columns: the rows of one V^T operand
constexpr int MAX_UNITS = 24;
constexpr int FIXED = 1024 /* alignment */ + 1024 /* barriers, statistics */;

struct Params {
  const int* block_table;        // [sequences, max_blocks]
  const int* seq;                // [rows] table row of each query row (null: row i)
  const int* positions;          // [rows]
  int max_blocks, bs, box, H, C, D, slabs, units, splits;      // box: rows per copy; units: of the ring
  float scale_log2;
  const __nv_bfloat16* q;        // [rows, H, D]
  __nv_bfloat16* out;            // [rows, H, C]
  float *partial, *stats;        // [rows, H, splits, C] and [rows, H, splits, 2], or null: one slice
  int* status;
};

__device__ __forceinline__ uint64_t desc_mn_sw128(const void* p, uint32_t lbo, uint32_t sbo) {
  uint64_t d = 0;
  d |= (uint64_t)((smem_u32(p) & 0x3FFFF) >> 4);
  d |= (uint64_t)(lbo >> 4) << 16;
  d |= (uint64_t)(sbo >> 4) << 32;
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;
  return d;
}
__device__ __forceinline__ void named_sync() { asm volatile("bar.sync 1, 128;" ::: "memory"); }
// Does any of the 128 threads say so?
__device__ __forceinline__ bool named_any(bool v) {
  uint32_t r;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.b32 p, %1, 0;\n\t"
      "bar.red.or.pred q, 1, 128, p;\n\t"
      "selp.b32 %0, 1, 0, q;\n\t}\n"
      : "=r"(r)
      : "r"((uint32_t)v)
      : "memory");
  return r != 0;
}

// SL: 64-column slabs of a cache row where it has no ragged end (loops the issuer has unrolled), or 0.
template <int N, int SL>
__global__ void __launch_bounds__(NTHREADS, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tmK, Params p) {
  constexpr uint32_t idesc_s = umma_idesc_bf16(128, KT);
  constexpr uint32_t idesc_o = umma_idesc_bf16(128, N) | (1u << 15);     // A is MN-major
  static_assert(N <= 32, "the heads of a CTA are the lanes of warp 0");
  extern __shared__ uint8_t smem_base[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_base) + 1023) & ~uintptr_t(1023));
  const int slabs = SL ? SL : p.slabs, ring = p.units, units = (slabs + 1) / 2, mt = (p.C + 127) / 128;   // units of a tile; of its latent
  uint8_t* sP = smem;                                   // [2][N rows x 64 keys]
  uint8_t* sK = sP + 2 * N * 128;                       // [ring] units
  float* s_alpha = reinterpret_cast<float*>(sK + ring * UNIT);    // [N] factors, later reciprocal sums
  uint64_t* full = reinterpret_cast<uint64_t*>(s_alpha + 64);
  uint64_t* empty = full + MAX_UNITS;
  uint64_t* q_full = empty + MAX_UNITS;
  uint64_t* s_full = q_full + 1;
  uint64_t* s_read = q_full + 2;
  uint64_t* p_full = q_full + 3;                        // per buffer of probabilities
  uint64_t* pv_done = q_full + 5;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(q_full + 7);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0), lane = threadIdx.x & 31;
  const int split = blockIdx.x, h0 = blockIdx.y * N, b = blockIdx.z;
  if (threadIdx.x == 0) {
    for (int i = 0; i < ring; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    mbar_init(q_full, 32);
    mbar_init(s_full, 1);
    mbar_init(s_read, 32);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&p_full[i], 128);
      mbar_init(&pv_done[i], 1);
    }
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 5) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = __shfl_sync(0xffffffffu, *tmem_slot, 0);
  const uint32_t S_COL = slabs * 32, O_COL = S_COL + KT;      // behind the queries
  pdl_launch_dependents();
  pdl_wait();

  const int n_keys = p.positions[b] + 1;
  const int per = ((n_keys + p.splits - 1) / p.splits + KT - 1) / KT * KT;
  const int k0 = split * per, k1 = min(n_keys, k0 + per);
  const int nt = __shfl_sync(0xffffffffu, k0 < k1 ? (k1 - k0 + KT - 1) / KT : 0, 0);      // a slice may be empty

  if (warp == 4) {
    if (lane == 0 && nt > 0) {
      tma_prefetch_desc(&tmK);
      const int* bt = p.block_table + (size_t)(p.seq ? p.seq[b] : b) * p.max_blocks;
      const int boxes = KT / p.box;
      bool ok = true;
      int st = 0;
      uint32_t ph = 1;
      for (int t = 0; t < nt && !*abort_flag; ++t) {
        int row[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int key = k0 + t * KT + i * p.box;
          row[i] = i < boxes && key < n_keys ? bt[key / p.bs] * p.bs + key % p.bs : 0;      // behind the context: page 0
        }
        for (int u = 0; u < units; ++u) {
          ok = mbar_wait(&empty[st], ph);
          if (!ok) break;
          const int n = min(2, slabs - 2 * u);
          mbar_expect_tx(&full[st], n * SLAB);
          for (int s = 0; s < n; ++s)
#pragma unroll
            for (int i = 0; i < 4; ++i)
              if (i < boxes)
                tma_load_2d(sK + st * UNIT + s * SLAB + i * p.box * 128, &tmK, &full[st], (2 * u + s) * 64, row[i]);
          if (++st == ring) { st = 0; ph ^= 1; }
        }
        if (!ok) break;
      }
      if (!ok) { atomicExch(p.status, ERR_WAIT_STAGE); *abort_flag = 1; }
    }
  } else if (warp == 5) {
    if (nt > 0) {
      // The whole warp walks the loop, and one elected lane issues.
      bool ok = true;
      auto wait = [&](uint64_t* bar, uint32_t parity) {
        ok = __all_sync(0xffffffffu, mbar_wait(bar, parity));
        return ok;
      };
      const int last_steps = SL ? 4 : (p.D - (slabs - 1) * 64) / 16;
      const uint32_t on = elect_one();
      const uint64_t dk0 = umma_desc_sw128(sK), dv0 = desc_mn_sw128(sK, SLAB, 1024);
      int ks = 0, ps = 0;                    // ring positions of the next scores' and of the next sums' tile
      uint32_t kp = 0;
      auto issue_s = [&](int t) {
        const uint32_t d = tmem + S_COL;
        if (t > 0 && !wait(s_read, (t - 1) & 1)) return;       // the scores of the tile before are in registers
#pragma unroll
        for (int u = 0; u < (SL ? (SL + 1) / 2 : units); ++u) {
          if (!wait(&full[ks], kp)) return;
          tc_fence_after();
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const int s = 2 * u + i;
            if (s < slabs) {
              const uint32_t q = tmem + s * 32;
              const uint64_t dk = dk0 + ks * (UNIT >> 4) + i * (SLAB >> 4);
              const int steps = s + 1 < slabs ? 4 : last_steps;
              umma_bf16_ts_warp(on, d, q, dk, idesc_s, s ? 1u : 0u);
#pragma unroll
              for (int kk = 1; kk < 4; ++kk)
                if (kk < steps) umma_bf16_ts_warp(on, d, q + kk * 8, dk + 2 * kk, idesc_s, 1u);
            }
          }
          if (u >= mt) umma_commit_warp(on, &empty[ks]);       // no part of the latent
          if (u + 1 == units) umma_commit_warp(on, s_full);
          if (++ks == ring) { ks = 0; kp ^= 1; }
        }
      };
      if (wait(q_full, 0)) {
        tc_fence_after();
        issue_s(0);
      }
      for (int t = 0; ok && t < nt && !*abort_flag; ++t) {
        if (t + 1 < nt) issue_s(t + 1);
        if (!ok || !wait(&p_full[t & 1], (t >> 1) & 1)) break;
        tc_fence_after();
        const uint64_t dp = umma_desc_sw128(sP + (t & 1) * N * 128);
        for (int i = 0; i < mt; ++i) {
          const int at = ps + i < ring ? ps + i : ps + i - ring;
          const uint64_t dv = dv0 + at * (UNIT >> 4);
#pragma unroll
          for (int kk = 0; kk < KT / 16; ++kk)
            umma_bf16_ss_warp(on, tmem + O_COL + i * N, dv + kk * 128, dp + 2 * kk, idesc_o, t || kk ? 1u : 0u);
          umma_commit_warp(on, &empty[at]);
          if (i + 1 == mt) umma_commit_warp(on, &pv_done[t & 1]);
        }
        ps += units;
        if (ps >= ring) ps -= ring;
      }
      if (!ok && lane == 0) { atomicExch(p.status, ERR_WAIT_TMA); *abort_flag = 1; }
    }
  } else {
    const int r = threadIdx.x;               // head of the group, and lane of tensor memory
    const uint32_t lane_off = uint32_t(warp * 32) << 16;
    const bool row_warp = warp == 0, row = r < N;
    if (row_warp && nt > 0) {
      // a lane's query as packed pairs, zeros behind its end and for heads that do not exist
      const __nv_bfloat16* src = p.q + ((size_t)b * p.H + h0 + r) * p.D;
      const bool real = row && h0 + r < p.H;
      for (int s = 0; s < slabs; ++s) {
        uint32_t w[32];
#pragma unroll
        for (int c = 0; c < 8; ++c) {
          uint4 u = make_uint4(0, 0, 0, 0);
          if (real && s * 64 + c * 8 < p.D) u = *reinterpret_cast<const uint4*>(src + s * 64 + c * 8);
          w[4 * c] = u.x; w[4 * c + 1] = u.y; w[4 * c + 2] = u.z; w[4 * c + 3] = u.w;
        }
        tmem_st_32x32(tmem + s * 32, w);
      }
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(q_full);
    }
    float m_run = -INFINITY, l_run = 0.f;
    bool alive = true;
    for (int t = 0; t < nt; ++t) {
      bool ok = true;                        // only the warp that reads the scores waits for them
      uint32_t sv[2][32];
      float alpha = 1.f;
      if (row_warp) {
        ok = mbar_wait(s_full, t & 1);
        if (t >= 2) ok = ok && mbar_wait(&pv_done[t & 1], ((t - 2) >> 1) & 1);     // the probabilities' buffer is free
        tc_fence_after();
        tmem_ld_32x32(tmem + S_COL, sv[0]);
        tmem_ld_32x32(tmem + S_COL + 32, sv[1]);
        tmem_ld_wait();
        tc_fence_before();
        mbar_arrive(s_read);
        const int kmax = k1 - 1 - k0 - t * KT;
        if (kmax < KT - 1) {
#pragma unroll
          for (int i = 0; i < KT; ++i)
            if (i > kmax) sv[i >> 5][i & 31] = 0xff800000u;      // -inf
        }
        float mx[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) mx[i] = __uint_as_float(sv[0][i]);
#pragma unroll
        for (int i = 4; i < KT; ++i) mx[i & 3] = fmaxf(mx[i & 3], __uint_as_float(sv[i >> 5][i & 31]));
        const float m_new = fmaxf(m_run, p.scale_log2 * fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])));   // a tile has a visible key
        if (t == 0) {
          m_run = m_new;
        } else if (m_new > m_run + 8.f) {
          alpha = exp2f(m_run - m_new);
          l_run *= alpha;
          m_run = m_new;
        }
      }
      // lanes behind the real heads hold nothing: their factor is not looked at
      if (row) s_alpha[r] = alpha;
      const bool grow = named_any((row && alpha != 1.f) || !ok);
      if (grow) {
        // either a factor or a wait that gave up: O^T may be rescaled once the sums of the tile before are complete
        ok = ok && mbar_wait(&pv_done[(t - 1) & 1], ((t - 1) >> 1) & 1);
        if (named_any(!ok) || *abort_flag) { alive = false; break; }
        tc_fence_after();
        for (int i = 0; i < mt; ++i)
#pragma unroll
          for (int c = 0; c < N; c += 16) {
            uint32_t v[16];
            tmem_ld_32x16(tmem + lane_off + O_COL + i * N + c, v);
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 16; ++j) v[j] = __float_as_uint(__uint_as_float(v[j]) * s_alpha[c + j]);
            asm volatile(
                "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};"
                ::"r"(tmem + lane_off + O_COL + i * N + c), "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]),
                "r"(v[7]), "r"(v[8]), "r"(v[9]), "r"(v[10]), "r"(v[11]), "r"(v[12]), "r"(v[13]), "r"(v[14]), "r"(v[15])
                : "memory");
          }
        tmem_st_wait();
      }
      if (row) {
        float lsum[4] = {0.f, 0.f, 0.f, 0.f};
        uint8_t* prow = sP + (t & 1) * N * 128 + r * 128;
#pragma unroll
        for (int c = 0; c < 8; ++c) {        // 8 keys = 16 bytes, at their swizzled place
          uint4 u;
          uint32_t* w = reinterpret_cast<uint32_t*>(&u);
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const int k = c * 8 + 2 * j;
            const float e0 = exp2f(fmaf(__uint_as_float(sv[k >> 5][k & 31]), p.scale_log2, -m_run));
            const float e1 = exp2f(fmaf(__uint_as_float(sv[k >> 5][(k & 31) + 1]), p.scale_log2, -m_run));
            lsum[j] += e0 + e1;
            const __nv_bfloat162 x = __floats2bfloat162_rn(e0, e1);
            w[j] = *reinterpret_cast<const uint32_t*>(&x);
          }
          *reinterpret_cast<uint4*>(prow + ((c ^ (r & 7)) << 4)) = u;
        }
        l_run += (lsum[0] + lsum[1]) + (lsum[2] + lsum[3]);
      }
      fence_proxy_async_smem();
      tc_fence_before();
      mbar_arrive(&p_full[t & 1]);
    }
    if (alive && nt > 0) {
      const bool ok = mbar_wait(&pv_done[(nt - 1) & 1], ((nt - 1) >> 1) & 1);
      alive = !named_any(!ok) && !*abort_flag;
      tc_fence_after();
    }
    if (alive) {
      const bool real = row && h0 + r < p.H;
      const size_t at = ((size_t)b * p.H + h0 + r) * p.splits + split;
      if (real && p.partial) {
        p.stats[2 * at] = m_run;
        p.stats[2 * at + 1] = l_run;
      }
      if (row) s_alpha[r] = p.partial ? 1.f : 1.f / l_run;
      named_sync();
      for (int i = 0; i < mt; ++i) {
        const int col = i * 128 + r;
#pragma unroll
        for (int c = 0; c < N; c += 16) {
          uint32_t v[16];
          if (nt > 0) {
            tmem_ld_32x16(tmem + lane_off + O_COL + i * N + c, v);
            tmem_ld_wait();
          }
          if (col < p.C) {
#pragma unroll
            for (int j = 0; j < 16; ++j) {
              const int h = h0 + c + j;
              if (h >= p.H) break;
              const float f = nt > 0 ? __uint_as_float(v[j]) * s_alpha[c + j] : 0.f;
              if (p.partial) p.partial[(((size_t)b * p.H + h) * p.splits + split) * p.C + col] = f;
              else p.out[((size_t)b * p.H + h) * p.C + col] = __float2bfloat16(f);
            }
          }
        }
      }
    } else {
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

inline size_t smem_bytes(int N, int ring) { return (size_t)2 * N * 128 + (size_t)ring * UNIT + FIXED; }
inline int heads_of(int H) { return H <= 16 ? 16 : 32; }
// Units of the ring; 0: the sums' units of one tile and all of the next do not fit, or tensor memory does not hold the queries.
inline int ring_of(int N, int C, int slabs) {
  int n = MAX_UNITS;
  while (n > 0 && smem_bytes(N, n) > 232448) --n;
  return n >= (C + 127) / 128 + (slabs + 1) / 2 && slabs * 32 + KT + (C + 127) / 128 * N <= 512 ? n : 0;
}

template <int N, int SL>
int launch_as(const CUtensorMap& k, const Params& p, int rows, cudaStream_t stream) {
  static PerDeviceOnce once_;
  bool& configured = once_.slot();
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<N, SL>, cudaFuncAttributeMaxDynamicSharedMemorySize, 232448);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  return (int)launch_pdl(latent_decode_kernel<N, SL>, dim3(p.splits, (p.H + N - 1) / N, rows), dim3(NTHREADS),
                         smem_bytes(N, p.units), stream, k, p);
}

template <int N>
int launch(const CUtensorMap& k, const Params& p, int rows, cudaStream_t stream) {
  return p.D == 576 ? launch_as<N, 9>(k, p, rows, stream) : launch_as<N, 0>(k, p, rows, stream);
}

}  // namespace latdec
}  // namespace b200

using namespace b200;

// Heads per CTA for sizes the kernel covers, else 0.
extern "C" int b200_attn_latent_decode_heads(int H, int C, int D, int block_size) {
  using namespace b200::latdec;
  if (H <= 0 || C <= 0 || C > 512 || D < C || (C & 15) || (D & 15)) return 0;
  if (block_size != 16 && block_size != 32 && block_size != 64 && block_size != 128) return 0;
  const int N = heads_of(H);
  return ring_of(N, C, (D + 63) / 64) ? N : 0;
}

// q [rows, H, D], cache [num_blocks * bs, D] (page 0 readable), out [rows, H, C], all bf16; partial: fp32
// [rows * H * splits * (C + 2)] when splits > 1 (sums, then maxima and weights: what b200_attn_latent_merge takes).
extern "C" int b200_attn_latent_decode(const void* q, const void* cache, void* out, const int* block_table, const int* seq,
                                       const int* positions, float* partial, int rows, int max_blocks, int num_blocks, int bs, int H,
                                       int C, int D, int splits, float scale, int* status, cudaStream_t stream) {
  using namespace b200::latdec;
  const int N = b200_attn_latent_decode_heads(H, C, D, bs);
  if (!N || rows <= 0 || rows > 65535 || splits <= 0 || (splits > 1 && !partial) || num_blocks <= 0) return -ERR_BAD_ARG;
  Params p;
  p.block_table = block_table; p.seq = seq; p.positions = positions; p.max_blocks = max_blocks; p.bs = bs; p.box = bs < KT ? bs : KT;
  p.H = H; p.C = C; p.D = D; p.slabs = (D + 63) / 64; p.units = ring_of(N, C, p.slabs); p.splits = splits;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.out = reinterpret_cast<__nv_bfloat16*>(out);
  p.partial = splits > 1 ? partial : nullptr;
  p.stats = splits > 1 ? partial + (size_t)rows * H * splits * C : nullptr;
  p.status = status;
  p.q = reinterpret_cast<const __nv_bfloat16*>(q);
  CUtensorMap tmK;
  const bool ok = make_tmap_2d(&tmK, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, cache, (uint64_t)num_blocks * bs, D, (uint64_t)D * 2, p.box, 64,
                               CU_TENSOR_MAP_SWIZZLE_128B);
  if (!ok) return -ERR_BAD_ARG;
  return N == 16 ? launch<16>(tmK, p, rows, stream) : launch<32>(tmK, p, rows, stream);
}
