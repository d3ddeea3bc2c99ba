// Recurrences with one decay per head (see decay_rule.cu) over prompt portions in chunks of CL rows, bf16 values.  With b_t the
// sum of the log decays of a chunk up to row t and S the state before the chunk:
//
//   retention   u_t = v_t
//   delta rule  u_t = beta_t (v_t - e^{b_t} S^T k_t - sum_{s < t} e^{b_t - b_s} (k_t . k_s) u_s),  that is  U = U0 - W S  with
//               T = (I + tril(beta_t e^{b_t - b_s} k_t . k_s, -1))^-1,   U0 = T diag(beta) V,   W = T diag(beta e^b) K
//   both        o_t = e^{b_t} S^T q_t + sum_{s <= t} A_ts u_s,   A_ts = e^{b_t - b_s} q_t . k_s
//               S'  = e^{b_end} S + sum_s (k_s e^{b_end - b_s}) u_s^T
//
// (the chunked form of the delta rule of Yang et al., "Parallelizing Linear Transformers with the Delta Rule over Sequence
// Length").  Every exponent is a difference taken towards the later row, so no factor grows.
//
//   decay_chunk_prep   one block per chunk and head: decayed q and k, A, and for the delta rule W and U0 -> workspace
//   decay_chunk_scan   four or eight warps per 16 value columns walk the chunks.  Each keeps its share of the channels of
//                      S^T in registers and updates it; for q S and W S, of which each takes 16 rows and 8 columns (or 16),
//                      the shares are exchanged through shared memory once per chunk
//
// fp32 operands enter the products as two bf16 terms (16 significant bits); sums are fp32.
#include <cuda_bf16.h>
#include <stdint.h>
#include "launch.h"
#include "ops.h"
#include "per_device.h"

namespace {
using namespace b200;

constexpr float LOG2E = 1.4426950408889634f;
constexpr float FLOOR = -126.f;          // log2 of a decay that leaves nothing

struct ChunkParams {
  const float *q, *k;              // [rows, G, D] prepared
  const __nv_bfloat16* v;          // head h of row t at v + t * ldv + h * V
  const float* log_decay;          // [rows, H] (delta rule)
  const float* beta;               // [rows, H]
  const float* decay;              // [H] (retention)
  float* state;                    // [slots, H, D, V]
  float* o;                        // [rows, H * V]
  const int *first, *length, *slot, *positions;
  __nv_bfloat16* ws;               // per chunk and head: q hi | q lo | (W hi | W lo |) k hi | k lo [CL, DT], A hi | A lo [CL, CL]
  float* u0;                       // per chunk and head: [CL, V] (delta rule)
  float* end;                      // per chunk and head: e^{b_end}
  int ldv, H, G, D, V, entries, min_len;
};

__device__ __forceinline__ float pow2(float v) {
  float e;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(v));
  return e;
}
__device__ __forceinline__ uint32_t pack_bf16(float a, float b) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&h);
}
// Two values as two bf16 terms each.
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = pack_bf16(a - f.x, b - f.y);
}
__device__ __forceinline__ void mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
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
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ int chunks_of(const ChunkParams& p, int e, int CL) {
  const int n = p.length[e];
  return n < p.min_len ? 0 : (n + CL - 1) / CL;
}

template <int DT, int CL, bool DELTA>
__host__ __device__ constexpr size_t ws_elems() { return (size_t)(DELTA ? 6 : 4) * CL * DT + 2 * CL * CL; }

constexpr int PT = 256;
constexpr int VT = 64;                   // value columns of U0 at a time

template <int DT, int CL, bool DELTA>
constexpr size_t prep_smem() {
  const size_t rows = (size_t)2 * CL * (DT + 8) * 2, later = (size_t)CL * (CL + 1) * 4 + (size_t)CL * (VT + 8) * 2;
  const size_t q = DELTA && later > rows ? later : rows, t = DELTA ? (size_t)2 * CL * (CL + 8) * 2 : 0;
  return rows + q + t + 2 * CL * 4;
}

// grid (chunks, H).
template <int DT, int CL, bool DELTA>
__global__ void __launch_bounds__(PT) decay_chunk_prep_kernel(ChunkParams p) {
  constexpr int LQ = DT + 8, LT = CL + 8, AP = CL + 1, MT = CL / 16;
  constexpr size_t ROWS = (size_t)2 * CL * LQ * 2, LATER = (size_t)CL * AP * 4 + (size_t)CL * (VT + 8) * 2;
  extern __shared__ __align__(16) uint8_t smem[];
  __nv_bfloat16* sk = reinterpret_cast<__nv_bfloat16*>(smem);                  // [hi, lo][CL][LQ]
  __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(smem + ROWS);           // [hi, lo][CL][LQ]
  uint8_t* area_t = smem + ROWS + (DELTA && LATER > ROWS ? LATER : ROWS);
  float* sL = reinterpret_cast<float*>(area_t);                                // [CL][AP] minus the strictly lower factors, then
  __nv_bfloat16* sT = reinterpret_cast<__nv_bfloat16*>(area_t);                // [hi, lo][CL][LT] T with scaled columns
  float* sX = reinterpret_cast<float*>(sq);                                    // [CL][AP] T, in the place of the queries
  __nv_bfloat16* sv = reinterpret_cast<__nv_bfloat16*>(sX + CL * AP);          // [CL][VT + 8]
  float* sb = reinterpret_cast<float*>(area_t + (DELTA ? (size_t)2 * CL * LT * 2 : 0));      // [CL] summed log2 decays
  float* sbeta = sb + CL;
  pdl_grid_trigger();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tig = lane & 3, h = blockIdx.y, kh = h / (p.H / p.G);
  pdl_grid_wait();
  int e = 0, c = blockIdx.x;
  for (; e < p.entries; ++e) {
    const int n = chunks_of(p, e, CL);
    if (c < n) break;
    c -= n;
  }
  if (e == p.entries) return;
  const int t0 = p.first[e] + c * CL, n = min(CL, p.length[e] - c * CL);
  const size_t at = (size_t)blockIdx.x * p.H + h;
  __nv_bfloat16* ws_q = p.ws + at * ws_elems<DT, CL, DELTA>();
  __nv_bfloat16* ws_w = ws_q + (size_t)2 * CL * DT;
  __nv_bfloat16* ws_k = ws_w + (DELTA ? (size_t)2 * CL * DT : 0);
  __nv_bfloat16 *a_hi = ws_k + (size_t)2 * CL * DT, *a_lo = a_hi + CL * CL;
  if (warp == 0) {                                        // inclusive sums over the chunk's rows
    float run = 0.f;
    const float fixed = DELTA ? 0.f : fmaxf(log2f(p.decay[h]), FLOOR);
#pragma unroll
    for (int r0 = 0; r0 < CL; r0 += 32) {
      const int t = r0 + lane;
      const bool on = t < n;
      float b = DELTA ? (on ? fmaxf(p.log_decay[(size_t)(t0 + t) * p.H + h] * LOG2E, FLOOR) : 0.f) : 0.f;
      if (DELTA) {
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const float x = __shfl_up_sync(0xffffffffu, b, o);
          if (lane >= o) b += x;
        }
        sb[t] = run + b;
        run += __shfl_sync(0xffffffffu, b, 31);
        sbeta[t] = on ? p.beta[(size_t)(t0 + t) * p.H + h] : 0.f;
      } else {
        sb[t] = (float)min(t + 1, n) * fixed;
      }
    }
  }
  __syncthreads();
  const float b_end = sb[CL - 1];
  if (tid == 0) p.end[at] = pow2(b_end);
  for (int i = tid; i < CL * (DT / 8); i += PT) {
    const int t = i / (DT / 8), d = i % (DT / 8) * 8;
    const bool ok = t < n && d < p.D;                               // D is a multiple of 16
    const size_t src = ((size_t)(t0 + t) * p.G + kh) * p.D + d;
    float q[8], k[8];
#pragma unroll
    for (int u = 0; u < 8; u += 4) {
      const float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
      const float4 fq = ok ? *reinterpret_cast<const float4*>(p.q + src + u) : z, fk = ok ? *reinterpret_cast<const float4*>(p.k + src + u) : z;
      q[u] = fq.x; q[u + 1] = fq.y; q[u + 2] = fq.z; q[u + 3] = fq.w;
      k[u] = fk.x; k[u + 1] = fk.y; k[u + 2] = fk.z; k[u + 3] = fk.w;
    }
    const float eq = pow2(sb[t]), ek = pow2(b_end - sb[t]);
    uint4 out[4];
    auto put = [&](const float (&f)[8], float s, uint4& hi, uint4& lo) {
      uint32_t *H = reinterpret_cast<uint32_t*>(&hi), *L = reinterpret_cast<uint32_t*>(&lo);
#pragma unroll
      for (int j = 0; j < 4; ++j) split2(f[2 * j] * s, f[2 * j + 1] * s, H[j], L[j]);
    };
    put(q, eq, out[0], out[1]);
    put(k, ek, out[2], out[3]);
    *reinterpret_cast<uint4*>(ws_q + t * DT + d) = out[0];
    *reinterpret_cast<uint4*>(ws_q + (size_t)CL * DT + t * DT + d) = out[1];
    *reinterpret_cast<uint4*>(ws_k + t * DT + d) = out[2];
    *reinterpret_cast<uint4*>(ws_k + (size_t)CL * DT + t * DT + d) = out[3];
    put(q, 1.f, out[0], out[1]);
    put(k, 1.f, out[2], out[3]);
    *reinterpret_cast<uint4*>(sq + t * LQ + d) = out[0];
    *reinterpret_cast<uint4*>(sq + CL * LQ + t * LQ + d) = out[1];
    *reinterpret_cast<uint4*>(sk + t * LQ + d) = out[2];
    *reinterpret_cast<uint4*>(sk + CL * LQ + t * LQ + d) = out[3];
  }
  __syncthreads();
  const int row16 = lane & 15, col8 = (lane >> 4) * 8, trow = (lane & 7) + ((lane >> 3) & 1) * 8;
  // q k^T and k k^T: rows [16 mt, 16 mt + 16), every second tile of 8 columns up to the diagonal
  const int mt = warp & 3, nh = warp >> 2;
  if (mt < MT) {
    constexpr int NT = MT;                                // tiles of a warp at most
    float aq[NT][4], ak[NT][4];
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int x = 0; x < 4; ++x) aq[j][x] = ak[j][x] = 0.f;
#pragma unroll 2
    for (int ks = 0; ks < DT / 16; ++ks) {
      uint32_t qh[4], ql[4], kmh[4], kml[4];
      const int off = (mt * 16 + row16) * LQ + ks * 16 + col8;
      ldmatrix_x4(qh, sq + off);
      ldmatrix_x4(ql, sq + CL * LQ + off);
      if (DELTA) {
        ldmatrix_x4(kmh, sk + off);
        ldmatrix_x4(kml, sk + CL * LQ + off);
      }
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        if (j > mt) break;
        const __nv_bfloat16* b = sk + ((2 * j + nh) * 8 + g) * LQ + ks * 16 + 2 * tig;
        const uint32_t h0 = *reinterpret_cast<const uint32_t*>(b), h1 = *reinterpret_cast<const uint32_t*>(b + 8);
        const uint32_t l0 = *reinterpret_cast<const uint32_t*>(b + CL * LQ), l1 = *reinterpret_cast<const uint32_t*>(b + CL * LQ + 8);
        mma(aq[j], qh, h0, h1);
        mma(aq[j], qh, l0, l1);
        mma(aq[j], ql, h0, h1);
        if (DELTA) {
          mma(ak[j], kmh, h0, h1);
          mma(ak[j], kmh, l0, l1);
          mma(ak[j], kml, h0, h1);
        }
      }
    }
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      if (j > mt) break;
#pragma unroll
      for (int w = 0; w < 2; ++w) {
        const int r = mt * 16 + g + 8 * w, s = (2 * j + nh) * 8 + 2 * tig;
        float a[2];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          const float dec = s + u <= r ? pow2(sb[r] - sb[s + u]) : 0.f;
          a[u] = aq[j][2 * w + u] * dec;
          if (DELTA) sL[r * AP + s + u] = s + u < r ? -sbeta[r] * ak[j][2 * w + u] * dec : 0.f;
        }
        uint32_t hi, lo;
        split2(a[0], a[1], hi, lo);
        *reinterpret_cast<uint32_t*>(a_hi + r * CL + s) = hi;
        *reinterpret_cast<uint32_t*>(a_lo + r * CL + s) = lo;
      }
    }
  }
  if constexpr (DELTA) {
    __syncthreads();
    // T = (I - L)^-1 by blocks of 16 (L strictly lower triangular, fp32):
    //   T_ii = (I - L_ii)^-1                       one warp per diagonal block, a column per lane in registers
    //   T_ij = T_ii (sum_{k=j}^{i-1} L_ik T_kj)    one block sub-diagonal at a time, one element per thread and block; the inner
    //                                              sums are staged in the unused upper blocks of L
    if (warp < MT) {
      if (lane < 16) {
        const int b0 = 16 * warp;
        float tr[16];
#pragma unroll
        for (int r = 0; r < 16; ++r) {
          float acc = lane == r ? 1.f : 0.f;
#pragma unroll
          for (int m = 0; m < r; ++m) acc = fmaf(sL[(b0 + r) * AP + b0 + m], tr[m], acc);
          tr[r] = acc;
          sX[(b0 + r) * AP + b0 + lane] = acc;
        }
      }
    } else {
      for (int i = tid - 32 * MT; i < CL * CL; i += PT - 32 * MT) {
        const int r = i / CL, s = i % CL;
        if (s / 16 > r / 16) sX[r * AP + s] = 0.f;
      }
    }
    __syncthreads();
    {
      const int r = tid >> 4, cc = tid & 15;
#pragma unroll 1
      for (int d = 1; d < MT; ++d) {
        float inner[MT > 1 ? MT - 1 : 1];
#pragma unroll
        for (int b = 0; b + 1 < MT; ++b) {                      // block (b + d, b)
          if (b + d >= MT) break;
          float acc = 0.f;
          for (int k = b; k < b + d; ++k) {
            const float *lr = sL + (16 * (b + d) + r) * AP + 16 * k, *xc = sX + 16 * k * AP + 16 * b + cc;
#pragma unroll
            for (int m = 0; m < 16; ++m) acc = fmaf(lr[m], xc[m * AP], acc);
          }
          inner[b] = acc;
        }
#pragma unroll
        for (int b = 0; b + 1 < MT; ++b)
          if (b + d < MT) sL[(16 * b + r) * AP + 16 * (b + d) + cc] = inner[b];
        __syncthreads();
#pragma unroll
        for (int b = 0; b + 1 < MT; ++b) {
          if (b + d >= MT) break;
          const float *tr = sX + (16 * (b + d) + r) * AP + 16 * (b + d), *mc = sL + 16 * b * AP + 16 * (b + d) + cc;
          float acc = 0.f;
#pragma unroll
          for (int m = 0; m < 16; ++m) acc = fmaf(tr[m], mc[m * AP], acc);
          sX[(16 * (b + d) + r) * AP + 16 * b + cc] = acc;
        }
        __syncthreads();
      }
    }
    constexpr int PER = CL * CL / PT;                       // neighbouring columns of T per thread
    const int tr = tid * PER / CL, tc = tid * PER % CL;
    float tv[PER];
#pragma unroll
    for (int x = 0; x < PER; ++x) tv[x] = sX[tr * AP + tc + x] * sbeta[tc + x];
    auto put_t = [&](bool decayed) {
#pragma unroll
      for (int x = 0; x < PER; x += 2) {
        const float f0 = decayed ? pow2(sb[tc + x]) : 1.f, f1 = decayed ? pow2(sb[tc + x + 1]) : 1.f;
        uint32_t hi, lo;
        split2(tv[x] * f0, tv[x + 1] * f1, hi, lo);
        *reinterpret_cast<uint32_t*>(sT + tr * LT + tc + x) = hi;
        *reinterpret_cast<uint32_t*>(sT + CL * LT + tr * LT + tc + x) = lo;
      }
    };
    put_t(true);                                            // L is dead: its last readers are behind the barrier above
    __syncthreads();
    // W: 16 rows, half the channels per warp; products past the diagonal are zero
    if (mt < MT) {
      constexpr int NN = DT / 16;                           // tiles of 8 channels of a warp
#pragma unroll 1
      for (int n0 = 0; n0 < NN; n0 += 4) {
        float acc[4][4] = {};
        for (int ks = 0; ks <= mt; ++ks) {
          uint32_t th[4], tl[4];
          ldmatrix_x4(th, sT + (mt * 16 + row16) * LT + ks * 16 + col8);
          ldmatrix_x4(tl, sT + CL * LT + (mt * 16 + row16) * LT + ks * 16 + col8);
#pragma unroll
          for (int j = 0; j < 4; j += 2) {
            uint32_t kh_[4], kl_[4];
            const int off = (ks * 16 + trow) * LQ + nh * (DT / 2) + (n0 + j) * 8 + col8;
            ldmatrix_x4_trans(kh_, sk + off);
            ldmatrix_x4_trans(kl_, sk + CL * LQ + off);
#pragma unroll
            for (int u = 0; u < 2; ++u) {
              mma(acc[j + u], th, kh_[2 * u], kh_[2 * u + 1]);
              mma(acc[j + u], th, kl_[2 * u], kl_[2 * u + 1]);
              mma(acc[j + u], tl, kh_[2 * u], kh_[2 * u + 1]);
            }
          }
        }
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
          for (int w = 0; w < 2; ++w) {
            uint32_t hi, lo;
            split2(acc[j][2 * w], acc[j][2 * w + 1], hi, lo);
            const size_t x = (size_t)(mt * 16 + g + 8 * w) * DT + nh * (DT / 2) + (n0 + j) * 8 + 2 * tig;
            *reinterpret_cast<uint32_t*>(ws_w + x) = hi;
            *reinterpret_cast<uint32_t*>(ws_w + (size_t)CL * DT + x) = lo;
          }
      }
    }
    __syncthreads();
    put_t(false);
    // U0, VT columns at a time, half of them per warp
    constexpr int LV = VT + 8;
    float* u0 = p.u0 + at * CL * p.V;
    for (int v0 = 0; v0 < p.V; v0 += VT) {
      __syncthreads();                                      // T is written, the last tile of values has been read
      for (int i = tid; i < CL * (VT / 8); i += PT) {
        const int t = i / (VT / 8), x = i % (VT / 8) * 8;
        *reinterpret_cast<uint4*>(sv + t * LV + x) = t < n && v0 + x < p.V
            ? *reinterpret_cast<const uint4*>(p.v + (size_t)(t0 + t) * p.ldv + (size_t)h * p.V + v0 + x) : make_uint4(0, 0, 0, 0);
      }
      __syncthreads();
      if (mt < MT) {
        float acc[4][4] = {};
        for (int ks = 0; ks <= mt; ++ks) {
          uint32_t th[4], tl[4];
          ldmatrix_x4(th, sT + (mt * 16 + row16) * LT + ks * 16 + col8);
          ldmatrix_x4(tl, sT + CL * LT + (mt * 16 + row16) * LT + ks * 16 + col8);
#pragma unroll
          for (int j = 0; j < 4; j += 2) {
            uint32_t b[4];
            ldmatrix_x4_trans(b, sv + (ks * 16 + trow) * LV + nh * (VT / 2) + j * 8 + col8);
#pragma unroll
            for (int u = 0; u < 2; ++u) {
              mma(acc[j + u], th, b[2 * u], b[2 * u + 1]);
              mma(acc[j + u], tl, b[2 * u], b[2 * u + 1]);
            }
          }
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int col = v0 + nh * (VT / 2) + j * 8 + 2 * tig;
          if (col < p.V)
#pragma unroll
            for (int w = 0; w < 2; ++w)
              *reinterpret_cast<float2*>(u0 + (size_t)(mt * 16 + g + 8 * w) * p.V + col) = make_float2(acc[j][2 * w], acc[j][2 * w + 1]);
        }
      }
    }
  }
}

constexpr int LU = 24;                   // padded row of the [CL x 16] tiles of U

// Shared memory of the scan: query (and W) rows of two chunks; key rows, A (and values) of one chunk or two.
template <int DT, int CL, bool DELTA>
__host__ __device__ constexpr size_t front_elems() { return (size_t)(DELTA ? 4 : 2) * CL * (DT + 8); }
template <int DT, int CL, bool DELTA>
__host__ __device__ constexpr size_t back_elems(int VB) { return (size_t)2 * CL * (DT + 8) + 2 * CL * (CL + 8) + (DELTA ? 0 : CL * (VB + 8)); }
template <int DT, int CL, bool DELTA>
constexpr size_t scan_smem(int VB) {
  return (2 * front_elems<DT, CL, DELTA>() + (DELTA ? 1 : 2) * back_elems<DT, CL, DELTA>(VB) + (size_t)(VB / 16) * 2 * 16 * (DT + 8) +
          (DELTA ? (size_t)(VB / 16) * 2 * CL * LU : 0)) * 2;
}

// grid (ceil(V / VB), H, entries), W VB / 16 warps: W of them (4 or 8) own value columns 16 i .. 16 i + 15.
template <int DT, int CL, int W, bool DELTA>
__global__ void __launch_bounds__(512) decay_chunk_scan_kernel(ChunkParams p) {
  constexpr int LQ = DT + 8, LA = CL + 8, MT = CL / 16, ND = DT / W, NS = ND / 8, NJ = W == 8 ? 1 : 2;
  // channels, fragments of S^T and 8-column tiles of the output of a warp
  extern __shared__ __align__(16) uint8_t smem[];
  const int tid = threadIdx.x, nthr = blockDim.x, lane = tid & 31, g = lane >> 2, tig = lane & 3;
  const int vg = tid / (32 * W), sub = (tid >> 5) % W;
  const int VB = nthr / (2 * W), LV = VB + 8, h = blockIdx.y, e = blockIdx.z, v0 = blockIdx.x * VB;
  __nv_bfloat16* front = reinterpret_cast<__nv_bfloat16*>(smem);
  __nv_bfloat16* back = front + 2 * front_elems<DT, CL, DELTA>();
  __nv_bfloat16* s_state = back + (DELTA ? 1 : 2) * back_elems<DT, CL, DELTA>(VB);
  __nv_bfloat16* ss = s_state + (size_t)vg * 2 * 16 * LQ;                                                    // [hi, lo][16][LQ]
  __nv_bfloat16* su = s_state + (size_t)(VB / 16) * 2 * 16 * LQ + (size_t)vg * 2 * CL * LU;                  // [hi, lo][CL][LU]
  pdl_grid_trigger();
  pdl_grid_wait();
  const int chunks = chunks_of(p, e, CL);
  if (chunks == 0) return;
  int base = 0;
  for (int i = 0; i < e; ++i) base += chunks_of(p, i, CL);
  const int r0 = p.first[e], len = p.length[e];
  auto ws_of = [&](int c) { return p.ws + ((size_t)(base + c) * p.H + h) * ws_elems<DT, CL, DELTA>(); };
  auto fetch_front = [&](int c) {
    const __nv_bfloat16* ws = ws_of(c);
    __nv_bfloat16* dst = front + (c & 1) * front_elems<DT, CL, DELTA>();
    for (int i = tid; i < (DELTA ? 4 : 2) * CL * (DT / 8); i += nthr) {
      const int r = i / (DT / 8), d = i % (DT / 8) * 8;
      cp16(dst + r * LQ + d, ws + (size_t)r * DT + d, true);
    }
  };
  auto fetch_back = [&](int c) {
    const __nv_bfloat16* ws = ws_of(c) + (size_t)(DELTA ? 4 : 2) * CL * DT;
    __nv_bfloat16* dst = back + (DELTA ? 0 : c & 1) * back_elems<DT, CL, DELTA>(VB);
    for (int i = tid; i < 2 * CL * (DT / 8); i += nthr) {
      const int r = i / (DT / 8), d = i % (DT / 8) * 8;
      cp16(dst + r * LQ + d, ws + (size_t)r * DT + d, true);
    }
    dst += 2 * CL * LQ;
    ws += (size_t)2 * CL * DT;
    for (int i = tid; i < 2 * CL * (CL / 8); i += nthr) {
      const int r = i / (CL / 8), s = i % (CL / 8) * 8;
      cp16(dst + r * LA + s, ws + r * CL + s, true);
    }
    if (!DELTA) {
      dst += 2 * CL * LA;
      for (int i = tid; i < CL * (VB / 8); i += nthr) {
        const int r = i / (VB / 8), x = i % (VB / 8) * 8;
        const bool ok = c * CL + r < len && v0 + x < p.V;
        cp16(dst + r * LV + x, p.v + (ok ? (size_t)(r0 + c * CL + r) * p.ldv + (size_t)h * p.V + v0 + x : 0), ok);
      }
    }
  };
  fetch_front(0);
  if (!DELTA) fetch_back(0);
  cp_commit();
  const int vw = v0 + vg * 16, d_own = sub * ND;
  const bool live = vw < p.V;
  const bool reads = live && sub < MT * 2 / NJ;         // takes part in the products with the state
  const int m = NJ == 2 ? sub : sub >> 1, j0 = NJ == 2 ? 0 : sub & 1;
  float* st = p.state + ((size_t)p.slot[e] * p.H + h) * p.D * p.V;
  const bool fresh = p.positions[r0] == 0;
  float S[NS][4];                                       // S^T: value columns g, g + 8; channels d_own + 8 i + 2 tig, + 1
#pragma unroll
  for (int i = 0; i < NS; ++i)
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int d = d_own + i * 8 + 2 * tig + (x & 1), v = vw + g + 8 * (x >> 1);
      S[i][x] = live && !fresh && d < p.D ? st[(size_t)d * p.V + v] : 0.f;
    }
  auto publish = [&]() {
#pragma unroll
    for (int i = 0; i < NS; ++i)
#pragma unroll
      for (int w = 0; w < 2; ++w) {
        uint32_t hi, lo;
        split2(S[i][2 * w], S[i][2 * w + 1], hi, lo);
        __nv_bfloat16* dst = ss + (g + 8 * w) * LQ + d_own + i * 8 + 2 * tig;
        *reinterpret_cast<uint32_t*>(dst) = hi;
        *reinterpret_cast<uint32_t*>(dst + 16 * LQ) = lo;
      }
  };
  publish();
  float2 u_next[NJ][2];                                 // U0 of the next chunk: rows g, g + 8 of the warp's tile
  float end_next;
  auto load_next = [&](int c) {
    const size_t at = (size_t)(base + c) * p.H + h;
    end_next = p.end[at];
    if (DELTA && reads)
#pragma unroll
      for (int j = 0; j < NJ; ++j)
#pragma unroll
        for (int w = 0; w < 2; ++w)
          u_next[j][w] = *reinterpret_cast<const float2*>(p.u0 + (at * CL + m * 16 + g + 8 * w) * p.V + vw + (j0 + j) * 8 + 2 * tig);
  };
  load_next(0);
  const int row16 = lane & 15, col8 = (lane >> 4) * 8;                       // non-transposed 16 x 16 tiles, left operand
  const int brow = (lane & 7) + (lane >> 4) * 8, bcol = ((lane >> 3) & 1) * 8;   // left operand, transposed
  const int trow = (lane & 7) + ((lane >> 3) & 1) * 8;                       // right operand, transposed
  for (int c = 0; c < chunks; ++c) {
    cp_wait<0>();
    __syncthreads();                                    // rows and state landed; the buffers' last readers are done
    const bool more = c + 1 < chunks;
    if (DELTA) {
      fetch_back(c);
      cp_commit();
      if (more) fetch_front(c + 1);
      cp_commit();
    } else if (more) {
      fetch_front(c + 1);
      fetch_back(c + 1);
      cp_commit();
    }
    float2 u[NJ][2];
#pragma unroll
    for (int j = 0; j < NJ; ++j) { u[j][0] = u_next[j][0]; u[j][1] = u_next[j][1]; }
    const float end = end_next;
    if (more) load_next(c + 1);
    const __nv_bfloat16* sq = front + (c & 1) * front_elems<DT, CL, DELTA>();
    const __nv_bfloat16* sw = sq + 2 * CL * LQ;
    const __nv_bfloat16* sk = back + (DELTA ? 0 : c & 1) * back_elems<DT, CL, DELTA>(VB);
    const __nv_bfloat16* sa = sk + 2 * CL * LQ;
    const __nv_bfloat16* sv = DELTA ? su : sa + 2 * CL * LA + vg * 16;       // rows of U (or of the values)
    const int lv = DELTA ? LU : LV;
    float o[NJ][4] = {}, ol[NJ][4] = {};                // sums of the leading and of the correcting products
    if (reads) {
      float w[NJ][4] = {}, wl[NJ][4] = {};
#pragma unroll
      for (int k2 = 0; k2 < DT / 32; ++k2) {
        uint32_t bh[NJ][4], bl[NJ][4];                  // two k-steps of 8 columns
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
          const __nv_bfloat16* b = ss + ((j0 + j) * 8 + (lane & 7)) * LQ + k2 * 32 + (lane >> 3) * 8;
          ldmatrix_x4(bh[j], b);
          ldmatrix_x4(bl[j], b + 16 * LQ);
        }
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          uint32_t ah[4], al[4];
          const int off = (m * 16 + row16) * LQ + k2 * 32 + x * 16 + col8;
          if (DELTA) {                                  // first: the rest of the chunk waits for these
            ldmatrix_x4(ah, sw + off);
            ldmatrix_x4(al, sw + CL * LQ + off);
#pragma unroll
            for (int j = 0; j < NJ; ++j) {
              mma(w[j], ah, bh[j][2 * x], bh[j][2 * x + 1]);
              mma(wl[j], ah, bl[j][2 * x], bl[j][2 * x + 1]);
              mma(wl[j], al, bh[j][2 * x], bh[j][2 * x + 1]);
            }
          }
          ldmatrix_x4(ah, sq + off);
          ldmatrix_x4(al, sq + CL * LQ + off);
#pragma unroll
          for (int j = 0; j < NJ; ++j) {
            mma(o[j], ah, bh[j][2 * x], bh[j][2 * x + 1]);
            mma(ol[j], ah, bl[j][2 * x], bl[j][2 * x + 1]);
            mma(ol[j], al, bh[j][2 * x], bh[j][2 * x + 1]);
          }
        }
      }
      if (DELTA) {
#pragma unroll
        for (int j = 0; j < NJ; ++j)
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            uint32_t hi, lo;
            split2(u[j][x].x - (w[j][2 * x] + wl[j][2 * x]), u[j][x].y - (w[j][2 * x + 1] + wl[j][2 * x + 1]), hi, lo);
            __nv_bfloat16* dst = su + (m * 16 + g + 8 * x) * LU + (j0 + j) * 8 + 2 * tig;
            *reinterpret_cast<uint32_t*>(dst) = hi;
            *reinterpret_cast<uint32_t*>(dst + CL * LU) = lo;
          }
      }
    }
    if (DELTA) cp_wait<1>();                            // the back half; the next front half may be on its way
    __syncthreads();                                    // U, keys and A landed; everyone has read the state of before the chunk
    if (live) {
#pragma unroll
      for (int i = 0; i < NS; ++i)
#pragma unroll
        for (int x = 0; x < 4; ++x) S[i][x] *= end;
#pragma unroll
      for (int ks = 0; ks < MT; ++ks) {
        uint32_t a[4], al[4];
        ldmatrix_x4_trans(a, sv + (ks * 16 + brow) * lv + bcol);
        if (DELTA) ldmatrix_x4_trans(al, sv + CL * LU + (ks * 16 + brow) * lv + bcol);
        constexpr int PAIRS = NS / 2;
#pragma unroll
        for (int i = 0; i < PAIRS; ++i) {
          uint32_t bh[4], bl[4];
          const int off = (ks * 16 + trow) * LQ + d_own + i * 16 + col8;
          ldmatrix_x4_trans(bh, sk + off);
          ldmatrix_x4_trans(bl, sk + CL * LQ + off);
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            mma(S[2 * i + x], a, bh[2 * x], bh[2 * x + 1]);
            mma(S[2 * i + x], a, bl[2 * x], bl[2 * x + 1]);
            if (DELTA) mma(S[2 * i + x], al, bh[2 * x], bh[2 * x + 1]);
          }
        }
      }
      publish();                                        // the next chunk starts from it: the outputs come after
    }
    if (reads) {
#pragma unroll
      for (int ks = 0; ks < MT; ++ks) {
        if (ks > m) break;
        uint32_t b[4], bl[4], ah[4], al[4];
        ldmatrix_x4_trans(b, sv + (ks * 16 + trow) * lv + col8);
        if (DELTA) ldmatrix_x4_trans(bl, sv + CL * LU + (ks * 16 + trow) * lv + col8);
        ldmatrix_x4(ah, sa + (m * 16 + row16) * LA + ks * 16 + col8);
        ldmatrix_x4(al, sa + (CL + m * 16 + row16) * LA + ks * 16 + col8);
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
          const uint32_t b0 = j0 + j ? b[2] : b[0], b1 = j0 + j ? b[3] : b[1];
          mma(o[j], ah, b0, b1);
          mma(ol[j], al, b0, b1);
          if (DELTA) mma(ol[j], ah, j0 + j ? bl[2] : bl[0], j0 + j ? bl[3] : bl[1]);
        }
      }
#pragma unroll
      for (int w = 0; w < 2; ++w) {
        const int t = c * CL + m * 16 + g + 8 * w;
        if (t < len) {
          float* dst = p.o + ((size_t)(r0 + t) * p.H + h) * p.V + vw + j0 * 8 + 2 * tig;
#pragma unroll
          for (int j = 0; j < NJ; ++j)
            *reinterpret_cast<float2*>(dst + j * 8) = make_float2(o[j][2 * w] + ol[j][2 * w], o[j][2 * w + 1] + ol[j][2 * w + 1]);
        }
      }
    }
  }
  cp_wait<0>();
  if (!live) return;
#pragma unroll
  for (int i = 0; i < NS; ++i)
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int d = d_own + i * 8 + 2 * tig + (x & 1), v = vw + g + 8 * (x >> 1);
      if (d < p.D) st[(size_t)d * p.V + v] = S[i][x];
    }
}

template <int DT, int CL, int W, bool DELTA>
int launch_scan(const ChunkParams& p, int groups, cudaStream_t stream) {
  static PerDeviceOnce once_;
  bool& configured = once_.slot();
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(decay_chunk_scan_kernel<DT, CL, W, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  return (int)launch_pdl(decay_chunk_scan_kernel<DT, CL, W, DELTA>, dim3((p.V + 16 * groups - 1) / (16 * groups), p.H, p.entries),
                         dim3(groups * W * 32), scan_smem<DT, CL, DELTA>(16 * groups), stream, p);
}

template <int DT, int CL, bool DELTA>
int launch(const ChunkParams& p, int chunks, cudaStream_t stream) {
  static PerDeviceOnce once_;
  bool& configured = once_.slot();
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(decay_chunk_prep_kernel<DT, CL, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const cudaError_t e = launch_pdl(decay_chunk_prep_kernel<DT, CL, DELTA>, dim3(chunks, p.H), dim3(PT), prep_smem<DT, CL, DELTA>(), stream, p);
  if (e != cudaSuccess) return (int)e;
  // 16 columns per block where one wave of blocks takes them, more otherwise
  constexpr int W = DT >= 128 ? 8 : 4;
  int groups = 1;
  while (groups * 2 * W * 32 <= 512 && (long long)p.entries * p.H * ((p.V + 16 * groups - 1) / (16 * groups)) > 148 && 16 * groups < p.V &&
         scan_smem<DT, CL, DELTA>(32 * groups) <= 227 * 1024)
    groups <<= 1;
  return launch_scan<DT, CL, W, DELTA>(p, groups, stream);
}

template <bool DELTA>
int pick(const ChunkParams& p, int chunks, cudaStream_t stream) {
  if (p.D <= 64) return launch<64, 64, DELTA>(p, chunks, stream);
  if (p.D <= 128) return launch<128, 64, DELTA>(p, chunks, stream);
  return launch<256, 32, DELTA>(p, chunks, stream);
}

}  // namespace

// Rows per chunk for D key channels; 0: not covered.
extern "C" int b200_decay_chunk_rows(int D) { return D <= 0 || D % 16 || D > 256 ? 0 : D <= 128 ? 64 : 32; }

// bf16 elements of workspace per chunk and head.
extern "C" int b200_decay_chunk_ws(int D, int delta) {
  if (delta) return D <= 64 ? ws_elems<64, 64, true>() : D <= 128 ? ws_elems<128, 64, true>() : ws_elems<256, 32, true>();
  return D <= 64 ? ws_elems<64, 64, false>() : D <= 128 ? ws_elems<128, 64, false>() : ws_elems<256, 32, false>();
}

// Entries with at least min_len rows; chunks: upper bound on their number (rows / chunk rows + entries).  q, k fp32 [rows, G, D]
// (b200_delta_prep, b200_rotate_prep), v bf16 rows `ldv` apart.  decay [H]: retention; else log_decay and beta [rows, H]: the delta
// rule, with u0 fp32 [chunks * H * chunk rows * V].  D, V multiples of 16, D <= 256; end fp32 [chunks * H]; state [slots, H, D, V]
// fp32 in place; o fp32 [rows, H * V].
extern "C" int b200_decay_chunk(const float* q, const float* k, const void* v, int ldv, const float* log_decay, const float* decay,
                                const float* beta, float* state, float* o, const int* first, const int* length, const int* slot,
                                const int* positions, int entries, int min_len, int chunks, void* ws, float* u0, float* end, int H, int G,
                                int D, int V, cudaStream_t stream) {
  if (!b200_decay_chunk_rows(D) || V <= 0 || (V & 15) || (ldv & 7) || entries <= 0 || entries > 65535 || H <= 0 || H > 65535 || G <= 0 ||
      H % G || chunks <= 0 || (!decay && (!log_decay || !beta || !u0)))
    return -6;
  ChunkParams p;
  p.q = q; p.k = k; p.v = reinterpret_cast<const __nv_bfloat16*>(v); p.log_decay = log_decay; p.beta = beta; p.decay = decay; p.state = state;
  p.o = o; p.first = first; p.length = length; p.slot = slot; p.positions = positions; p.ws = reinterpret_cast<__nv_bfloat16*>(ws);
  p.u0 = u0; p.end = end; p.ldv = ldv; p.H = H; p.G = G; p.D = D; p.V = V; p.entries = entries; p.min_len = min_len;
  return decay ? pick<false>(p, chunks, stream) : pick<true>(p, chunks, stream);
}
