// Gated delta rule (see decay_rule.cu) over prompt portions in chunks of CL rows, bf16 values.  With b_t the sum of the log decays
// of a chunk up to row t and S the state before the chunk:
//
//   u_t = beta_t (v_t - e^{b_t} S^T k_t - sum_{s < t} e^{b_t - b_s} (k_t . k_s) u_s)
//       that is   U = T diag(beta) (V - diag(e^b) K S),   T = (I + tril(beta_t e^{b_t - b_s} k_t . k_s, -1))^-1
//   o_t = e^{b_t} S^T q_t + sum_{s <= t} A_ts u_s,   A_ts = e^{b_t - b_s} q_t . k_s
//   S'  = e^{b_end} S + sum_s k_s (e^{b_end - b_s} u_s)^T
//
// (the chunked form of Yang et al., "Parallelizing Linear Transformers with the Delta Rule over Sequence Length", with the
// decays outside the products).  Every exponent is a difference taken towards the later row, so no factor grows.  The products
// among queries and keys do not depend on the head's decay: the heads that share them share that work and its rows.
//
//   delta_prep   one block per chunk and query / key head: the rows of q and k as two bf16 terms, their products, and per head
//                A, T diag(beta) and the decays -> workspace.  Two groups of four warps take the heads in turn
//   delta_scan   eight warps per 16 or 32 value columns walk the chunks.  Four take K S (and X = V - e^b K S), four q S, 16 rows
//                each; all of them U = T X; then each updates its share of the channels of S^T, which stays in registers and is
//                published once per chunk
//
// fp32 operands enter the products as two bf16 terms (16 significant bits); sums are fp32.
#include <cuda_bf16.h>
#include <stdint.h>
#include "launch.h"
#include "ops.h"
#include "per_device.h"
#include "split_mma.cuh"

namespace {
using namespace b200;

constexpr float LOG2E = 1.4426950408889634f;
constexpr float FLOOR = -126.f;          // log2 of a decay that leaves nothing

struct DeltaParams {
  const float *q, *k;              // [rows, G, D] unit vectors, queries scaled
  const __nv_bfloat16* v;          // head h of row t at v + t * ldv + h * V
  const float *log_decay, *beta;   // [rows, H]
  float* state;                    // [slots, H, D, V]
  float* o;                        // [rows, H * V]
  const int *first, *length, *slot, *positions;
  __nv_bfloat16* rows;             // per chunk and query / key head: k hi | k lo | q hi | q lo [CL, DT]
  __nv_bfloat16* mats;             // per chunk and head: A hi | A lo | T diag(beta) hi | lo [CL, CL]
  float* fade;                     // per chunk and head: e^{b_t}, e^{b_end - b_t} [2, CL]
  int ldv, H, G, D, V, entries, min_len;
};

__device__ __forceinline__ int chunks_of(const DeltaParams& p, int e, int CL) {
  const int n = p.length[e];
  return n < p.min_len ? 0 : (n + CL - 1) / CL;
}

constexpr int PT = 256;
constexpr int TD = 24;                   // padded row of a 16 x 16 tile

// Bytes of one four-warp group: diagonal blocks fp32, their inverses as two terms, the lower factors (then T) as two terms, sums.
template <int CL>
__host__ __device__ constexpr size_t quad_bytes() {
  return (size_t)(CL / 16) * 16 * 17 * 4 + (size_t)2 * (CL / 16) * 16 * TD * 2 + (size_t)2 * CL * (CL + 8) * 2 + 2 * CL * 4;
}
template <int DT, int CL>
constexpr size_t prep_smem() {
  const size_t rows = (size_t)4 * CL * (DT + 8) * 2, later = (size_t)2 * CL * (CL + 1) * 4 + 2 * quad_bytes<CL>();
  return rows > later ? rows : later;
}

__device__ __forceinline__ void quad_sync(int quad) { asm volatile("bar.sync %0, 128;" ::"r"(quad + 1) : "memory"); }

// grid (chunks, G).
template <int DT, int CL>
__global__ void __launch_bounds__(PT) delta_prep_kernel(DeltaParams p) {
  constexpr int LQ = DT + 8, AP = CL + 1, LT = CL + 8, MT = CL / 16;
  extern __shared__ __align__(16) uint8_t smem[];
  __nv_bfloat16* sk = reinterpret_cast<__nv_bfloat16*>(smem);          // [hi, lo][CL][LQ]
  __nv_bfloat16* sq = sk + 2 * CL * LQ;
  float* qk = reinterpret_cast<float*>(smem);                          // [CL][AP] q k^T and k k^T, over the rows once they are used
  float* kk = qk + CL * AP;
  pdl_grid_trigger();
  const int tid = threadIdx.x, warp = __shfl_sync(0xffffffffu, tid >> 5, 0), lane = tid & 31, g = lane >> 2, tig = lane & 3, kh = blockIdx.y;
  pdl_grid_wait();
  int e = 0, c = blockIdx.x;
  for (; e < p.entries; ++e) {
    const int n = chunks_of(p, e, CL);
    if (c < n) break;
    c -= n;
  }
  if (e == p.entries) return;
  const int t0 = p.first[e] + c * CL, n = min(CL, p.length[e] - c * CL);
  __nv_bfloat16* ws_k = p.rows + ((size_t)blockIdx.x * p.G + kh) * 4 * CL * DT;
  __nv_bfloat16* ws_q = ws_k + (size_t)2 * CL * DT;
  for (int i = tid; i < CL * (DT / 8); i += PT) {
    const int t = i / (DT / 8), d = i % (DT / 8) * 8;
    const bool ok = t < n && d < p.D;                                  // D is a multiple of 16
    const size_t src = ((size_t)(t0 + t) * p.G + kh) * p.D + d;
    const float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
    const float4 q0 = ok ? *reinterpret_cast<const float4*>(p.q + src) : z, q1 = ok ? *reinterpret_cast<const float4*>(p.q + src + 4) : z;
    const float4 k0 = ok ? *reinterpret_cast<const float4*>(p.k + src) : z, k1 = ok ? *reinterpret_cast<const float4*>(p.k + src + 4) : z;
    uint4 hi, lo;
    split2(k0.x, k0.y, hi.x, lo.x); split2(k0.z, k0.w, hi.y, lo.y); split2(k1.x, k1.y, hi.z, lo.z); split2(k1.z, k1.w, hi.w, lo.w);
    *reinterpret_cast<uint4*>(ws_k + t * DT + d) = hi;
    *reinterpret_cast<uint4*>(ws_k + (size_t)CL * DT + t * DT + d) = lo;
    *reinterpret_cast<uint4*>(sk + t * LQ + d) = hi;
    *reinterpret_cast<uint4*>(sk + CL * LQ + t * LQ + d) = lo;
    split2(q0.x, q0.y, hi.x, lo.x); split2(q0.z, q0.w, hi.y, lo.y); split2(q1.x, q1.y, hi.z, lo.z); split2(q1.z, q1.w, hi.w, lo.w);
    *reinterpret_cast<uint4*>(ws_q + t * DT + d) = hi;
    *reinterpret_cast<uint4*>(ws_q + (size_t)CL * DT + t * DT + d) = lo;
    *reinterpret_cast<uint4*>(sq + t * LQ + d) = hi;
    *reinterpret_cast<uint4*>(sq + CL * LQ + t * LQ + d) = lo;
  }
  __syncthreads();
  const int row16 = lane & 15, col8 = (lane >> 4) * 8;
  {
    // rows [16 mt, 16 mt + 16), every second tile of 8 columns up to the diagonal
    const int mt = warp & 3, nh = warp >> 2;
    float aq[MT][4], ak[MT][4];
#pragma unroll
    for (int j = 0; j < MT; ++j)
#pragma unroll
      for (int x = 0; x < 4; ++x) aq[j][x] = ak[j][x] = 0.f;
    if (mt < MT) {
#pragma unroll 2
      for (int ks = 0; ks < DT / 16; ++ks) {
        uint32_t qh[4], ql[4], mh[4], ml[4];
        const int off = (mt * 16 + row16) * LQ + ks * 16 + col8;
        ldmatrix_x4(qh, sq + off);
        ldmatrix_x4(ql, sq + CL * LQ + off);
        ldmatrix_x4(mh, sk + off);
        ldmatrix_x4(ml, sk + CL * LQ + off);
#pragma unroll
        for (int j = 0; j < MT; ++j) {
          if (j > mt) break;
          const __nv_bfloat16* b = sk + ((2 * j + nh) * 8 + g) * LQ + ks * 16 + 2 * tig;
          const uint32_t h0 = *reinterpret_cast<const uint32_t*>(b), h1 = *reinterpret_cast<const uint32_t*>(b + 8);
          const uint32_t l0 = *reinterpret_cast<const uint32_t*>(b + CL * LQ), l1 = *reinterpret_cast<const uint32_t*>(b + CL * LQ + 8);
          mma(aq[j], qh, h0, h1);
          mma(ak[j], mh, h0, h1);
          mma(aq[j], qh, l0, l1);
          mma(ak[j], mh, l0, l1);
          mma(aq[j], ql, h0, h1);
          mma(ak[j], ml, h0, h1);
        }
      }
    }
    __syncthreads();                                                   // the rows have been read
    if (mt < MT) {
#pragma unroll
      for (int j = 0; j < MT; ++j) {
        if (j > mt) break;
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const int at = (mt * 16 + g + 8 * (x >> 1)) * AP + (2 * j + nh) * 8 + 2 * tig + (x & 1);
          qk[at] = aq[j][x];
          kk[at] = ak[j][x];
        }
      }
    }
  }
  __syncthreads();

  const int quad = warp >> 2, qw = warp & 3, qt = tid & 127, per = p.H / p.G;
  uint8_t* mine = reinterpret_cast<uint8_t*>(kk + CL * AP) + quad * quad_bytes<CL>();
  float* sL = reinterpret_cast<float*>(mine);                          // [MT][16][17] diagonal blocks, minus the factors
  __nv_bfloat16* sI = reinterpret_cast<__nv_bfloat16*>(sL + MT * 16 * 17);       // [hi, lo][MT][16][TD] their inverses
  __nv_bfloat16* sT = sI + 2 * MT * 16 * TD;                           // [hi, lo][CL][LT] minus the factors, then T diag(beta)
  float* sb = reinterpret_cast<float*>(sT + 2 * CL * LT);              // [CL] summed log2 decays
  float* sbeta = sb + CL;
  for (int hh = quad; hh < per; hh += 2) {                             // a quad's own heads: its barriers are its own
    const int h = kh * per + hh;
    const size_t at = (size_t)blockIdx.x * p.H + h;
    __nv_bfloat16 *a_hi = p.mats + at * 4 * CL * CL, *a_lo = a_hi + CL * CL, *t_hi = a_lo + CL * CL;
    quad_sync(quad);                                                   // the last head's tiles have been read
    if (qw == 0) {                                                     // inclusive sums over the chunk's rows
      float run = 0.f;
#pragma unroll
      for (int r0 = 0; r0 < CL; r0 += 32) {
        const int t = r0 + lane;
        float b = t < n ? fmaxf(p.log_decay[(size_t)(t0 + t) * p.H + h] * LOG2E, FLOOR) : 0.f;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const float x = __shfl_up_sync(0xffffffffu, b, o);
          if (lane >= o) b += x;
        }
        sb[t] = run + b;
        run += __shfl_sync(0xffffffffu, b, 31);
        sbeta[t] = t < n ? p.beta[(size_t)(t0 + t) * p.H + h] : 0.f;
      }
    }
    quad_sync(quad);
    for (int i = qt; i < CL; i += 128) {
      p.fade[at * 2 * CL + i] = pow2(sb[i]);
      p.fade[at * 2 * CL + CL + i] = pow2(sb[CL - 1] - sb[i]);
    }
    // A, and the factors with their sign turned: two neighbouring columns at a time, up to the end of the diagonal block
    for (int i = qt; i < CL * (CL / 2); i += 128) {
      const int r = i / (CL / 2), s = i % (CL / 2) * 2;
      if (s / 16 > r / 16) continue;
      float a[2], l[2];
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const float dec = s + u <= r ? pow2(sb[r] - sb[s + u]) : 0.f;
        a[u] = s + u <= r ? qk[r * AP + s + u] * dec : 0.f;
        l[u] = s + u < r ? -sbeta[r] * kk[r * AP + s + u] * dec : 0.f;
      }
      uint32_t hi, lo;
      split2(a[0], a[1], hi, lo);
      *reinterpret_cast<uint32_t*>(a_hi + r * CL + s) = hi;
      *reinterpret_cast<uint32_t*>(a_lo + r * CL + s) = lo;
      if (s / 16 == r / 16) {
        sL[(r / 16 * 16 + r % 16) * 17 + s % 16] = l[0];
        sL[(r / 16 * 16 + r % 16) * 17 + s % 16 + 1] = l[1];
      } else {
        split2(l[0], l[1], hi, lo);
        *reinterpret_cast<uint32_t*>(sT + r * LT + s) = hi;
        *reinterpret_cast<uint32_t*>(sT + CL * LT + r * LT + s) = lo;
      }
    }
    quad_sync(quad);
    // T_ii = (I - L_ii)^-1: a warp per block, a column per lane in registers
    if (qw < MT && lane < 16) {
      float x[16];
#pragma unroll
      for (int r = 0; r < 16; ++r) {
        float acc0 = lane == r ? 1.f : 0.f, acc1 = 0.f;
#pragma unroll
        for (int m = 0; m < r; ++m) {
          if (m & 1) acc1 = fmaf(sL[(qw * 16 + r) * 17 + m], x[m], acc1);
          else acc0 = fmaf(sL[(qw * 16 + r) * 17 + m], x[m], acc0);
        }
        x[r] = acc0 + acc1;
        const __nv_bfloat16 hi = __float2bfloat16(x[r]);
        sI[(qw * 16 + r) * TD + lane] = hi;
        sI[(MT * 16 + qw * 16 + r) * TD + lane] = __float2bfloat16(x[r] - __bfloat162float(hi));
      }
    }
    quad_sync(quad);
    // below the diagonal, T_ij = T_ii sum_{k=j}^{i-1} L_ik T_kj: a warp per block column j, transposed, so that a block's
    // accumulators are the left operand of the products it enters.  The warp's blocks stay in registers until L has been read
    uint32_t th[MT][4], tl[MT][4];                                     // T_ij^T, as left operands
    const int j = qw;
    if (j < MT) {
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        if (i == j) {
          ldmatrix_x4_trans(th[i], sI + (i * 16 + (lane & 7) + (lane >> 4) * 8) * TD + ((lane >> 3) & 1) * 8);
          ldmatrix_x4_trans(tl[i], sI + (MT * 16 + i * 16 + (lane & 7) + (lane >> 4) * 8) * TD + ((lane >> 3) & 1) * 8);
        } else if (i > j) {
          float acc[2][4] = {};
#pragma unroll
          for (int k = 0; k < MT; ++k) {
            if (k < j || k >= i) continue;
            uint32_t bh[4], bl[4];                                     // L_ik^T: rows of L_ik are columns
            const int off = (i * 16 + (lane & 7) + (lane >> 4) * 8) * LT + k * 16 + ((lane >> 3) & 1) * 8;
            ldmatrix_x4(bh, sT + off);
            ldmatrix_x4(bl, sT + CL * LT + off);
#pragma unroll
            for (int x = 0; x < 2; ++x) {
              mma(acc[x], th[k], bh[2 * x], bh[2 * x + 1]);
              mma(acc[x], th[k], bl[2 * x], bl[2 * x + 1]);
              mma(acc[x], tl[k], bh[2 * x], bh[2 * x + 1]);
            }
          }
          uint32_t ah[4], al[4], bh[4], bl[4];
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            split2(acc[x][0], acc[x][1], ah[2 * x], al[2 * x]);
            split2(acc[x][2], acc[x][3], ah[2 * x + 1], al[2 * x + 1]);
          }
          const int off = (i * 16 + (lane & 7) + (lane >> 4) * 8) * TD + ((lane >> 3) & 1) * 8;
          ldmatrix_x4(bh, sI + off);
          ldmatrix_x4(bl, sI + MT * 16 * TD + off);
          float t[2][4] = {};
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            mma(t[x], ah, bh[2 * x], bh[2 * x + 1]);
            mma(t[x], ah, bl[2 * x], bl[2 * x + 1]);
            mma(t[x], al, bh[2 * x], bh[2 * x + 1]);
            split2(t[x][0], t[x][1], th[i][2 * x], tl[i][2 * x]);
            split2(t[x][2], t[x][3], th[i][2 * x + 1], tl[i][2 * x + 1]);
          }
        }
      }
    }
    quad_sync(quad);
    if (j < MT) {
      // element (m, n) of T_ij^T is T[16 i + n][16 j + m], times the beta of its column
      const float b0 = sbeta[j * 16 + g], b1 = sbeta[j * 16 + g + 8];
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        if (i < j) continue;
#pragma unroll
        for (int x = 0; x < 4; ++x) {                                  // rows g + 8 (x & 1), columns 2 tig (+ 1) + 8 (x >> 1)
          const float2 h2 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&th[i][x]));
          const float2 l2 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&tl[i][x]));
          const float f = x & 1 ? b1 : b0;
          uint32_t hi, lo;
          split2((h2.x + l2.x) * f, (h2.y + l2.y) * f, hi, lo);
          const int col = j * 16 + g + 8 * (x & 1), row = i * 16 + 2 * tig + 8 * (x >> 1);
          const __nv_bfloat162 h = *reinterpret_cast<const __nv_bfloat162*>(&hi), l = *reinterpret_cast<const __nv_bfloat162*>(&lo);
          sT[row * LT + col] = h.x;
          sT[(row + 1) * LT + col] = h.y;
          sT[CL * LT + row * LT + col] = l.x;
          sT[CL * LT + (row + 1) * LT + col] = l.y;
        }
      }
    }
    quad_sync(quad);
    for (int i = qt; i < 2 * CL * (CL / 8); i += 128) {
      const int r = i / (CL / 8), s = i % (CL / 8) * 8;                // rows of the second term follow the first's
      if (s / 16 <= (r % CL) / 16) *reinterpret_cast<uint4*>(t_hi + r * CL + s) = *reinterpret_cast<const uint4*>(sT + r * LT + s);
    }
  }
}

// Shared memory of the scan: rows of two chunks, matrices of one, state, X, U and the faded U (two terms each).
template <int DT, int CL>
__host__ __device__ constexpr size_t front_elems() { return (size_t)4 * CL * (DT + 8); }
template <int CL>
__host__ __device__ constexpr size_t back_elems() { return (size_t)4 * CL * (CL + 8); }
template <int DT, int CL>
constexpr size_t scan_smem(int VB) {
  return (2 * front_elems<DT, CL>() + back_elems<CL>() + (size_t)2 * VB * (DT + 8) + (size_t)6 * CL * (VB + 8)) * 2 + (size_t)4 * CL * 4;
}

// grid (ceil(V / (16 NG)), H, entries), eight warps.
template <int DT, int CL, int NG>
__global__ void __launch_bounds__(256) delta_scan_kernel(DeltaParams p) {
  constexpr int LQ = DT + 8, LA = CL + 8, MT = CL / 16, ND = DT / 8, NS = ND / 8, VB = 16 * NG, LX = VB + 8, NN = 2 * NG, NW = 256;
  // channels and fragments of S^T of a warp; 8-column tiles of a row of X or O
  extern __shared__ __align__(16) uint8_t smem[];
  __nv_bfloat16* front = reinterpret_cast<__nv_bfloat16*>(smem);
  __nv_bfloat16* back = front + 2 * front_elems<DT, CL>();
  __nv_bfloat16* ss = back + back_elems<CL>();                         // [hi, lo][VB][LQ] S^T
  __nv_bfloat16* sx = ss + 2 * VB * LQ;                                // [hi, lo][CL][LX] X
  __nv_bfloat16* su = sx + 2 * CL * LX;                                // [hi, lo][CL][LX] U
  __nv_bfloat16* sf = su + 2 * CL * LX;                                // [hi, lo][CL][LX] faded U
  float* fade = reinterpret_cast<float*>(sf + 2 * CL * LX);            // [2 chunks][2][CL]
  const int tid = threadIdx.x, warp = __shfl_sync(0xffffffffu, tid >> 5, 0), lane = tid & 31, g = lane >> 2, tig = lane & 3;
  const int h = blockIdx.y, e = blockIdx.z, v0 = blockIdx.x * VB, kh = h / (p.H / p.G);
  pdl_grid_trigger();
  pdl_grid_wait();
  const int chunks = chunks_of(p, e, CL);
  if (chunks == 0) return;
  int base = 0;
  for (int i = 0; i < e; ++i) base += chunks_of(p, i, CL);
  const int r0 = p.first[e], len = p.length[e];
  auto fetch_front = [&](int c) {
    const __nv_bfloat16* src = p.rows + ((size_t)(base + c) * p.G + kh) * 4 * CL * DT;
    __nv_bfloat16* dst = front + (c & 1) * front_elems<DT, CL>();
#pragma unroll 4
    for (int i = tid; i < 4 * CL * (DT / 8); i += NW) {
      const int r = i / (DT / 8), d = i % (DT / 8) * 8;
      cp16(dst + r * LQ + d, src + (size_t)r * DT + d, true);
    }
    const float* f = p.fade + ((size_t)(base + c) * p.H + h) * 2 * CL;
    if (tid < 2 * CL / 4) cp16(fade + (c & 1) * 2 * CL + tid * 4, f + tid * 4, true);
  };
  auto fetch_back = [&](int c) {
    const __nv_bfloat16* src = p.mats + ((size_t)(base + c) * p.H + h) * 4 * CL * CL;
#pragma unroll 4
    for (int i = tid; i < 4 * CL * (CL / 8); i += NW) {
      const int r = i / (CL / 8), s = i % (CL / 8) * 8;
      if (s / 16 <= (r % CL) / 16) cp16(back + r * LA + s, src + (size_t)r * CL + s, true);
    }
  };
  fetch_front(0);
  cp_commit();
  const int m = warp & 3, d_own = warp * ND;
  const bool keys = warp < 4, reads = m < MT;
  float* st = p.state + ((size_t)p.slot[e] * p.H + h) * p.D * p.V;
  const bool fresh = p.positions[r0] == 0;
  float S[NG][NS][4];                                                  // S^T: columns 16 n + g (+ 8), channels d_own + 8 i + 2 tig (+ 1)
#pragma unroll
  for (int n = 0; n < NG; ++n)
#pragma unroll
    for (int i = 0; i < NS; ++i)
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int d = d_own + i * 8 + 2 * tig + (x & 1), v = v0 + n * 16 + g + 8 * (x >> 1);
        S[n][i][x] = !fresh && d < p.D && v < p.V ? st[(size_t)d * p.V + v] : 0.f;
      }
  auto publish = [&]() {
#pragma unroll
    for (int n = 0; n < NG; ++n)
#pragma unroll
      for (int i = 0; i < NS; ++i)
#pragma unroll
        for (int w = 0; w < 2; ++w) {
          uint32_t hi, lo;
          split2(S[n][i][2 * w], S[n][i][2 * w + 1], hi, lo);
          __nv_bfloat16* dst = ss + (n * 16 + g + 8 * w) * LQ + d_own + i * 8 + 2 * tig;
          *reinterpret_cast<uint32_t*>(dst) = hi;
          *reinterpret_cast<uint32_t*>(dst + VB * LQ) = lo;
        }
  };
  publish();
  uint32_t v_next[NN][2];                                              // values of the next chunk: rows g, g + 8 of the warp's tile
  auto load_v = [&](int c) {
    if (keys && reads)
#pragma unroll
      for (int w = 0; w < 2; ++w) {
        const int t = c * CL + m * 16 + g + 8 * w;
#pragma unroll
        for (int n = 0; n < NN; ++n) {
          const int v = v0 + n * 8 + 2 * tig;
          v_next[n][w] = t < len && v < p.V ? *reinterpret_cast<const uint32_t*>(p.v + (size_t)(r0 + t) * p.ldv + (size_t)h * p.V + v) : 0u;
        }
      }
  };
  load_v(0);
  const int row16 = lane & 15, col8 = (lane >> 4) * 8;                           // non-transposed 16 x 16 tiles, left operand
  const int brow = (lane & 7) + (lane >> 4) * 8, bcol = ((lane >> 3) & 1) * 8;   // left operand, transposed
  const int trow = (lane & 7) + ((lane >> 3) & 1) * 8;                           // right operand, transposed
  for (int c = 0; c < chunks; ++c) {
    cp_wait<0>();
    __syncthreads();                                    // rows, decays and state landed; the buffers' last readers are done
    fetch_back(c);
    cp_commit();
    const bool more = c + 1 < chunks;
    if (more) fetch_front(c + 1);
    cp_commit();
    const __nv_bfloat16* sk = front + (c & 1) * front_elems<DT, CL>();
    const __nv_bfloat16* sa = back;
    const __nv_bfloat16* st_ = back + 2 * CL * LA;      // T diag(beta)
    const float* eb = fade + (c & 1) * 2 * CL;
    // K S or q S: 16 rows, all columns
    float o[NN][4] = {}, ol[NN][4] = {};                // sums of the leading and of the correcting products
    if (reads) {
      const __nv_bfloat16* a_rows = sk + (keys ? 0 : 2 * CL * LQ) + (m * 16 + row16) * LQ + col8;
#pragma unroll
      for (int k2 = 0; k2 < DT / 32; ++k2) {
        uint32_t bh[NN][4], bl[NN][4];                  // two k-steps of 8 columns
#pragma unroll
        for (int n = 0; n < NN; ++n) {
          const __nv_bfloat16* b = ss + (n * 8 + (lane & 7)) * LQ + k2 * 32 + (lane >> 3) * 8;
          ldmatrix_x4(bh[n], b);
          ldmatrix_x4(bl[n], b + VB * LQ);
        }
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          uint32_t ah[4], al[4];
          ldmatrix_x4(ah, a_rows + k2 * 32 + x * 16);
          ldmatrix_x4(al, a_rows + CL * LQ + k2 * 32 + x * 16);
#pragma unroll
          for (int n = 0; n < NN; ++n) mma(o[n], ah, bh[n][2 * x], bh[n][2 * x + 1]);
#pragma unroll
          for (int n = 0; n < NN; ++n) mma(ol[n], ah, bl[n][2 * x], bl[n][2 * x + 1]);
#pragma unroll
          for (int n = 0; n < NN; ++n) mma(ol[n], al, bh[n][2 * x], bh[n][2 * x + 1]);
        }
      }
      const float e0 = eb[m * 16 + g], e1 = eb[m * 16 + g + 8];
#pragma unroll
      for (int n = 0; n < NN; ++n) {
        o[n][0] = (o[n][0] + ol[n][0]) * e0;
        o[n][1] = (o[n][1] + ol[n][1]) * e0;
        o[n][2] = (o[n][2] + ol[n][2]) * e1;
        o[n][3] = (o[n][3] + ol[n][3]) * e1;
        if (keys) {
#pragma unroll
          for (int w = 0; w < 2; ++w) {
            const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v_next[n][w]));
            uint32_t hi, lo;
            split2(v.x - o[n][2 * w], v.y - o[n][2 * w + 1], hi, lo);
            __nv_bfloat16* dst = sx + (m * 16 + g + 8 * w) * LX + n * 8 + 2 * tig;
            *reinterpret_cast<uint32_t*>(dst) = hi;
            *reinterpret_cast<uint32_t*>(dst + CL * LX) = lo;
          }
        }
      }
    }
    if (more) load_v(c + 1);
    cp_wait<1>();                                       // the matrices; the next rows may be on their way
    __syncthreads();                                    // X and the matrices landed; everyone has read the state of before the chunk
    if (reads) {
      // U: 16 rows, half the columns
      const int n0 = keys ? 0 : NG;                     // first 8-column tile
      float u[NG][4] = {}, ul[NG][4] = {};
      uint32_t bh[4], bl[4], ah[4], al[4];
#pragma unroll
      for (int ks = 0; ks < MT; ++ks) {
        if (ks > m) break;
        ldmatrix_x4(ah, st_ + (m * 16 + row16) * LA + ks * 16 + col8);
        ldmatrix_x4(al, st_ + (CL + m * 16 + row16) * LA + ks * 16 + col8);
        if (NG == 2) {
          ldmatrix_x4_trans(bh, sx + (ks * 16 + trow) * LX + n0 * 8 + col8);
          ldmatrix_x4_trans(bl, sx + CL * LX + (ks * 16 + trow) * LX + n0 * 8 + col8);
#pragma unroll
          for (int n = 0; n < NG; ++n) mma(u[n], ah, bh[2 * n], bh[2 * n + 1]);
#pragma unroll
          for (int n = 0; n < NG; ++n) {
            mma(ul[n], ah, bl[2 * n], bl[2 * n + 1]);
            mma(ul[n], al, bh[2 * n], bh[2 * n + 1]);
          }
        } else {                                        // eight columns: both terms in one load
          ldmatrix_x4_trans(bh, sx + (lane >> 4) * CL * LX + (ks * 16 + trow) * LX + n0 * 8);
          mma(u[0], ah, bh[0], bh[1]);
          mma(ul[0], ah, bh[2], bh[3]);
          mma(ul[0], al, bh[0], bh[1]);
        }
      }
      const float f0 = eb[CL + m * 16 + g], f1 = eb[CL + m * 16 + g + 8];
#pragma unroll
      for (int n = 0; n < NG; ++n)
#pragma unroll
        for (int w = 0; w < 2; ++w) {
          const float a = u[n][2 * w] + ul[n][2 * w], b = u[n][2 * w + 1] + ul[n][2 * w + 1], f = w ? f1 : f0;
          uint32_t hi, lo;
          const int at = (m * 16 + g + 8 * w) * LX + (n0 + n) * 8 + 2 * tig;
          split2(a, b, hi, lo);
          *reinterpret_cast<uint32_t*>(su + at) = hi;
          *reinterpret_cast<uint32_t*>(su + CL * LX + at) = lo;
          split2(a * f, b * f, hi, lo);
          *reinterpret_cast<uint32_t*>(sf + at) = hi;
          *reinterpret_cast<uint32_t*>(sf + CL * LX + at) = lo;
        }
    }
    __syncthreads();
    {
      const float end = eb[CL - 1];
#pragma unroll
      for (int n = 0; n < NG; ++n)
#pragma unroll
        for (int i = 0; i < NS; ++i)
#pragma unroll
          for (int x = 0; x < 4; ++x) S[n][i][x] *= end;
#pragma unroll
      for (int ks = 0; ks < MT; ++ks) {
        uint32_t ah[NG][4], al[NG][4];
#pragma unroll
        for (int n = 0; n < NG; ++n) {
          ldmatrix_x4_trans(ah[n], sf + (ks * 16 + brow) * LX + n * 16 + bcol);
          ldmatrix_x4_trans(al[n], sf + CL * LX + (ks * 16 + brow) * LX + n * 16 + bcol);
        }
#pragma unroll
        for (int i = 0; i < NS; ++i) {
          uint32_t b[4];                                // eight channels: both terms in one load
          ldmatrix_x4_trans(b, sk + (lane >> 4) * CL * LQ + (ks * 16 + trow) * LQ + d_own + i * 8);
#pragma unroll
          for (int n = 0; n < NG; ++n) mma(S[n][i], ah[n], b[0], b[1]);
#pragma unroll
          for (int n = 0; n < NG; ++n) mma(S[n][i], ah[n], b[2], b[3]);
#pragma unroll
          for (int n = 0; n < NG; ++n) mma(S[n][i], al[n], b[0], b[1]);
        }
      }
      publish();                                        // the next chunk starts from it: the outputs come after
    }
    if (!keys && reads) {
#pragma unroll
      for (int n = 0; n < NN; ++n)
#pragma unroll
        for (int x = 0; x < 4; ++x) ol[n][x] = 0.f;
#pragma unroll
      for (int ks = 0; ks < MT; ++ks) {
        if (ks > m) break;
        uint32_t ah[4], al[4];
        ldmatrix_x4(ah, sa + (m * 16 + row16) * LA + ks * 16 + col8);
        ldmatrix_x4(al, sa + (CL + m * 16 + row16) * LA + ks * 16 + col8);
#pragma unroll
        for (int n = 0; n < NG; ++n) {
          uint32_t bh[4], bl[4];
          ldmatrix_x4_trans(bh, su + (ks * 16 + trow) * LX + n * 16 + col8);
          ldmatrix_x4_trans(bl, su + CL * LX + (ks * 16 + trow) * LX + n * 16 + col8);
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            mma(o[2 * n + x], ah, bh[2 * x], bh[2 * x + 1]);
            mma(ol[2 * n + x], ah, bl[2 * x], bl[2 * x + 1]);
            mma(ol[2 * n + x], al, bh[2 * x], bh[2 * x + 1]);
          }
        }
      }
#pragma unroll
      for (int w = 0; w < 2; ++w) {
        const int t = c * CL + m * 16 + g + 8 * w;
        if (t < len) {
          float* dst = p.o + ((size_t)(r0 + t) * p.H + h) * p.V + v0 + 2 * tig;
#pragma unroll
          for (int n = 0; n < NN; ++n)
            if (v0 + n * 8 < p.V)
              *reinterpret_cast<float2*>(dst + n * 8) = make_float2(o[n][2 * w] + ol[n][2 * w], o[n][2 * w + 1] + ol[n][2 * w + 1]);
        }
      }
    }
  }
  cp_wait<0>();
#pragma unroll
  for (int n = 0; n < NG; ++n)
#pragma unroll
    for (int i = 0; i < NS; ++i)
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int d = d_own + i * 8 + 2 * tig + (x & 1), v = v0 + n * 16 + g + 8 * (x >> 1);
        if (d < p.D && v < p.V) st[(size_t)d * p.V + v] = S[n][i][x];
      }
}

template <typename K>
int configure(K kernel, bool& configured) {
  if (configured) return 0;
  const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
  configured = e == cudaSuccess;
  return (int)e;
}

template <int DT, int CL, int NG>
int launch_scan(const DeltaParams& p, cudaStream_t stream) {
  static PerDeviceOnce once_;
  const int e = configure(delta_scan_kernel<DT, CL, NG>, once_.slot());
  return e ? e : (int)launch_pdl(delta_scan_kernel<DT, CL, NG>, dim3((p.V + 16 * NG - 1) / (16 * NG), p.H, p.entries), dim3(256),
                                 scan_smem<DT, CL>(16 * NG), stream, p);
}

template <int DT, int CL>
int launch(const DeltaParams& p, int chunks, cudaStream_t stream) {
  static PerDeviceOnce once_;
  int e = configure(delta_prep_kernel<DT, CL>, once_.slot());
  if (e) return e;
  e = (int)launch_pdl(delta_prep_kernel<DT, CL>, dim3(chunks, p.G), dim3(PT), prep_smem<DT, CL>(), stream, p);
  if (e) return e;
  // 16 columns per block where one wave of blocks takes them, 32 otherwise
  if (p.V > 16 && (long long)p.entries * p.H * ((p.V + 15) / 16) > 148) return launch_scan<DT, CL, 2>(p, stream);
  return launch_scan<DT, CL, 1>(p, stream);
}

}  // namespace

// Rows per chunk for D key channels (0: not covered), and channels per row of the workspace.
extern "C" int b200_delta_chunk_rows(int D) { return D <= 0 || D % 16 || D > 256 ? 0 : D <= 128 ? 64 : 32; }
extern "C" int b200_delta_chunk_width(int D) { return D <= 64 ? 64 : D <= 128 ? 128 : 256; }

// Entries with at least min_len rows; chunks: upper bound on their number (rows / chunk rows + entries).  q, k fp32 [rows, G, D]
// (b200_delta_prep), v bf16 rows `ldv` apart, log_decay and beta fp32 [rows, H].  D, V multiples of 16, D <= 256.  Workspace, with
// n rows per chunk and w channels: `rows` bf16 [chunks, G, 4 n w], `mats` bf16 [chunks, H, 4 n n], `fade` fp32 [chunks, H, 2 n].
// state [slots, H, D, V] fp32 in place; o fp32 [rows, H * V].
extern "C" int b200_delta_chunk(const float* q, const float* k, const void* v, int ldv, const float* log_decay, const float* beta,
                                float* state, float* o, const int* first, const int* length, const int* slot, const int* positions,
                                int entries, int min_len, int chunks, void* rows, void* mats, float* fade, int H, int G, int D, int V,
                                cudaStream_t stream) {
  if (!b200_delta_chunk_rows(D) || V <= 0 || (V & 15) || (ldv & 7) || entries <= 0 || entries > 65535 || H <= 0 || H > 65535 || G <= 0 ||
      H % G || chunks <= 0 || !log_decay || !beta)
    return -6;
  DeltaParams p;
  p.q = q; p.k = k; p.v = reinterpret_cast<const __nv_bfloat16*>(v); p.log_decay = log_decay; p.beta = beta; p.state = state; p.o = o;
  p.first = first; p.length = length; p.slot = slot; p.positions = positions; p.rows = reinterpret_cast<__nv_bfloat16*>(rows);
  p.mats = reinterpret_cast<__nv_bfloat16*>(mats); p.fade = fade; p.ldv = ldv; p.H = H; p.G = G; p.D = D; p.V = V; p.entries = entries;
  p.min_len = min_len;
  if (D <= 64) return launch<64, 64>(p, chunks, stream);
  if (D <= 128) return launch<128, 64>(p, chunks, stream);
  return launch<256, 32>(p, chunks, stream);
}
