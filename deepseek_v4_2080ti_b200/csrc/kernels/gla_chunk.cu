// Gated linear attention (see gated_linear.cu) over prompt portions in chunks of CL rows, bf16 inputs.  With b_t the sum of the
// log decays of a chunk up to row t (per key channel), S the state before the chunk:
//
//   o_t  = (q_t e^{b_t}) S + sum_{s <= t} A_ts v_s,       A_ts = sum_d q_td k_sd e^{b_td - b_sd}
//   S'   = diag(e^{b_end}) S + sum_s (k_s e^{b_end - b_s}) v_s^T
//
// No factor ever grows: exponents are differences taken towards the later row.  A is built from blocks of 16 rows: blocks below
// the diagonal as products of q e^{b_t - b_ref} and k e^{b_ref - b_s} with the reference between the two blocks, diagonal
// blocks element by element (the two-level chunking of Yang et al., "Gated Linear Attention Transformers with
// Hardware-Efficient Training").
//
//   gla_chunk_prep   one block per chunk and head: decayed q and k, A, e^{b_end} -> workspace
//   gla_chunk_scan   four or eight warps per 16 value columns walk the chunks.  Each keeps its share of the channels of
//                    S^T in registers and updates it; for q S, of which each takes 16 rows and 8 columns (or 16), the
//                    shares are exchanged through shared memory once per chunk
//
// Decayed operands, A and the state enter the products as two bf16 terms (16 significant bits); sums are fp32.
#include <cuda_bf16.h>
#include <stdint.h>
#include "launch.h"
#include "ops.h"
#include "per_device.h"
#include "split_mma.cuh"

namespace {
using namespace b200;

constexpr float LOG2E = 1.4426950408889634f;

struct ChunkParams {
  const __nv_bfloat16 *q, *k, *v;  // head h of row t at ptr + t * ld + h * D (V)
  const float* la;                 // [rows, H * D] log decays
  float* state;                    // [slots, H, D, V]
  float* o;                        // [rows, H * V]
  const int *first, *length, *slot, *positions;
  __nv_bfloat16* ws;               // per chunk and head: q hi | q lo | k hi | k lo [CL, DT], A hi | A lo [CL, CL]
  float* end;                      // per chunk and head: [DT] e^{b_end}
  int ld, H, D, V, entries, min_len;
  float scale;
};

__device__ __forceinline__ int chunks_of(const ChunkParams& p, int e, int CL) {
  const int n = p.length[e];
  return n < p.min_len ? 0 : (n + CL - 1) / CL;
}

template <int DT, int CL>
constexpr size_t ws_elems() { return (size_t)4 * CL * DT + 2 * CL * CL; }

constexpr int PT = 256;

// grid (chunks, H).  Warps 0 .. CL / 16 - 1 take the diagonal blocks of A, the next ones the blocks to the left.
template <int DT, int CL>
__global__ void __launch_bounds__(PT) gla_chunk_prep_kernel(ChunkParams p) {
  constexpr int LB = DT + 4, LQ = DT + 8, X = DT / 32;
  extern __shared__ __align__(16) uint8_t smem[];
  float* sb = reinterpret_cast<float*>(smem);                       // [CL][LB] summed log2 decays
  __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(sb + CL * LB);   // [CL][LQ]
  __nv_bfloat16* sk = sq + CL * LQ;
  pdl_grid_trigger();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tig = lane & 3, h = blockIdx.y;
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
  __nv_bfloat16* ws = p.ws + at * ws_elems<DT, CL>();
  const uint4 zero = make_uint4(0, 0, 0, 0);
  for (int i = tid; i < CL * (DT / 8); i += PT) {
    const int t = i / (DT / 8), d = i % (DT / 8) * 8;
    const bool ok = t < n && d < p.D;                               // D is a multiple of 16
    const size_t row = (size_t)(t0 + t);
    *reinterpret_cast<uint4*>(sq + t * LQ + d) = ok ? *reinterpret_cast<const uint4*>(p.q + row * p.ld + h * p.D + d) : zero;
    *reinterpret_cast<uint4*>(sk + t * LQ + d) = ok ? *reinterpret_cast<const uint4*>(p.k + row * p.ld + h * p.D + d) : zero;
    const float4* la = reinterpret_cast<const float4*>(p.la + (row * p.H + h) * p.D + d);
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      float4 f = ok ? la[u] : make_float4(0.f, 0.f, 0.f, 0.f);
      f.x *= LOG2E; f.y *= LOG2E; f.z *= LOG2E; f.w *= LOG2E;
      *reinterpret_cast<float4*>(sb + t * LB + d + 4 * u) = f;
    }
  }
  __syncthreads();
  for (int d = tid; d < DT; d += PT) {
    float acc = 0.f;
    for (int t = 0; t < CL; t += 16) {
      float f[16];
#pragma unroll
      for (int j = 0; j < 16; ++j) f[j] = sb[(t + j) * LB + d];
#pragma unroll
      for (int j = 0; j < 16; ++j) sb[(t + j) * LB + d] = acc += f[j];
    }
    p.end[at * DT + d] = pow2(acc);
  }
  __syncthreads();
  // decayed queries and keys
  for (int i = tid; i < CL * (DT / 8); i += PT) {
    const int t = i / (DT / 8), d = i % (DT / 8) * 8;
    uint4 hi[2], lo[2];
    uint32_t* H[2] = {reinterpret_cast<uint32_t*>(&hi[0]), reinterpret_cast<uint32_t*>(&hi[1])};
    uint32_t* L[2] = {reinterpret_cast<uint32_t*>(&lo[0]), reinterpret_cast<uint32_t*>(&lo[1])};
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 q = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sq + t * LQ + d + 2 * j));
      const float2 k = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sk + t * LQ + d + 2 * j));
      const float2 b = *reinterpret_cast<const float2*>(sb + t * LB + d + 2 * j);
      const float2 z = *reinterpret_cast<const float2*>(sb + (CL - 1) * LB + d + 2 * j);
      split2(q.x * p.scale * pow2(b.x), q.y * p.scale * pow2(b.y), H[0][j], L[0][j]);
      split2(k.x * pow2(z.x - b.x), k.y * pow2(z.y - b.y), H[1][j], L[1][j]);
    }
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      *reinterpret_cast<uint4*>(ws + (size_t)(2 * u) * CL * DT + t * DT + d) = hi[u];
      *reinterpret_cast<uint4*>(ws + (size_t)(2 * u + 1) * CL * DT + t * DT + d) = lo[u];
    }
  }
  __nv_bfloat16 *a_hi = ws + (size_t)4 * CL * DT, *a_lo = a_hi + CL * CL;
  const int i0 = warp % (CL / 16) * 16;
  // diagonal block: a lane owns channels lane, lane + 32, ...
  if (warp < CL / 16) {
#pragma unroll 1
    for (int t = 0; t < 16; ++t) {
      float q[X], b[X], mine = 0.f;
#pragma unroll
      for (int x = 0; x < X; ++x) {
        q[x] = __bfloat162float(sq[(i0 + t) * LQ + lane + 32 * x]) * p.scale;
        b[x] = sb[(i0 + t) * LB + lane + 32 * x];
      }
#pragma unroll 4
      for (int s = 0; s <= t; ++s) {
        float a = 0.f;
#pragma unroll
        for (int x = 0; x < X; ++x)
          a = fmaf(q[x] * __bfloat162float(sk[(i0 + s) * LQ + lane + 32 * x]), pow2(b[x] - sb[(i0 + s) * LB + lane + 32 * x]), a);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) a += __shfl_xor_sync(0xffffffffu, a, o);
        if (lane == s) mine = a;
      }
      if (lane < 16) {
        const __nv_bfloat16 hi = __float2bfloat16(mine);
        a_hi[(i0 + t) * CL + i0 + lane] = hi;
        a_lo[(i0 + t) * CL + i0 + lane] = __float2bfloat16(mine - __bfloat162float(hi));
      }
    }
    return;
  }
  // blocks to the left, 8 columns at a time, against the last row before this block
  if (i0 == 0 || warp >= CL / 8) return;
  constexpr int NT = (CL / 16 - 1) * 2;
  float acc[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
  const float* ref = sb + (i0 - 1) * LB;
#pragma unroll 1
  for (int d0 = 0; d0 < DT; d0 += 16) {
    uint32_t ah[4], al[4];
    float2 r[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int d = d0 + u * 8 + 2 * tig;
      r[u] = *reinterpret_cast<const float2*>(ref + d);
#pragma unroll
      for (int w = 0; w < 2; ++w) {
        const int t = i0 + g + 8 * w;
        const float2 q = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sq + t * LQ + d));
        const float2 b = *reinterpret_cast<const float2*>(sb + t * LB + d);
        split2(q.x * p.scale * pow2(b.x - r[u].x), q.y * p.scale * pow2(b.y - r[u].y), ah[u * 2 + w], al[u * 2 + w]);
      }
    }
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      if (j * 8 >= i0) continue;
      uint32_t bh[2], bl[2];
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int d = d0 + u * 8 + 2 * tig, s = j * 8 + g;
        const float2 k = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sk + s * LQ + d));
        const float2 b = *reinterpret_cast<const float2*>(sb + s * LB + d);
        split2(k.x * pow2(r[u].x - b.x), k.y * pow2(r[u].y - b.y), bh[u], bl[u]);
      }
      mma(acc[j], ah, bh[0], bh[1]);
      mma(acc[j], ah, bl[0], bl[1]);
      mma(acc[j], al, bh[0], bh[1]);
    }
  }
#pragma unroll
  for (int j = 0; j < NT; ++j) {
    if (j * 8 >= i0) continue;
#pragma unroll
    for (int w = 0; w < 2; ++w) {
      uint32_t hi, lo;
      split2(acc[j][2 * w], acc[j][2 * w + 1], hi, lo);
      const size_t x = (size_t)(i0 + g + 8 * w) * CL + j * 8 + 2 * tig;
      *reinterpret_cast<uint32_t*>(a_hi + x) = hi;
      *reinterpret_cast<uint32_t*>(a_lo + x) = lo;
    }
  }
}

template <int DT, int CL>
__host__ __device__ constexpr size_t stage_bytes(int VB) {
  return ((size_t)4 * CL * (DT + 8) + 2 * CL * (CL + 8) + CL * (VB + 8)) * 2 + DT * 4;
}
template <int DT, int CL>
constexpr size_t scan_smem(int VB) { return 2 * stage_bytes<DT, CL>(VB) + (size_t)2 * VB * (DT + 8) * 2; }

// grid (ceil(V / VB), H, entries), W VB / 16 warps: W of them (4 or 8) own value columns 16 i .. 16 i + 15.
template <int DT, int CL, int W>
__global__ void __launch_bounds__(512) gla_chunk_scan_kernel(ChunkParams p) {
  constexpr int LQ = DT + 8, LA = CL + 8, MT = CL / 16, ND = DT / W, NS = ND / 8, NJ = W == 8 ? 1 : 2;
  // channels, fragments of S^T and 8-column tiles of the output of a warp
  extern __shared__ __align__(16) uint8_t smem[];
  const int tid = threadIdx.x, nthr = blockDim.x, lane = tid & 31, g = lane >> 2, tig = lane & 3;
  const int vg = tid / (32 * W), sub = (tid >> 5) % W;
  const int VB = nthr / (2 * W), LV = VB + 8, h = blockIdx.y, e = blockIdx.z, v0 = blockIdx.x * VB;
  const size_t stage = stage_bytes<DT, CL>(VB);
  __nv_bfloat16* ss = reinterpret_cast<__nv_bfloat16*>(smem + 2 * stage) + (size_t)vg * 2 * 16 * LQ;     // [hi, lo][16][LQ]
  pdl_grid_trigger();
  pdl_grid_wait();
  const int chunks = chunks_of(p, e, CL);
  if (chunks == 0) return;
  int base = 0;
  for (int i = 0; i < e; ++i) base += chunks_of(p, i, CL);
  const int r0 = p.first[e], len = p.length[e];
  auto fetch = [&](int c, int buf) {
    const size_t at = (size_t)(base + c) * p.H + h;
    const __nv_bfloat16* ws = p.ws + at * ws_elems<DT, CL>();
    __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(smem + buf * stage);
    for (int i = tid; i < 4 * CL * (DT / 8); i += nthr) {
      const int r = i / (DT / 8), d = i % (DT / 8) * 8;
      cp16(dst + r * LQ + d, ws + (size_t)r * DT + d, true);
    }
    dst += 4 * CL * LQ;
    ws += (size_t)4 * CL * DT;
    for (int i = tid; i < 2 * CL * (CL / 8); i += nthr) {
      const int r = i / (CL / 8), s = i % (CL / 8) * 8;
      cp16(dst + r * LA + s, ws + r * CL + s, true);
    }
    dst += 2 * CL * LA;
    for (int i = tid; i < CL * (VB / 8); i += nthr) {
      const int r = i / (VB / 8), x = i % (VB / 8) * 8;
      const bool ok = c * CL + r < len && v0 + x < p.V;
      cp16(dst + r * LV + x, p.v + (ok ? (size_t)(r0 + c * CL + r) * p.ld + h * p.V + v0 + x : 0), ok);
    }
    float* end = reinterpret_cast<float*>(dst + CL * LV);
    for (int i = tid; i < DT / 4; i += nthr) cp16(end + i * 4, p.end + at * DT + i * 4, true);
    cp_commit();
  };
  fetch(0, 0);
  const int vw = v0 + vg * 16, d_own = sub * ND;
  const bool live = vw < p.V;
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
  const int row16 = lane & 15, col8 = (lane >> 4) * 8;                       // non-transposed 16 x 16 tiles, left operand
  const int brow = (lane & 7) + (lane >> 4) * 8, bcol = ((lane >> 3) & 1) * 8;   // right operand stored by column; left, transposed
  const int trow = (lane & 7) + ((lane >> 3) & 1) * 8;                       // right operand, transposed
  for (int c = 0; c < chunks; ++c) {
    cp_wait<0>();
    __syncthreads();                                    // chunk and state landed; the other buffer's readers are done
    if (c + 1 < chunks) fetch(c + 1, (c + 1) & 1);
    const __nv_bfloat16* sq = reinterpret_cast<const __nv_bfloat16*>(smem + (c & 1) * stage);
    const __nv_bfloat16* sk = sq + 2 * CL * LQ;
    const __nv_bfloat16* sa = sk + 2 * CL * LQ;
    const __nv_bfloat16* sv = sa + 2 * CL * LA;
    const float* end = reinterpret_cast<const float*>(sv + CL * LV);
    if (live && sub < MT * 2 / NJ) {
      const int m = NJ == 2 ? sub : sub >> 1, j0 = NJ == 2 ? 0 : sub & 1;
      float o[NJ][4] = {}, ol[NJ][4] = {};              // sums of the leading and of the correcting products
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
        for (int u = 0; u < 2; ++u) {
          uint32_t ah[4], al[4];
          ldmatrix_x4(ah, sq + (m * 16 + row16) * LQ + k2 * 32 + u * 16 + col8);
          ldmatrix_x4(al, sq + (CL + m * 16 + row16) * LQ + k2 * 32 + u * 16 + col8);
#pragma unroll
          for (int j = 0; j < NJ; ++j) {
            mma(o[j], ah, bh[j][2 * u], bh[j][2 * u + 1]);
            mma(ol[j], ah, bl[j][2 * u], bl[j][2 * u + 1]);
            mma(ol[j], al, bh[j][2 * u], bh[j][2 * u + 1]);
          }
        }
      }
#pragma unroll
      for (int ks = 0; ks < MT; ++ks) {
        if (ks > m) break;
        uint32_t b[4], ah[4], al[4];
        ldmatrix_x4_trans(b, sv + (ks * 16 + trow) * LV + vg * 16 + col8);
        ldmatrix_x4(ah, sa + (m * 16 + row16) * LA + ks * 16 + col8);
        ldmatrix_x4(al, sa + (CL + m * 16 + row16) * LA + ks * 16 + col8);
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
          const uint32_t b0 = j0 + j ? b[2] : b[0], b1 = j0 + j ? b[3] : b[1];
          mma(o[j], ah, b0, b1);
          mma(ol[j], al, b0, b1);
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
    if (live) {
#pragma unroll
      for (int i = 0; i < NS; ++i) {
        const float2 f = *reinterpret_cast<const float2*>(end + d_own + i * 8 + 2 * tig);
        S[i][0] *= f.x; S[i][1] *= f.y;
        S[i][2] *= f.x; S[i][3] *= f.y;
      }
#pragma unroll
      for (int ks = 0; ks < MT; ++ks) {
        uint32_t a[4];
        ldmatrix_x4_trans(a, sv + (ks * 16 + brow) * LV + vg * 16 + bcol);
#pragma unroll
        for (int i = 0; i < NS / 2; ++i) {
          uint32_t bh[4], bl[4];
          ldmatrix_x4_trans(bh, sk + (ks * 16 + trow) * LQ + d_own + i * 16 + col8);
          ldmatrix_x4_trans(bl, sk + (CL + ks * 16 + trow) * LQ + d_own + i * 16 + col8);
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            mma(S[2 * i + u], a, bh[2 * u], bh[2 * u + 1]);
            mma(S[2 * i + u], a, bl[2 * u], bl[2 * u + 1]);
          }
        }
      }
    }
    __syncthreads();                                    // everyone has read the state of before the chunk
    publish();
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

template <int DT, int CL, int W>
int launch_scan(const ChunkParams& p, int groups, cudaStream_t stream) {
  static PerDeviceOnce once_;
  bool& configured = once_.slot();
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(gla_chunk_scan_kernel<DT, CL, W>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  return (int)launch_pdl(gla_chunk_scan_kernel<DT, CL, W>, dim3((p.V + 16 * groups - 1) / (16 * groups), p.H, p.entries),
                         dim3(groups * W * 32), scan_smem<DT, CL>(16 * groups), stream, p);
}

template <int DT, int CL>
int launch(ChunkParams p, int chunks, cudaStream_t stream) {
  static PerDeviceOnce once_;
  bool& configured = once_.slot();
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(gla_chunk_prep_kernel<DT, CL>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const size_t prep = (size_t)CL * (DT + 4) * 4 + (size_t)2 * CL * (DT + 8) * 2;
  const cudaError_t e = launch_pdl(gla_chunk_prep_kernel<DT, CL>, dim3(chunks, p.H), dim3(PT), prep, stream, p);
  if (e != cudaSuccess) return (int)e;
  // 16 columns per block where one wave of blocks takes them, more otherwise
  int groups = 1;
  while (groups < 4 && (long long)p.entries * p.H * ((p.V + 16 * groups - 1) / (16 * groups)) > 148 && 16 * groups < p.V &&
         scan_smem<DT, CL>(32 * groups) <= 227 * 1024)
    groups <<= 1;
  if constexpr (DT >= 128)
    if (groups <= 2) return launch_scan<DT, CL, 8>(p, groups, stream);
  return launch_scan<DT, CL, 4>(p, groups, stream);
}

}  // namespace

// Rows per chunk for D key channels; 0: not covered.
extern "C" int b200_gla_chunk_rows(int D) { return D <= 0 || D % 16 || D > 256 ? 0 : D <= 128 ? 64 : 32; }

// bf16 elements of workspace per chunk and head, and fp32 ones.
extern "C" int b200_gla_chunk_ws(int D) {
  return D <= 64 ? ws_elems<64, 64>() : D <= 128 ? ws_elems<128, 64>() : ws_elems<256, 32>();
}
extern "C" int b200_gla_chunk_end(int D) { return D <= 64 ? 64 : D <= 128 ? 128 : 256; }

// Entries with at least min_len rows; chunks: upper bound on their number (rows / chunk rows + entries).  D, V multiples of 16,
// D <= 256; state [slots, H, D, V] fp32 in place; o fp32 [rows, H * V].
extern "C" int b200_gla_chunk(const void* q, const void* k, const void* v, int ld, const float* la, float* state, float* o,
                              const int* first, const int* length, const int* slot, const int* positions, int entries, int min_len,
                              int chunks, void* ws, float* end, int H, int D, int V, float scale, cudaStream_t stream) {
  if (!b200_gla_chunk_rows(D) || V <= 0 || (V & 15) || (ld & 7) || entries <= 0 || entries > 65535 || H <= 0 || H > 65535 || chunks <= 0)
    return -6;
  ChunkParams p;
  p.q = reinterpret_cast<const __nv_bfloat16*>(q); p.k = reinterpret_cast<const __nv_bfloat16*>(k);
  p.v = reinterpret_cast<const __nv_bfloat16*>(v); p.la = la; p.state = state; p.o = o; p.first = first; p.length = length; p.slot = slot;
  p.positions = positions; p.ws = reinterpret_cast<__nv_bfloat16*>(ws); p.end = end; p.ld = ld; p.H = H; p.D = D; p.V = V;
  p.entries = entries; p.min_len = min_len; p.scale = scale;
  if (D <= 64) return launch<64, 64>(p, chunks, stream);
  if (D <= 128) return launch<128, 64>(p, chunks, stream);
  return launch<256, 32>(p, chunks, stream);
}
