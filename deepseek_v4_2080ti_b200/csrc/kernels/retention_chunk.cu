// Retention (see decay_rule.cu) over prompt portions in chunks of CL rows, bf16 values.  With b_t the sum of the log decays of a
// chunk up to row t and S the state before the chunk:
//
//   o_t = (q_t e^{b_t}) S + sum_{s <= t} A_ts v_s,   A_ts = e^{b_t - b_s} q_t . k_s
//   S'  = e^{b_end} S + sum_s (k_s e^{b_end - b_s}) v_s^T
//
// Every exponent is a difference taken towards the later row, so no factor grows.
//
//   retention_prep   one block per chunk and head: decayed q and k, A -> workspace
//   retention_scan   four or eight warps per 16 value columns walk the chunks.  Each keeps its share of the channels of S^T
//                    in registers and updates it; for q S, of which each takes 16 rows and 8 columns (or 16), the shares are
//                    exchanged through shared memory once per chunk
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

constexpr float FLOOR = -126.f;          // log2 of a decay that leaves nothing

struct ChunkParams {
  const float *q, *k;              // [rows, H, D] rotated
  const __nv_bfloat16* v;          // head h of row t at v + t * ldv + h * V
  const float* log2_decay;         // [H]
  float* state;                    // [slots, H, D, V]
  float* o;                        // [rows, H * V]
  const int *first, *length, *slot, *positions;
  __nv_bfloat16* ws;               // per chunk and head: q hi | q lo | k hi | k lo [CL, DT], A hi | A lo [CL, CL]
  float* end;                      // per chunk and head: e^{b_end}
  int ldv, H, D, V, entries, min_len;
};

__device__ __forceinline__ int chunks_of(const ChunkParams& p, int e, int CL) {
  const int n = p.length[e];
  return n < p.min_len ? 0 : (n + CL - 1) / CL;
}

template <int DT, int CL>
__host__ __device__ constexpr size_t ws_elems() { return (size_t)4 * CL * DT + 2 * CL * CL; }

constexpr int PT = 256;

template <int DT, int CL>
constexpr size_t prep_smem() { return (size_t)4 * CL * (DT + 8) * 2 + CL * 4; }

// grid (chunks, H).
template <int DT, int CL>
__global__ void __launch_bounds__(PT) retention_prep_kernel(ChunkParams p) {
  constexpr int LQ = DT + 8, MT = CL / 16;
  extern __shared__ __align__(16) uint8_t smem[];
  __nv_bfloat16* sk = reinterpret_cast<__nv_bfloat16*>(smem);                  // [hi, lo][CL][LQ]
  __nv_bfloat16* sq = sk + 2 * CL * LQ;
  float* sb = reinterpret_cast<float*>(sq + 2 * CL * LQ);                      // [CL] summed log2 decays
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
  __nv_bfloat16 *ws_q = p.ws + at * ws_elems<DT, CL>(), *ws_k = ws_q + (size_t)2 * CL * DT;
  __nv_bfloat16 *a_hi = ws_k + (size_t)2 * CL * DT, *a_lo = a_hi + CL * CL;
  if (tid < CL) sb[tid] = (float)min(tid + 1, n) * fmaxf(p.log2_decay[h], FLOOR);
  __syncthreads();
  const float b_end = sb[CL - 1];
  if (tid == 0) p.end[at] = pow2(b_end);
  for (int i = tid; i < CL * (DT / 8); i += PT) {
    const int t = i / (DT / 8), d = i % (DT / 8) * 8;
    const bool ok = t < n && d < p.D;                               // D is a multiple of 16
    const size_t src = ((size_t)(t0 + t) * p.H + h) * p.D + d;
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
  const int row16 = lane & 15, col8 = (lane >> 4) * 8;
  // q k^T: rows [16 mt, 16 mt + 16), every second tile of 8 columns up to the diagonal
  const int mt = warp & 3, nh = warp >> 2;
  if (mt < MT) {
    constexpr int NT = MT;                                // tiles of a warp at most
    float aq[NT][4];
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int x = 0; x < 4; ++x) aq[j][x] = 0.f;
#pragma unroll 2
    for (int ks = 0; ks < DT / 16; ++ks) {
      uint32_t qh[4], ql[4];
      const int off = (mt * 16 + row16) * LQ + ks * 16 + col8;
      ldmatrix_x4(qh, sq + off);
      ldmatrix_x4(ql, sq + CL * LQ + off);
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        if (j > mt) break;
        const __nv_bfloat16* b = sk + ((2 * j + nh) * 8 + g) * LQ + ks * 16 + 2 * tig;
        const uint32_t h0 = *reinterpret_cast<const uint32_t*>(b), h1 = *reinterpret_cast<const uint32_t*>(b + 8);
        const uint32_t l0 = *reinterpret_cast<const uint32_t*>(b + CL * LQ), l1 = *reinterpret_cast<const uint32_t*>(b + CL * LQ + 8);
        mma(aq[j], qh, h0, h1);
        mma(aq[j], qh, l0, l1);
        mma(aq[j], ql, h0, h1);
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
        for (int u = 0; u < 2; ++u) a[u] = s + u <= r ? aq[j][2 * w + u] * pow2(sb[r] - sb[s + u]) : 0.f;
        uint32_t hi, lo;
        split2(a[0], a[1], hi, lo);
        *reinterpret_cast<uint32_t*>(a_hi + r * CL + s) = hi;
        *reinterpret_cast<uint32_t*>(a_lo + r * CL + s) = lo;
      }
    }
  }
}

// Shared memory of a chunk: query and key rows, A, values.
template <int DT, int CL>
__host__ __device__ constexpr size_t stage_elems(int VB) { return (size_t)4 * CL * (DT + 8) + 2 * CL * (CL + 8) + CL * (VB + 8); }
template <int DT, int CL>
constexpr size_t scan_smem(int VB) { return (2 * stage_elems<DT, CL>(VB) + (size_t)(VB / 16) * 2 * 16 * (DT + 8)) * 2; }

// grid (ceil(V / VB), H, entries), W VB / 16 warps: W of them (4 or 8) own value columns 16 i .. 16 i + 15.
template <int DT, int CL, int W>
__global__ void __launch_bounds__(512) retention_scan_kernel(ChunkParams p) {
  constexpr int LQ = DT + 8, LA = CL + 8, MT = CL / 16, ND = DT / W, NS = ND / 8, NJ = W == 8 ? 1 : 2;
  // channels, fragments of S^T and 8-column tiles of the output of a warp
  extern __shared__ __align__(16) uint8_t smem[];
  const int tid = threadIdx.x, nthr = blockDim.x, lane = tid & 31, g = lane >> 2, tig = lane & 3;
  const int vg = tid / (32 * W), sub = (tid >> 5) % W;
  const int VB = nthr / (2 * W), LV = VB + 8, h = blockIdx.y, e = blockIdx.z, v0 = blockIdx.x * VB;
  __nv_bfloat16* stages = reinterpret_cast<__nv_bfloat16*>(smem);
  __nv_bfloat16* ss = stages + 2 * stage_elems<DT, CL>(VB) + (size_t)vg * 2 * 16 * LQ;                      // [hi, lo][16][LQ]
  pdl_grid_trigger();
  pdl_grid_wait();
  const int chunks = chunks_of(p, e, CL);
  if (chunks == 0) return;
  int base = 0;
  for (int i = 0; i < e; ++i) base += chunks_of(p, i, CL);
  const int r0 = p.first[e], len = p.length[e];
  auto fetch = [&](int c) {
    const __nv_bfloat16* ws = p.ws + ((size_t)(base + c) * p.H + h) * ws_elems<DT, CL>();
    __nv_bfloat16* dst = stages + (c & 1) * stage_elems<DT, CL>(VB);
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
      cp16(dst + r * LV + x, p.v + (ok ? (size_t)(r0 + c * CL + r) * p.ldv + (size_t)h * p.V + v0 + x : 0), ok);
    }
    cp_commit();
  };
  fetch(0);
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
  float end_next = p.end[(size_t)base * p.H + h];
  const int row16 = lane & 15, col8 = (lane >> 4) * 8;                       // non-transposed 16 x 16 tiles, left operand
  const int brow = (lane & 7) + (lane >> 4) * 8, bcol = ((lane >> 3) & 1) * 8;   // left operand, transposed
  const int trow = (lane & 7) + ((lane >> 3) & 1) * 8;                       // right operand, transposed
  for (int c = 0; c < chunks; ++c) {
    cp_wait<0>();
    __syncthreads();                                    // rows and state landed; the buffers' last readers are done
    const float end = end_next;
    if (c + 1 < chunks) {
      fetch(c + 1);
      end_next = p.end[(size_t)(base + c + 1) * p.H + h];
    }
    const __nv_bfloat16* sq = stages + (c & 1) * stage_elems<DT, CL>(VB);
    const __nv_bfloat16* sk = sq + 2 * CL * LQ;
    const __nv_bfloat16* sa = sk + 2 * CL * LQ;
    const __nv_bfloat16* sv = sa + 2 * CL * LA + vg * 16;
    float o[NJ][4] = {}, ol[NJ][4] = {};                // sums of the leading and of the correcting products
    if (reads) {
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
    }
    __syncthreads();                                    // everyone has read the state of before the chunk
    if (live) {
#pragma unroll
      for (int i = 0; i < NS; ++i)
#pragma unroll
        for (int x = 0; x < 4; ++x) S[i][x] *= end;
#pragma unroll
      for (int ks = 0; ks < MT; ++ks) {
        uint32_t a[4];
        ldmatrix_x4_trans(a, sv + (ks * 16 + brow) * LV + bcol);
#pragma unroll
        for (int i = 0; i < NS / 2; ++i) {
          uint32_t bh[4], bl[4];
          const int off = (ks * 16 + trow) * LQ + d_own + i * 16 + col8;
          ldmatrix_x4_trans(bh, sk + off);
          ldmatrix_x4_trans(bl, sk + CL * LQ + off);
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            mma(S[2 * i + x], a, bh[2 * x], bh[2 * x + 1]);
            mma(S[2 * i + x], a, bl[2 * x], bl[2 * x + 1]);
          }
        }
      }
      publish();                                        // the next chunk starts from it: the outputs come after
    }
    if (reads) {
#pragma unroll
      for (int ks = 0; ks < MT; ++ks) {
        if (ks > m) break;
        uint32_t b[4], ah[4], al[4];
        ldmatrix_x4_trans(b, sv + (ks * 16 + trow) * LV + col8);
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
    const cudaError_t e = cudaFuncSetAttribute(retention_scan_kernel<DT, CL, W>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  return (int)launch_pdl(retention_scan_kernel<DT, CL, W>, dim3((p.V + 16 * groups - 1) / (16 * groups), p.H, p.entries),
                         dim3(groups * W * 32), scan_smem<DT, CL>(16 * groups), stream, p);
}

template <int DT, int CL>
int launch(const ChunkParams& p, int chunks, cudaStream_t stream) {
  static PerDeviceOnce once_;
  bool& configured = once_.slot();
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(retention_prep_kernel<DT, CL>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const cudaError_t e = launch_pdl(retention_prep_kernel<DT, CL>, dim3(chunks, p.H), dim3(PT), prep_smem<DT, CL>(), stream, p);
  if (e != cudaSuccess) return (int)e;
  // 16 columns per block where one wave of blocks takes them, more otherwise
  constexpr int W = DT >= 128 ? 8 : 4;
  int groups = 1;
  while (groups * 2 * W * 32 <= 512 && (long long)p.entries * p.H * ((p.V + 16 * groups - 1) / (16 * groups)) > 148 && 16 * groups < p.V &&
         scan_smem<DT, CL>(32 * groups) <= 227 * 1024)
    groups <<= 1;
  return launch_scan<DT, CL, W>(p, groups, stream);
}

}  // namespace

// Rows per chunk for D key channels; 0: not covered.
extern "C" int b200_retention_chunk_rows(int D) { return D <= 0 || D % 16 || D > 256 ? 0 : D <= 128 ? 64 : 32; }

// bf16 elements of workspace per chunk and head.
extern "C" int b200_retention_chunk_ws(int D) { return D <= 64 ? ws_elems<64, 64>() : D <= 128 ? ws_elems<128, 64>() : ws_elems<256, 32>(); }

// Entries with at least min_len rows; chunks: upper bound on their number (rows / chunk rows + entries).  q, k fp32 [rows, H, D]
// (b200_rotate_prep), v bf16 rows `ldv` apart, log2_decay fp32 [H].  D, V multiples of 16, D <= 256; end fp32 [chunks * H]; state
// [slots, H, D, V] fp32 in place; o fp32 [rows, H * V].
extern "C" int b200_retention_chunk(const float* q, const float* k, const void* v, int ldv, const float* log2_decay, float* state, float* o,
                                    const int* first, const int* length, const int* slot, const int* positions, int entries, int min_len,
                                    int chunks, void* ws, float* end, int H, int D, int V, cudaStream_t stream) {
  if (!b200_retention_chunk_rows(D) || V <= 0 || (V & 15) || (ldv & 7) || entries <= 0 || entries > 65535 || H <= 0 || H > 65535 ||
      chunks <= 0 || !log2_decay)
    return -6;
  ChunkParams p;
  p.q = q; p.k = k; p.v = reinterpret_cast<const __nv_bfloat16*>(v); p.log2_decay = log2_decay; p.state = state; p.o = o; p.first = first;
  p.length = length; p.slot = slot; p.positions = positions; p.ws = reinterpret_cast<__nv_bfloat16*>(ws); p.end = end; p.ldv = ldv; p.H = H;
  p.D = D; p.V = V; p.entries = entries; p.min_len = min_len;
  if (D <= 64) return launch<64, 64>(p, chunks, stream);
  if (D <= 128) return launch<128, 64>(p, chunks, stream);
  return launch<256, 32>(p, chunks, stream);
}
