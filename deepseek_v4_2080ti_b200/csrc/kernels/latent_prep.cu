// Prologues of latent attention: queries and keys / values go through low-rank latents, the cache holds one row per token,
// [latent | rotated key part], shared by all heads.  Rotation pairs element i with element i + dims / 2; elements past
// `dims` pass unchanged.  Widths are padded to multiples of 16 with zero columns.
//
//   latent_prep    one projection row [query latent | key/value latent | key part] -> normalised query latent; normalised
//                  latent and rotated key part to the token's cache row (a layer that reads another layer's cache: the query
//                  part only)
//   rotate_heads   the rotated part of every head of a query row, in place or into another layout
//   latent_gather  cache pages of several sequences -> contiguous latents and key parts, zero rows behind each sequence
#include "launch.h"
#include "ops.h"
#include "rotary.cuh"
#include "vec8.cuh"

namespace {
using namespace b200;

template <typename T>
struct LatentPrepParams {
  const T* proj;             // [rows, ld]
  T* q_out;                  // [rows, q_pad]
  T* cache;                  // [pages * block, c_pad + r_pad], or null: no keys of its own
  const float *q_w, *c_w;    // [q_pad], [c_pad]
  const double* freq;        // [dims / 2]
  const int *positions, *slots;
  int ld, q_rank, q_pad, c_rank, c_pad, r_dim, r_pad, dims;
  float eps, mscale;
};

template <typename T>
__global__ void latent_prep_kernel(LatentPrepParams<T> p) {
  __shared__ float red[32];
  pdl_grid_trigger();
  pdl_grid_wait();
  const size_t t = blockIdx.x;
  const T* row = p.proj + t * p.ld;
  auto norm = [&](const T* src, int n, int pad, const float* w, T* dst) {
    float ss = 0.f;
    for (int v = threadIdx.x; v < pad / 8; v += blockDim.x) {
      float f[8];
      load8(src + v * 8, f);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += v * 8 + j < n ? f[j] * f[j] : 0.f;
    }
    const float inv = 1.f / sqrtf(block_sum_all(ss, red) / (float)n + p.eps);
    for (int v = threadIdx.x; v < pad / 8; v += blockDim.x) {
      float f[8], g[8];
      load8(src + v * 8, f);
      load8(w + v * 8, g);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] = v * 8 + j < n ? f[j] * inv * g[j] : 0.f;
      store8(dst + v * 8, f);
    }
  };
  norm(row, p.q_rank, p.q_pad, p.q_w, p.q_out + t * p.q_pad);
  if (!p.cache) return;
  T* dst = p.cache + (size_t)p.slots[t] * (p.c_pad + p.r_pad);
  norm(row + p.q_pad, p.c_rank, p.c_pad, p.c_w, dst);
  const T* key = row + p.q_pad + p.c_pad;
  dst += p.c_pad;
  const int half = p.dims / 2, pos = p.positions[t];
  for (int i = threadIdx.x; i < p.r_pad; i += blockDim.x) {
    if (i < half) {
      float c, s;
      rotary_angle(pos, p.freq[i], p.mscale, c, s);
      const float u = (float)key[i], v = (float)key[i + half];
      dst[i] = (T)(u * c - v * s);
      dst[i + half] = (T)(v * c + u * s);
    } else if (i >= 2 * half) {
      dst[i] = i < p.r_dim ? key[i] : (T)0.f;
    }
  }
}

// src rows (src_ld apart) of H heads of src_head values with the rotated part at src_off of each -> dst likewise (may be the
// same).
template <typename T>
__global__ void rotate_heads_kernel(const T* src, T* dst, const double* __restrict__ freq, const int* __restrict__ positions, int H,
                                    int src_ld, int src_head, int src_off, int dst_ld, int dst_head, int dst_off, int r_pad, int dims,
                                    float mscale) {
  extern __shared__ float cs[];            // [dims / 2] cosine, [dims / 2] sine
  pdl_grid_trigger();
  const int half = dims / 2;
  pdl_grid_wait();
  const size_t t = blockIdx.x;
  const int pos = positions[t];
  for (int i = threadIdx.x; i < half; i += blockDim.x) rotary_angle(pos, freq[i], mscale, cs[i], cs[half + i]);
  __syncthreads();
  const int rest = r_pad - 2 * half, per = half + rest;
  for (int i = threadIdx.x; i < H * per; i += blockDim.x) {
    const int h = i / per, j = i - h * per;
    const T* s = src + t * src_ld + h * src_head + src_off;
    T* d = dst + t * dst_ld + h * dst_head + dst_off;
    if (j < half) {
      const float u = (float)s[j], v = (float)s[j + half];
      d[j] = (T)(u * cs[j] - v * cs[half + j]);
      d[j + half] = (T)(v * cs[j] + u * cs[half + j]);
    } else {
      d[half + j] = s[half + j];
    }
  }
}

// grid (rows): row r of the output belongs to entry e with start[e] <= r < start[e + 1].
__global__ void latent_gather_kernel(const __nv_bfloat16* __restrict__ cache, const int* __restrict__ block_table,
                                     const int* __restrict__ seq, const int* __restrict__ kv_len, const int* __restrict__ start,
                                     int entries, int max_blocks, int bs, int c_pad, int r_pad, int key_ld,
                                     __nv_bfloat16* __restrict__ latent, __nv_bfloat16* __restrict__ key) {
  pdl_grid_trigger();
  pdl_grid_wait();
  const int r = blockIdx.x;
  int e = 0;
  while (e + 1 < entries && start[e + 1] <= r) ++e;
  const int pos = r - start[e];
  const bool real = pos < kv_len[e];
  const __nv_bfloat16* src = nullptr;
  if (real) src = cache + ((size_t)block_table[(size_t)seq[e] * max_blocks + pos / bs] * bs + pos % bs) * (c_pad + r_pad);
  const uint4 zero = make_uint4(0, 0, 0, 0);
  const int nc = c_pad / 8, nr = r_pad / 8, nk = key_ld / 8;
  for (int v = threadIdx.x; v < nc + nk; v += blockDim.x) {
    const uint4 u = real && v < nc + nr ? *reinterpret_cast<const uint4*>(src + v * 8) : zero;
    if (v < nc) *reinterpret_cast<uint4*>(latent + (size_t)r * c_pad + v * 8) = u;
    else *reinterpret_cast<uint4*>(key + (size_t)r * key_ld + (v - nc) * 8) = u;
  }
}

template <typename T>
int run_prep(const void* proj, int ld, void* q_out, int q_rank, int q_pad, const float* q_w, void* cache, int c_rank, int c_pad,
             const float* c_w, int r_dim, int r_pad, int dims, const double* freq, float mscale, float eps, const int* positions,
             const int* slots, int rows, cudaStream_t stream) {
  LatentPrepParams<T> p;
  p.proj = reinterpret_cast<const T*>(proj); p.q_out = reinterpret_cast<T*>(q_out); p.cache = reinterpret_cast<T*>(cache);
  p.q_w = q_w; p.c_w = c_w; p.freq = freq; p.positions = positions; p.slots = slots; p.ld = ld; p.q_rank = q_rank; p.q_pad = q_pad;
  p.c_rank = c_rank; p.c_pad = c_pad; p.r_dim = r_dim; p.r_pad = r_pad; p.dims = dims; p.eps = eps; p.mscale = mscale;
  return (int)launch_pdl(latent_prep_kernel<T>, dim3(rows), dim3(128), 0, stream, p);
}

template <typename T>
int run_rotate(const void* src, void* dst, const double* freq, const int* positions, int rows, int H, int src_ld, int src_head,
               int src_off, int dst_ld, int dst_head, int dst_off, int r_pad, int dims, float mscale, cudaStream_t stream) {
  return (int)launch_pdl(rotate_heads_kernel<T>, dim3(rows), dim3(128), (size_t)dims * sizeof(float) + 16, stream,
                         reinterpret_cast<const T*>(src), reinterpret_cast<T*>(dst), freq, positions, H, src_ld, src_head, src_off,
                         dst_ld, dst_head, dst_off, r_pad, dims, mscale);
}

}  // namespace

// proj rows [q_pad | c_pad | r_pad] (without keys of its own: [q_pad]); pads are multiples of 8.
extern "C" int b200_latent_prep(const void* proj, int ld, void* q_out, int q_rank, int q_pad, const float* q_w, void* cache, int c_rank,
                                int c_pad, const float* c_w, int r_dim, int r_pad, int dims, const double* freq, float mscale,
                                float eps, const int* positions, const int* slots, int rows, int f32, cudaStream_t stream) {
  if (rows <= 0 || (ld & 7) || (q_pad & 7) || (c_pad & 7) || (r_pad & 7) || q_rank <= 0 || q_rank > q_pad || dims & 1) return -6;
  if (cache && (c_rank <= 0 || c_rank > c_pad || r_dim > r_pad || dims > r_dim || ld < q_pad + c_pad + r_pad)) return -6;
  return f32 ? run_prep<float>(proj, ld, q_out, q_rank, q_pad, q_w, cache, c_rank, c_pad, c_w, r_dim, r_pad, dims, freq, mscale, eps,
                               positions, slots, rows, stream)
             : run_prep<__nv_bfloat16>(proj, ld, q_out, q_rank, q_pad, q_w, cache, c_rank, c_pad, c_w, r_dim, r_pad, dims, freq,
                                       mscale, eps, positions, slots, rows, stream);
}

extern "C" int b200_rotate_heads(const void* src, void* dst, const double* freq, const int* positions, int rows, int H, int src_ld,
                                 int src_head, int src_off, int dst_ld, int dst_head, int dst_off, int r_pad, int dims, float mscale, int f32,
                                 cudaStream_t stream) {
  if (rows <= 0 || H <= 0 || dims < 0 || dims & 1 || dims > r_pad || src_off + r_pad > src_head || dst_off + r_pad > dst_head ||
      src_ld < H * src_head || dst_ld < H * dst_head)
    return -6;
  return f32 ? run_rotate<float>(src, dst, freq, positions, rows, H, src_ld, src_head, src_off, dst_ld, dst_head, dst_off, r_pad, dims,
                                 mscale, stream)
             : run_rotate<__nv_bfloat16>(src, dst, freq, positions, rows, H, src_ld, src_head, src_off, dst_ld, dst_head, dst_off,
                                         r_pad, dims, mscale, stream);
}

// latent [rows, c_pad], key [rows, key_ld] (key_ld >= r_pad, zero columns behind); start: first output row of every entry.
extern "C" int b200_latent_gather(const void* cache, const int* block_table, const int* seq, const int* kv_len, const int* start,
                                  int entries, int max_blocks, int bs, int c_pad, int r_pad, int key_ld, void* latent, void* key,
                                  int rows, cudaStream_t stream) {
  if (rows <= 0 || entries <= 0 || (c_pad & 7) || (r_pad & 7) || (key_ld & 7) || key_ld < r_pad) return -6;
  return (int)launch_pdl(latent_gather_kernel, dim3(rows), dim3(96), 0, stream, reinterpret_cast<const __nv_bfloat16*>(cache),
                         block_table, seq, kv_len, start, entries, max_blocks, bs, c_pad, r_pad, key_ld,
                         reinterpret_cast<__nv_bfloat16*>(latent), reinterpret_cast<__nv_bfloat16*>(key));
}
