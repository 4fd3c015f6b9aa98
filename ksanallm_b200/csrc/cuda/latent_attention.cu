// Latent attention over pages of 16 tokens: the cache holds one RMS-normed latent and one rotated key part per token,
// [block][16 x (rank + rot)].
#include "host_common.h"
#include "mixer_common.cuh"

namespace ksana {

// ---- what happens between the projections and the scores -------------------------------------------------------------
// One warp per (token, head): the last rot dimensions of a query head are rotated in place (pairs (2i, 2i + 1)), and
// also written behind the head's absorbed query in q_cat for tokens from cat_from on. One further warp per token: the
// latent's RMS norm and the rotated key part go to the cache.
template <typename T>
__global__ void __launch_bounds__(256)
latent_append_kernel(T* __restrict__ q, int ldq, int dim, T* __restrict__ q_cat, int cat_from, const T* __restrict__ x,
                     int ldx, const float* __restrict__ norm_w, float eps, const int* __restrict__ positions,
                     const float* __restrict__ rotary, const int* __restrict__ slots, T* __restrict__ cache, int tokens,
                     int h, int rank, int rd) {
  const int units = h + 1;
  const long long unit = static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (unit >= static_cast<long long>(tokens) * units) return;
  const int t = static_cast<int>(unit / units), hd = static_cast<int>(unit % units);
  const float* cs = rotary + static_cast<size_t>(positions[t]) * rd;
  const int half = rd / 2;
  if (hd < h) {
    T* src = q + static_cast<size_t>(t) * ldq + static_cast<size_t>(hd) * (dim + rd) + dim;
    T* cat = q_cat && t >= cat_from ? q_cat + (static_cast<size_t>(t - cat_from) * h + hd) * (rank + rd) + rank : nullptr;
    for (int i = lane; i < half; i += 32) {
      const float a = to_f(src[2 * i]), b = to_f(src[2 * i + 1]), c = cs[i], s = cs[half + i];
      const T u = from_f<T>(a * c - b * s), v = from_f<T>(b * c + a * s);
      src[2 * i] = u;
      src[2 * i + 1] = v;
      if (cat) {
        cat[2 * i] = u;
        cat[2 * i + 1] = v;
      }
    }
    return;
  }
  if (slots[t] < 0) return;
  const T* a = x + static_cast<size_t>(t) * ldx;
  T* dst = cache + static_cast<size_t>(slots[t]) * (rank + rd);
  float ss = 0.f;
  for (int i = lane; i < rank; i += 32) {
    const float f = to_f(a[i]);
    ss += f * f;
  }
  const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(rank) + eps);
  for (int i = lane; i < rank; i += 32) dst[i] = from_f<T>(to_f(a[i]) * inv * norm_w[i]);
  for (int i = lane; i < half; i += 32) {
    const float u = to_f(a[rank + 2 * i]), v = to_f(a[rank + 2 * i + 1]), c = cs[i], s = cs[half + i];
    dst[rank + 2 * i] = from_f<T>(u * c - v * s);
    dst[rank + 2 * i + 1] = from_f<T>(v * c + u * s);
  }
}

// The contexts of sequences [seq_base, seq_base + gridDim.y), row by row behind one another: [rows][rank + rot]. One warp
// per row, 16 bytes per lane.
__global__ void __launch_bounds__(256)
latent_gather_kernel(const uint4* __restrict__ cache, const int* __restrict__ block_tables, int max_blocks,
                     const int* __restrict__ kv_lens, int seq_base, int bs, int words, uint4* __restrict__ out) {
  const int b = seq_base + blockIdx.y, L = kv_lens[b];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int j0 = blockIdx.x * 32;
  if (j0 >= L) return;
  int row0 = 0;
  for (int i = seq_base + lane; i < b; i += 32) row0 += kv_lens[i];
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) row0 += __shfl_xor_sync(0xffffffffu, row0, o);
  for (int j = j0 + warp; j < min(j0 + 32, L); j += 8) {
    const uint4* src = cache + (static_cast<size_t>(block_tables[static_cast<size_t>(b) * max_blocks + j / bs]) * bs + j % bs) * words;
    uint4* dst = out + static_cast<size_t>(row0 + j) * words;
    for (int i = lane; i < words; i += 32) dst[i] = src[i];
  }
}

}  // namespace ksana

using namespace ksana;

// bf16. -1: rows are not multiples of 16 bytes.
KSANA_API int ksana_latent_gather(const void* cache, const int* block_tables, int max_blocks, const int* kv_lens,
                                  int seq_base, int num_seqs, int max_kv, int bs, int width, void* out, cudaStream_t st) {
  if (num_seqs <= 0 || max_kv <= 0) return 0;
  if (width & 7) return -1;
  latent_gather_kernel<<<dim3((max_kv + 31) / 32, num_seqs), 256, 0, st>>>(
      static_cast<const uint4*>(cache), block_tables, max_blocks, kv_lens, seq_base, bs, width / 8,
      static_cast<uint4*>(out));
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

// q: [tokens, h * (dim + rot)] (pitch ldq); q_cat: [tokens - cat_from, h, rank + rot] or null; x: [tokens, rank + rot]
// (pitch ldx). A slot is a row of the cache. kind: 0 fp32, 1 bf16.
KSANA_API int ksana_latent_append(void* q, int ldq, int dim, void* q_cat, int cat_from, const void* x, int ldx,
                                  const float* norm_w, float eps, const int* positions, const float* rotary,
                                  const int* slots, void* cache, int tokens, int h, int rank, int rot, int kind,
                                  cudaStream_t st) {
  if (tokens <= 0) return 0;
  if (rot < 0 || (rot & 1) || rank < 1) return -2;
  const unsigned grid = static_cast<unsigned>((static_cast<long long>(tokens) * (h + 1) + 7) / 8);
#define KSANA_LA(T)                                                                                                 \
  latent_append_kernel<T><<<grid, 256, 0, st>>>(static_cast<T*>(q), ldq, dim, static_cast<T*>(q_cat), cat_from,     \
                                                static_cast<const T*>(x), ldx, norm_w, eps, positions, rotary,      \
                                                slots, static_cast<T*>(cache), tokens, h, rank, rot)
  if (kind) KSANA_LA(__nv_bfloat16); else KSANA_LA(float);
#undef KSANA_LA
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}
