// Routing by the largest logits, the sort of (token, slot) pairs by expert in one launch, and expert GEMMs for sizes and
// number formats the tensor-core pipeline in moe.cu does not take. Compiled with accurate math: routing is specified in
// 32-bit floats.
#include "host_common.h"
#include "mixer_common.cuh"

namespace ksana {

// ---- router: top-k of logits (+ bias), softmax over the chosen ones or (sigmoid) each one's sigmoid, times scale ------------------------------------------------
// One warp per token; the token's logits sit in shared memory. Ties go to the lower index. Of `groups` equal groups of
// neighbours only the `keep` with the largest logits take part.
__device__ __forceinline__ void warp_argmax(float& v, int& i) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, v, o);
    const int oi = __shfl_xor_sync(0xffffffffu, i, o);
    if (ov > v || (ov == v && oi < i)) {
      v = ov;
      i = oi;
    }
  }
}
__global__ void __launch_bounds__(128)
moe_topk_kernel(const float* __restrict__ logits, int ld, const float* __restrict__ bias, int T, int E, int k,
                int groups, int keep, int sigmoid, float scale, int* __restrict__ ids, float* __restrict__ weights) {
  extern __shared__ float sm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * 4 + warp;
  if (t >= T) return;
  const int G = keep < groups ? groups : 0, size = E / groups;
  float* z = sm + warp * (E + 2 * G);
  for (int e = lane; e < E; e += 32) z[e] = logits[static_cast<size_t>(t) * ld + e] + (bias ? bias[e] : 0.f);
  __syncwarp();
  if (G > 0) {
    float *best = z + E, *open = best + G;
    for (int g = lane; g < G; g += 32) {
      float v = -INFINITY;
      for (int e = g * size; e < (g + 1) * size; ++e) v = fmaxf(v, z[e]);
      best[g] = v;
      open[g] = 0.f;
    }
    __syncwarp();
    for (int r = 0; r < keep; ++r) {
      float v = -INFINITY;
      int vi = G;
      for (int g = lane; g < G; g += 32)
        if (open[g] == 0.f && (best[g] > v || vi == G)) {
          v = best[g];
          vi = g;
        }
      warp_argmax(v, vi);
      if (lane == 0 && vi < G) open[vi] = 1.f;
      __syncwarp();
    }
    for (int e = lane; e < E; e += 32)
      if (open[e / size] == 0.f) z[e] = -INFINITY;
    __syncwarp();
  }
  int* my_ids = ids + static_cast<size_t>(t) * k;
  float* my_w = weights + static_cast<size_t>(t) * k;
  float top = 0.f, sum = 0.f;
  for (int r = 0; r < k; ++r) {
    float v = -INFINITY;
    int vi = E;
    for (int e = lane; e < E; e += 32)
      if (z[e] > v) {
        v = z[e];
        vi = e;
      }
    warp_argmax(v, vi);
    if (vi >= E) vi = 0;  // (no finite logit is left)
    if (r == 0) top = v;
    const float p = v == -INFINITY ? 0.f : sigmoid ? sigmoid_f(v) : expf(v - top);
    sum += p;
    if (lane == 0) {
      my_ids[r] = vi;
      my_w[r] = p;
      z[vi] = -INFINITY;
    }
    __syncwarp();
  }
  for (int r = lane; r < k; r += 32) my_w[r] = sigmoid ? my_w[r] * scale : sum > 0.f ? my_w[r] / sum * scale : 0.f;
}

// ---- counting sort by expert in one CTA ----------------------------------------------------------------------------
// offsets[0 .. E]: first sorted row of each expert; pos[i]: sorted row of pair i (-1: not a local expert); row_src: its
// inverse. Pairs of one warp that go to the same expert take their places together.
__global__ void __launch_bounds__(1024)
moe_sort_kernel(const int* __restrict__ ids, int n, int expert_offset, int E, int* __restrict__ offsets,
                int* __restrict__ pos, int* __restrict__ row_src) {
  extern __shared__ int cnt[];  // [E]
  const int tid = threadIdx.x, lane = tid & 31;
  const int n_up = (n + 31) & ~31;
  for (int e = tid; e < E; e += 1024) cnt[e] = 0;
  __syncthreads();
  auto expert = [&](int i) {
    const int e = i < n ? ids[i] - expert_offset : -1;
    return e >= 0 && e < E ? e : -1;
  };
  for (int i = tid; i < n_up; i += 1024) {
    const int e = expert(i);
    const unsigned peers = __match_any_sync(0xffffffffu, e);
    if (e >= 0 && lane == __ffs(peers) - 1) atomicAdd(&cnt[e], __popc(peers));
  }
  __syncthreads();
  if (tid < 32) {
    int base = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + lane;
      const int c = e < E ? cnt[e] : 0;
      int s = c;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int u = __shfl_up_sync(0xffffffffu, s, o);
        if (lane >= o) s += u;
      }
      if (e < E) offsets[e] = cnt[e] = base + s - c;
      base += __shfl_sync(0xffffffffu, s, 31);
    }
    if (lane == 0) offsets[E] = base;
  }
  __syncthreads();
  for (int i = tid; i < n_up; i += 1024) {
    const int e = expert(i);
    const unsigned peers = __match_any_sync(0xffffffffu, e);
    const int leader = __ffs(peers) - 1;
    int first = 0;
    if (e >= 0 && lane == leader) first = atomicAdd(&cnt[e], __popc(peers));
    first = __shfl_sync(0xffffffffu, first, leader);
    if (i < n) {
      const int p = e < 0 ? -1 : first + __popc(peers & ((1u << lane) - 1));
      pos[i] = p;
      if (p >= 0) row_src[p] = i;
    }
  }
}

// ---- expert GEMM of any size: C[rows of expert e] = A[rows of e] W[e]^T in 32-bit arithmetic --------------------------
// Sorted row p reads row row_src[p] / k of A (row_src null: row p). One CTA = 32 rows x 64 columns of one expert.
template <typename T>
__global__ void __launch_bounds__(128)
moe_gemm_any_kernel(const T* __restrict__ A, int lda, const int* __restrict__ row_src, int k, const T* __restrict__ W,
                    T* __restrict__ C, const int* __restrict__ offsets, int E, int N, int K) {
  __shared__ float sA[16][36], sB[16][68];
  int tile = blockIdx.x, e = 0;
  for (; e < E; ++e) {
    const int tiles = (offsets[e + 1] - offsets[e] + 31) / 32;
    if (tile < tiles) break;
    tile -= tiles;
  }
  if (e == E) return;
  const int row0 = offsets[e] + tile * 32, rows = min(32, offsets[e + 1] - row0), col0 = blockIdx.y * 64;
  const T* w = W + static_cast<size_t>(e) * N * K;
  const int tid = threadIdx.x, tr = tid >> 4, tc = tid & 15;
  float acc[4][4] = {};
  const int ar = tid >> 2, ak = (tid & 3) * 4;  // this thread's part of a tile of A: one row, 4 columns
  const T* arow = nullptr;
  if (ar < rows) arow = A + static_cast<size_t>(row_src ? row_src[row0 + ar] / k : row0 + ar) * lda;
  const int br = tid >> 1, bk = (tid & 1) * 8;  // of W: one output column, 8 columns
  const T* brow = col0 + br < N ? w + static_cast<size_t>(col0 + br) * K : nullptr;
  for (int k0 = 0; k0 < K; k0 += 16) {
#pragma unroll
    for (int j = 0; j < 4; ++j) sA[ak + j][ar] = arow && k0 + ak + j < K ? to_f(arow[k0 + ak + j]) : 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) sB[bk + j][br] = brow && k0 + bk + j < K ? to_f(brow[k0 + bk + j]) : 0.f;
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < 16; ++kk) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) a[i] = sA[kk][tr * 4 + i];
#pragma unroll
      for (int j = 0; j < 4; ++j) b[j] = sB[kk][tc + 16 * j];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int r = tr * 4 + i, c = col0 + tc + 16 * j;
      if (r < rows && c < N) C[static_cast<size_t>(row0 + r) * N + c] = from_f<T>(acc[i][j]);
    }
}

// out = silu(gate) * up over rows [gate | up]
template <typename T>
__global__ void silu_mul_any_kernel(const T* __restrict__ x, T* __restrict__ out, int I) {
  const size_t row = blockIdx.x;
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c < I) out[row * I + c] = from_f<T>(silu_f(to_f(x[row * 2 * I + c])) * to_f(x[row * 2 * I + I + c]));
}

static int launched() { return cudaGetLastError() == cudaSuccess ? 0 : -5; }

}  // namespace ksana

using namespace ksana;

// scoring: 0 softmax over the chosen logits, 1 each one's sigmoid.
KSANA_API int ksana_moe_topk(const float* logits, int ld, const float* bias, int T, int E, int k, int groups, int keep,
                             int scoring, float scale, int* ids, float* weights, cudaStream_t st) {
  if (T <= 0) return 0;
  if (groups < 1 || E % groups || keep < 1 || keep > groups || k > E / groups * keep) return -2;
  const int smem = 4 * (E + (keep < groups ? 2 * groups : 0)) * static_cast<int>(sizeof(float));
  if (k < 1 || E > 2048 || smem > 48 * 1024) return -1;
  moe_topk_kernel<<<(T + 3) / 4, 128, smem, st>>>(logits, ld, bias, T, E, k, groups, keep, scoring, scale,
                                                    ids, weights);
  return launched();
}

KSANA_API int ksana_moe_sort(const int* ids, int n, int expert_offset, int E, int* offsets, int* pos, int* row_src,
                             cudaStream_t st) {
  if (n <= 0) return 0;
  if (E < 1 || E > 8192) return -1;
  moe_sort_kernel<<<1, 1024, E * static_cast<int>(sizeof(int)), st>>>(ids, n, expert_offset, E, offsets, pos, row_src);
  return launched();
}

// n: rows of C at most. kind: 0 fp32, 1 bf16.
KSANA_API int ksana_moe_gemm_any(const void* A, int lda, const int* row_src, int k, const void* W, void* C,
                                 const int* offsets, int E, int n, int N, int K, int kind, cudaStream_t st) {
  if (n <= 0) return 0;
  const dim3 grid(n / 32 + (E < n ? E : n), (N + 63) / 64);
  if (kind)
    moe_gemm_any_kernel<<<grid, 128, 0, st>>>(static_cast<const __nv_bfloat16*>(A), lda, row_src, k,
                                              static_cast<const __nv_bfloat16*>(W), static_cast<__nv_bfloat16*>(C),
                                              offsets, E, N, K);
  else
    moe_gemm_any_kernel<<<grid, 128, 0, st>>>(static_cast<const float*>(A), lda, row_src, k,
                                              static_cast<const float*>(W), static_cast<float*>(C), offsets, E, N, K);
  return launched();
}

KSANA_API int ksana_silu_mul_any(const void* x, void* out, int rows, int I, int kind, cudaStream_t st) {
  if (rows <= 0 || I <= 0) return 0;
  const dim3 grid(rows, (I + 255) / 256);
  if (kind)
    silu_mul_any_kernel<<<grid, 256, 0, st>>>(static_cast<const __nv_bfloat16*>(x), static_cast<__nv_bfloat16*>(out),
                                              I);
  else
    silu_mul_any_kernel<<<grid, 256, 0, st>>>(static_cast<const float*>(x), static_cast<float*>(out), I);
  return launched();
}
