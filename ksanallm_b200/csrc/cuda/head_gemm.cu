// One small matrix product per head (or per block of a block-diagonal matrix), for sizes and number formats the batched
// tensor-core GEMM does not take: C[t, b, :] = A[t, b, :] W[b]^T in 32-bit arithmetic.
#include "host_common.h"
#include "mixer_common.cuh"

namespace ksana {

// One CTA = 32 rows x 64 columns of one head.
template <typename T, typename O>
__global__ void __launch_bounds__(128)
head_gemm_any_kernel(const T* __restrict__ A, long long a_row, long long a_head, const T* __restrict__ W,
                     O* __restrict__ C, long long c_row, long long c_head, int rows, int N, int K) {
  __shared__ float sA[16][36], sB[16][68];
  const int row0 = blockIdx.x * 32, col0 = blockIdx.y * 64, b = blockIdx.z;
  const T* w = W + static_cast<size_t>(b) * N * K;
  const int tid = threadIdx.x, tr = tid >> 4, tc = tid & 15;
  float acc[4][4] = {};
  const int ar = tid >> 2, ak = (tid & 3) * 4;
  const T* arow = row0 + ar < rows ? A + (row0 + ar) * a_row + b * a_head : nullptr;
  const int br = tid >> 1, bk = (tid & 1) * 8;
  const T* brow = col0 + br < N ? w + static_cast<size_t>(col0 + br) * K : nullptr;
  for (int k0 = 0; k0 < K; k0 += 16) {
#pragma unroll
    for (int j = 0; j < 4; ++j) sA[ak + j][ar] = arow && k0 + ak + j < K ? to_f(arow[k0 + ak + j]) : 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) sB[bk + j][br] = brow && k0 + bk + j < K ? to_f(brow[k0 + bk + j]) : 0.f;
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < 16; ++kk) {
      float a[4], v[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) a[i] = sA[kk][tr * 4 + i];
#pragma unroll
      for (int j = 0; j < 4; ++j) v[j] = sB[kk][tc + 16 * j];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], v[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int r = row0 + tr * 4 + i, c = col0 + tc + 16 * j;
      if (r < rows && c < N) C[r * c_row + b * c_head + c] = from_f<O>(acc[i][j]);
    }
}

}  // namespace ksana

using namespace ksana;

// A element (t, b, k) at A + t * a_row + b * a_head + k, C element (t, b, n) at C + t * c_row + b * c_head + n, W
// [heads, N, K] contiguous. kind: 0 all fp32, 1 all bf16, 2 bf16 with fp32 results.
KSANA_API int ksana_head_gemm_any(const void* A, long long a_row, long long a_head, const void* W, void* C,
                                  long long c_row, long long c_head, int rows, int heads, int N, int K, int kind,
                                  cudaStream_t st) {
  if (rows <= 0 || heads <= 0 || N <= 0) return 0;
  const dim3 grid((rows + 31) / 32, (N + 63) / 64, heads);
  using bf16 = __nv_bfloat16;
#define KSANA_HG(T, O)                                                                                                   \
  head_gemm_any_kernel<T, O><<<grid, 128, 0, st>>>(static_cast<const T*>(A), a_row, a_head, static_cast<const T*>(W),    \
                                                   static_cast<O*>(C), c_row, c_head, rows, N, K)
  if (kind == 0) KSANA_HG(float, float); else if (kind == 1) KSANA_HG(bf16, bf16); else KSANA_HG(bf16, float);
#undef KSANA_HG
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}
