// Small helpers of the kernels behind layers with mixers of their own sizes: typed loads and stores that compute in
// 32-bit floats whatever the storage type, and the accurate activations (these files are compiled without fast math).
#pragma once
#include "sm100.cuh"

namespace ksana {

template <typename T>
__device__ __forceinline__ float to_f(T v);
template <>
__device__ __forceinline__ float to_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// N consecutive elements, N = 1, 4 or 8; for N > 1 the address is aligned to N elements.
template <int N>
__device__ __forceinline__ void load_n(const float* p, float* f) {
  if constexpr (N == 1) {
    f[0] = p[0];
  } else {
#pragma unroll
    for (int i = 0; i < N; i += 4) {
      float4 v = *reinterpret_cast<const float4*>(p + i);
      f[i] = v.x; f[i + 1] = v.y; f[i + 2] = v.z; f[i + 3] = v.w;
    }
  }
}
// eight bf16 of one 16-byte word
__device__ __forceinline__ void unpack8(uint4 v, float* f) {
  const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    f[2 * i] = __uint_as_float(w[i] << 16);
    f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
  }
}
template <int N>
__device__ __forceinline__ void load_n(const __nv_bfloat16* p, float* f) {
  if constexpr (N == 1) {
    f[0] = __bfloat162float(p[0]);
  } else if constexpr (N == 4) {
    uint2 v = *reinterpret_cast<const uint2*>(p);
    float2 a = __bfloat1622float2(*reinterpret_cast<__nv_bfloat162*>(&v.x));
    float2 b = __bfloat1622float2(*reinterpret_cast<__nv_bfloat162*>(&v.y));
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  } else {
    unpack8(*reinterpret_cast<const uint4*>(p), f);
  }
}
template <int N>
__device__ __forceinline__ void store_n(float* p, const float* f) {
  if constexpr (N == 1) {
    p[0] = f[0];
  } else {
#pragma unroll
    for (int i = 0; i < N; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(f[i], f[i + 1], f[i + 2], f[i + 3]);
  }
}
template <int N>
__device__ __forceinline__ void store_n(__nv_bfloat16* p, const float* f) {
  if constexpr (N == 1) {
    p[0] = __float2bfloat16_rn(f[0]);
  } else if constexpr (N == 4) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]));
  } else {
    *reinterpret_cast<uint4*>(p) =
        make_uint4(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]), pack_bf16(f[4], f[5]), pack_bf16(f[6], f[7]));
  }
}

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
// The same through the fast exponential and division (relative error about 1e-6): inputs and results here are 16-bit.
__device__ __forceinline__ float silu_fast(float x) { return __fdividef(x, 1.f + __expf(-x)); }
// 0.5 z (1 + tanh u) with u = sqrt(2 / pi) (z + 0.044715 z^3)
__device__ __forceinline__ float gelu_tanh_f(float z) {
  const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
  return z / (1.f + expf(-2.f * u));
}

// For storage type T: 16-bit results take the fast exponential and division.
template <typename T>
__device__ __forceinline__ float gelu_tanh_as(float z) {
  if constexpr (sizeof(T) == 2) {
    const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
    return __fdividef(z, 1.f + __expf(-2.f * u));
  } else {
    return gelu_tanh_f(z);
  }
}

// Hardware approximations (relative error about 1e-7) without the handling of denormal numbers around them.
__device__ __forceinline__ float ex2_ftz(float x) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}
__device__ __forceinline__ float rcp_ftz(float x) {
  float r;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}
__device__ __forceinline__ float rsqrt_ftz(float x) {
  float r;
  asm("rsqrt.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}
constexpr float LOG2E = 1.4426950408889634f;

// v = hi + lo with both parts bf16: the pair keeps 16 bits of the mantissa through 16-bit tensor-core operands. Packs
// two values; *lo is exact up to its own rounding.
__device__ __forceinline__ uint32_t split_bf16(float a, float b, uint32_t* lo) {
  const uint32_t hi = pack_bf16(a, b);
  *lo = pack_bf16(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
  return hi;
}

// ---- warp-wide products of 16-bit operands in registers: c [16 x 8] += a [16 x 16] b [16 x 8] ----
__device__ __forceinline__ void mma_16816(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
template <bool TRANS>
__device__ __forceinline__ void ldmatrix_x4(uint32_t* r, uint32_t addr) {
  if constexpr (TRANS)
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
  else
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
// an 8 x 8 matrix of 16-bit values held across the warp, transposed
__device__ __forceinline__ uint32_t transpose_8x8(uint32_t v) {
  uint32_t r;
  asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(r) : "r"(v));
  return r;
}

// Sum over the block (a multiple of 32 threads, at most 1024); every thread gets it. `red` holds 32 floats.
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();  // earlier readers of red are done
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  for (unsigned i = 0; i < (blockDim.x >> 5); ++i) t += red[i];
  return t;
}

}  // namespace ksana
