// Linear attention with a fixed decay per head over a pool of fp32 state slots: S <- decay S + k v^T, o = S^T q.
//
// q, k, v are the projections as they left the GEMM; the activation, the rotation and the key's scale are applied here
// in 32-bit floats. A sequence whose first token is part of the step starts from a zero state whatever its slot holds.
#include "host_common.h"
#include "mixer_common.cuh"

namespace ksana {

struct LinearAttnArgs {
  const void* q;
  const void* k;
  const void* v;
  int ldq, ldk, ldv;          // token pitches (elements)
  float* state;               // [slots][h][d][dv]
  const int* slots;           // [B]
  const int* cu_q;            // [B + 1]
  const int* kv_lens;         // [B]
  const int* positions;       // [T]
  const float* decay;         // [h]
  const float* rotary;        // [positions][rd] = [cos | sin], or null
  int rd, act, h, d, dv;      // act: 0 none, 1 silu
  float key_scale;
  void* out;                  // [T][h][dv]
};

template <typename T>
__device__ __forceinline__ float la_act(float x, int act) {
  return act ? silu_f(x) : x;
}

// Element c of a head of q or k after activation and rotation.
template <typename T>
__device__ __forceinline__ float la_feature(const T* head, int c, const float* cs, int rd, int act) {
  float x = la_act<T>(to_f(head[c]), act);
  if (c < rd) {
    const int half = rd >> 1;
    const bool low = c < half;
    const int i = low ? c : c - half;
    const float y = la_act<T>(to_f(head[low ? c + half : i]), act);
    x = low ? x * cs[i] - y * cs[half + i] : x * cs[i] + y * cs[half + i];
  }
  return x;
}

// ---- token by token ---------------------------------------------------------------------------------------------
// One CTA = one (sequence, head, 32 columns of the state). Thread (tx, ty) owns VEC columns and every 128 / TX-th row.
// A single new token reads and writes the state in global memory once; several keep it in shared memory between them.
template <typename T, int VEC, bool ONE>
__global__ void __launch_bounds__(128)
linear_recurrent_kernel(LinearAttnArgs a, int seq_base) {
  constexpr int TX = 32 / VEC, TY = 128 / TX;
  extern __shared__ float sm[];
  float* sq = sm;                 // [d]
  float* sk = sq + a.d;           // [d]
  float* sv = sk + a.d;           // [32]
  float* red = sv + 32;           // [TY][32]
  float* sS = red + TY * 32;      // [d][32], several tokens only
  const int b = blockIdx.z + seq_base, head = blockIdx.y, col0 = blockIdx.x * 32;
  const int slot = a.slots[b];
  const int t0 = a.cu_q[b], t1 = a.cu_q[b + 1];
  if (t1 <= t0 || slot < 0) return;
  const bool fresh = a.kv_lens[b] == t1 - t0;
  const int tid = threadIdx.x, tx = tid % TX, ty = tid / TX;
  const int col = col0 + tx * VEC;
  const bool live = col < a.dv;
  float* S = a.state + (static_cast<size_t>(slot) * a.h + head) * a.d * a.dv + col;
  const float dec = a.decay[head];
  if (!ONE && live) {
    for (int r = ty; r < a.d; r += TY) {
      float s[VEC];
#pragma unroll
      for (int j = 0; j < VEC; ++j) s[j] = 0.f;
      if (!fresh) load_n<VEC>(S + static_cast<size_t>(r) * a.dv, s);
      store_n<VEC>(sS + r * 32 + tx * VEC, s);
    }
  }
  for (int t = t0; t < t1; ++t) {
    const T* q = static_cast<const T*>(a.q) + static_cast<size_t>(t) * a.ldq + head * a.d;
    const T* k = static_cast<const T*>(a.k) + static_cast<size_t>(t) * a.ldk + head * a.d;
    const T* v = static_cast<const T*>(a.v) + static_cast<size_t>(t) * a.ldv + head * a.dv;
    const float* cs = a.rotary ? a.rotary + static_cast<size_t>(a.positions[t]) * a.rd : nullptr;
    for (int c = tid; c < a.d; c += 128) {
      sq[c] = la_feature(q, c, cs, a.rd, a.act);
      sk[c] = la_feature(k, c, cs, a.rd, a.act) * a.key_scale;
    }
    if (tid < 32 && col0 + tid < a.dv) sv[tid] = to_f(from_f<T>(la_act<T>(to_f(v[col0 + tid]), a.act)));
    __syncthreads();
    float acc[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) acc[j] = 0.f;
    if (live) {
      float vv[VEC];
#pragma unroll
      for (int j = 0; j < VEC; ++j) vv[j] = sv[tx * VEC + j];
#pragma unroll 8
      for (int r = ty; r < a.d; r += TY) {
        float s[VEC];
        if (ONE) {
#pragma unroll
          for (int j = 0; j < VEC; ++j) s[j] = 0.f;
          if (!fresh) load_n<VEC>(S + static_cast<size_t>(r) * a.dv, s);
        } else {
          load_n<VEC>(sS + r * 32 + tx * VEC, s);
        }
        const float kr = sk[r], qr = sq[r];
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          s[j] = dec * s[j] + kr * vv[j];
          acc[j] += qr * s[j];
        }
        if (ONE)
          store_n<VEC>(S + static_cast<size_t>(r) * a.dv, s);
        else
          store_n<VEC>(sS + r * 32 + tx * VEC, s);
      }
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) red[ty * 32 + tx * VEC + j] = acc[j];
    __syncthreads();
    if (tid < 32 && col0 + tid < a.dv) {
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < TY; ++i) o += red[i * 32 + tid];
      static_cast<T*>(a.out)[(static_cast<size_t>(t) * a.h + head) * a.dv + col0 + tid] = from_f<T>(o);
    }
  }
  if (!ONE && live) {
    for (int r = ty; r < a.d; r += TY) {
      float s[VEC];
      load_n<VEC>(sS + r * 32 + tx * VEC, s);
      store_n<VEC>(S + static_cast<size_t>(r) * a.dv, s);
    }
  }
}

template <typename T, int VEC, bool ONE>
static int launch_recurrent(const LinearAttnArgs& a, int seq_base, int num_seqs, cudaStream_t st) {
  constexpr int TY = 128 / (32 / VEC);
  const int smem = static_cast<int>(sizeof(float)) * (2 * a.d + 32 + TY * 32 + (ONE ? 0 : a.d * 32));
  auto kern = linear_recurrent_kernel<T, VEC, ONE>;
  if (smem > 227 * 1024) return -1;
  if (smem > 48 * 1024 && KSANA_SMEM_ONCE(kern, 227 * 1024) != 0) return -4;
  kern<<<dim3((a.dv + 31) / 32, a.h, num_seqs), 128, smem, st>>>(a, seq_base);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

}  // namespace ksana

using namespace ksana;

// Token-by-token form for sequences [seq_base, seq_base + num_seqs). kind: 0 fp32, 1 bf16 storage of q, k, v and out.
// one_token: every one of these sequences has exactly one new token.
KSANA_API int ksana_linear_recurrent(const void* q, int ldq, const void* k, int ldk, const void* v, int ldv, float* state,
                                     const int* slots, const int* cu_q, const int* kv_lens, const int* positions,
                                     const float* decay, const float* rotary, int rd, int act, float key_scale, int h,
                                     int d, int dv, void* out, int seq_base, int num_seqs, int one_token, int kind,
                                     cudaStream_t st) {
  if (num_seqs <= 0) return 0;
  LinearAttnArgs a{q, k, v, ldq, ldk, ldv, state, slots, cu_q, kv_lens, positions, decay, rotary, rd, act, h, d, dv,
                   key_scale, out};
  const bool vec = (dv & 3) == 0;
#define KSANA_LR(T)                                                                                 \
  (vec ? (one_token ? launch_recurrent<T, 4, true>(a, seq_base, num_seqs, st)                       \
                    : launch_recurrent<T, 4, false>(a, seq_base, num_seqs, st))                     \
       : (one_token ? launch_recurrent<T, 1, true>(a, seq_base, num_seqs, st)                       \
                    : launch_recurrent<T, 1, false>(a, seq_base, num_seqs, st)))
  return kind ? KSANA_LR(__nv_bfloat16) : KSANA_LR(float);
#undef KSANA_LR
}
