// Time mixing: every token's vector mixed with the previous one's, and a linear recurrence whose decay is a function of the
// token, per head and key channel:
//   o_t = (S + diag(u) k_t v_t^T)^T r_t,   S <- diag(w_t) S + k_t v_t^T,   w_t = exp(-exp(z_t + w0))
// over a pool of fp32 slots: a slot holds every head's state [h][d key][d value], then (in its last W numbers) the vector of
// the previous token. A sequence whose first token is part of the step starts from zeros whatever its slot holds. Decays,
// states and sums are 32-bit.
#include "host_common.h"
#include "mixer_common.cuh"

namespace ksana {

// ---- mixes with the previous token ------------------------------------------------------------------------------------
// out[n][t] = h_t + (h_(t-1) - h_t) mu[n]. The first new token of a sequence reads the previous one from the slot; the same
// thread then puts the sequence's last new token there.
template <typename T, int N>
__global__ void __launch_bounds__(256)
token_mix_kernel(const T* __restrict__ h, const float* __restrict__ mu, float* __restrict__ last, long long slot_pitch,
                 const int* __restrict__ slots, const int* __restrict__ cu_q, const int* __restrict__ kv_lens,
                 const int* __restrict__ seq_of_token, T* __restrict__ out, int tokens, int W, int rows) {
  const size_t t = blockIdx.x;
  const int c = (blockIdx.y * 256 + threadIdx.x) * N;
  if (c >= W) return;
  const int b = seq_of_token[t], t0 = cu_q[b], t1 = cu_q[b + 1];
  float x[N], p[N], m[N];
  load_n<N>(h + t * W + c, x);
  if (static_cast<int>(t) != t0) {
    load_n<N>(h + (t - 1) * W + c, p);
  } else {
    const int slot = slots[b];
#pragma unroll
    for (int j = 0; j < N; ++j) p[j] = 0.f;
    if (slot >= 0) {
      float* mem = last + static_cast<size_t>(slot) * slot_pitch + c;
      if (kv_lens[b] != t1 - t0) {
#pragma unroll
        for (int j = 0; j < N; ++j) p[j] = mem[j];
      }
      load_n<N>(h + static_cast<size_t>(t1 - 1) * W + c, m);
#pragma unroll
      for (int j = 0; j < N; ++j) mem[j] = m[j];
    }
  }
  for (int n = 0; n < rows; ++n) {
    load_n<N>(mu + static_cast<size_t>(n) * W + c, m);
#pragma unroll
    for (int j = 0; j < N; ++j) m[j] = fmaf(p[j] - x[j], m[j], x[j]);
    store_n<N>(out + (static_cast<size_t>(n) * tokens + t) * W + c, m);
  }
}

// ---- tanh, as two 16-bit parts where the storage type is 16-bit ------------------------------------------------------------
__global__ void tanh_parts_kernel(const float* __restrict__ x, __nv_bfloat16* __restrict__ out, int n, int total) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= total) return;
  const float v = tanhf(x[i]);
  const __nv_bfloat16 hi = __float2bfloat16_rn(v);
  const size_t row = i / n, c = i % n;
  out[row * 2 * n + c] = hi;
  out[row * 2 * n + n + c] = __float2bfloat16_rn(v - __bfloat162float(hi));
}
__global__ void tanh_kernel(const float* __restrict__ x, float* __restrict__ out, int total) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i < total) out[i] = tanhf(x[i]);
}

// ---- the recurrence, token by token ------------------------------------------------------------------------------------
struct TimeMixArgs {
  const void *r, *k, *v;
  int ldr, ldk, ldv;
  const float* z;    // [T][ldz]
  int ldz;
  const float* w0;   // [h * d]
  const float* u;    // [h * d]
  float* state;
  long long slot_pitch;
  const int* slots;
  const int* cu_q;
  const int* kv_lens;
  int h, d;
  void* out;         // [T][h][d]
};

// One CTA = one (sequence, head, 32 value columns). Thread (tx, ty) owns VEC columns and every 128 / TX-th row. A single new
// token reads and writes the state in global memory once; several keep it in shared memory between them.
template <typename T, int VEC, bool ONE>
__global__ void __launch_bounds__(128)
time_mix_recurrent_kernel(TimeMixArgs a, int seq_base) {
  constexpr int TX = 32 / VEC, TY = 128 / TX;
  extern __shared__ float sm[];
  float* sr = sm;                 // [d]
  float* sk = sr + a.d;           // [d]
  float* sw = sk + a.d;           // [d]: w - 1 (the rounding of a w close to 1 would add up over many tokens)
  float* sv = sw + a.d;           // [32]
  float* part = sv + 32;          // [TY][32]
  float* red = part + TY * 32;    // [32]
  float* sS = red + 32;           // [d][32], several tokens only
  const int b = blockIdx.z + seq_base, head = blockIdx.y, col0 = blockIdx.x * 32, d = a.d;
  const int slot = a.slots[b];
  const int t0 = a.cu_q[b], t1 = a.cu_q[b + 1];
  if (t1 <= t0 || slot < 0) return;
  const bool fresh = a.kv_lens[b] == t1 - t0;
  const int tid = threadIdx.x, tx = tid % TX, ty = tid / TX;
  const int col = col0 + tx * VEC;
  const bool live = col < d;
  float* S = a.state + slot * a.slot_pitch + static_cast<size_t>(head) * d * d + col;
  constexpr int RMAX = ONE ? 8 : 1;
  float pre[RMAX][VEC];  // the single token's share of the state is requested before anything else
  if (ONE && live) {
#pragma unroll
    for (int i = 0; i < RMAX; ++i) {
#pragma unroll
      for (int j = 0; j < VEC; ++j) pre[i][j] = 0.f;
      const int r = ty + i * TY;
      if (r < d && !fresh) load_n<VEC>(S + static_cast<size_t>(r) * d, pre[i]);
    }
  }
  if (!ONE && live) {
    for (int r = ty; r < d; r += TY) {
      float s[VEC];
#pragma unroll
      for (int j = 0; j < VEC; ++j) s[j] = 0.f;
      if (!fresh) load_n<VEC>(S + static_cast<size_t>(r) * d, s);
      store_n<VEC>(sS + r * 32 + tx * VEC, s);
    }
  }
  for (int t = t0; t < t1; ++t) {
    const T* pr = static_cast<const T*>(a.r) + static_cast<size_t>(t) * a.ldr + head * d;
    const T* pk = static_cast<const T*>(a.k) + static_cast<size_t>(t) * a.ldk + head * d;
    const T* pv = static_cast<const T*>(a.v) + static_cast<size_t>(t) * a.ldv + head * d;
    const float* pz = a.z + static_cast<size_t>(t) * a.ldz + head * d;
    float own = 0.f;
    for (int c = tid; c < d; c += 128) {
      const float rv = to_f(pr[c]), kv = to_f(pk[c]);
      sr[c] = rv;
      sk[c] = kv;
      sw[c] = expm1f(-expf(pz[c] + a.w0[head * d + c]));
      own += rv * a.u[head * d + c] * kv;
    }
    if (tid < 32) sv[tid] = col0 + tid < d ? to_f(pv[col0 + tid]) : 0.f;
    own = block_sum(own, red);  // (its barriers also publish the vectors)
    float acc[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) acc[j] = 0.f;
    if (live) {
      float vv[VEC];
#pragma unroll
      for (int j = 0; j < VEC; ++j) vv[j] = sv[tx * VEC + j];
      if (ONE) {
#pragma unroll
        for (int i = 0; i < RMAX; ++i) {
          const int r = ty + i * TY;
          if (r < d) {
            const float kr = sk[r], rr = sr[r], wr = sw[r];
#pragma unroll
            for (int j = 0; j < VEC; ++j) {
              acc[j] += rr * pre[i][j];
              pre[i][j] += fmaf(wr, pre[i][j], kr * vv[j]);
            }
            store_n<VEC>(S + static_cast<size_t>(r) * d, pre[i]);
          }
        }
      }
      for (int r = ty + (ONE ? RMAX * TY : 0); r < d; r += TY) {
        float s[VEC];
        if (ONE) {
#pragma unroll
          for (int j = 0; j < VEC; ++j) s[j] = 0.f;
          if (!fresh) load_n<VEC>(S + static_cast<size_t>(r) * d, s);
        } else {
          load_n<VEC>(sS + r * 32 + tx * VEC, s);
        }
        const float kr = sk[r], rr = sr[r], wr = sw[r];
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          acc[j] += rr * s[j];
          s[j] += fmaf(wr, s[j], kr * vv[j]);
        }
        if (ONE)
          store_n<VEC>(S + static_cast<size_t>(r) * d, s);
        else
          store_n<VEC>(sS + r * 32 + tx * VEC, s);
      }
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) part[ty * 32 + tx * VEC + j] = acc[j];
    __syncthreads();
    if (tid < 32 && col0 + tid < d) {
      float o = own * sv[tid];
#pragma unroll
      for (int i = 0; i < TY; ++i) o += part[i * 32 + tid];
      static_cast<T*>(a.out)[(static_cast<size_t>(t) * a.h + head) * d + col0 + tid] = from_f<T>(o);
    }
    __syncthreads();
  }
  if (!ONE && live) {
    for (int r = ty; r < d; r += TY) {
      float s[VEC];
      load_n<VEC>(sS + r * 32 + tx * VEC, s);
      store_n<VEC>(S + static_cast<size_t>(r) * d, s);
    }
  }
}

template <typename T, int VEC, bool ONE>
static int launch_recurrent(const TimeMixArgs& a, int seq_base, int num_seqs, cudaStream_t st) {
  constexpr int TY = 128 / (32 / VEC);
  const int smem = static_cast<int>(sizeof(float)) * (3 * a.d + 64 + TY * 32 + (ONE ? 0 : a.d * 32));
  auto kern = time_mix_recurrent_kernel<T, VEC, ONE>;
  if (smem > 227 * 1024) return -1;
  if (smem > 48 * 1024 && KSANA_SMEM_ONCE(kern, 227 * 1024) != 0) return -4;
  kern<<<dim3((a.d + 31) / 32, a.h, num_seqs), 128, smem, st>>>(a, seq_base);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

}  // namespace ksana

using namespace ksana;
using bf16 = __nv_bfloat16;

// h [tokens, W], mu [rows, W] -> out [rows, tokens, W]; `last` + slot * slot_pitch: the W numbers of a slot. kind: 0 fp32,
// 1 bf16.
KSANA_API int ksana_token_mix(const void* h, const float* mu, float* last, long long slot_pitch, long long slots_total,
                              const int* slots, const int* cu_q, const int* kv_lens, const int* seq_of_token, void* out,
                              int tokens, int W, int rows, int kind, cudaStream_t st) {
  if (tokens <= 0 || W <= 0) return 0;
  if (slots_total <= 0) return -2;
  auto al = [](const void* p, int n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; };
  const bool vec = !(W & 7) && al(h, 32) && al(out, 32) && al(mu, 16);
  const dim3 grid(tokens, ((vec ? W / 8 : W) + 255) / 256);
#define KSANA_TM(T, N)                                                                                                 \
  token_mix_kernel<T, N><<<grid, 256, 0, st>>>(static_cast<const T*>(h), mu, last, slot_pitch, slots, cu_q, kv_lens,   \
                                               seq_of_token, static_cast<T*>(out), tokens, W, rows)
  if (kind) {
    if (vec) KSANA_TM(bf16, 8); else KSANA_TM(bf16, 1);
  } else {
    if (vec) KSANA_TM(float, 8); else KSANA_TM(float, 1);
  }
#undef KSANA_TM
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

// x [rows, n] fp32 -> tanh; kind 1: [rows, 2 n] bf16 = [hi | lo].
KSANA_API int ksana_tanh_parts(const float* x, int n, void* out, int rows, int kind, cudaStream_t st) {
  const int total = rows * n;
  if (total <= 0) return 0;
  if (kind)
    tanh_parts_kernel<<<(total + 255) / 256, 256, 0, st>>>(x, static_cast<bf16*>(out), n, total);
  else
    tanh_kernel<<<(total + 255) / 256, 256, 0, st>>>(x, static_cast<float*>(out), total);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

// Sequences [seq_base, seq_base + num_seqs); one_token: each has exactly one new token. kind: 0 fp32, 1 bf16 storage of r,
// k, v and out.
KSANA_API int ksana_time_mix_recurrent(const void* r, int ldr, const void* k, int ldk, const void* v, int ldv,
                                       const float* z, int ldz, const float* w0, const float* u, float* state,
                                       long long slot_pitch, const int* slots, const int* cu_q, const int* kv_lens, int h,
                                       int d, void* out, int seq_base, int num_seqs, int one_token, int kind,
                                       cudaStream_t st) {
  if (num_seqs <= 0) return 0;
  TimeMixArgs a{r, k, v, ldr, ldk, ldv, z, ldz, w0, u, state, slot_pitch, slots, cu_q, kv_lens, h, d, out};
  const bool vec = (d & 3) == 0 && (slot_pitch & 3) == 0 && (reinterpret_cast<uintptr_t>(state) & 15) == 0;
#define KSANA_TR(T)                                                                                 \
  (vec ? (one_token ? launch_recurrent<T, 4, true>(a, seq_base, num_seqs, st)                       \
                    : launch_recurrent<T, 4, false>(a, seq_base, num_seqs, st))                     \
       : (one_token ? launch_recurrent<T, 1, true>(a, seq_base, num_seqs, st)                       \
                    : launch_recurrent<T, 1, false>(a, seq_base, num_seqs, st)))
  return kind ? KSANA_TR(bf16) : KSANA_TR(float);
#undef KSANA_TR
}
