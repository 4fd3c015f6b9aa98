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

// ---- prompts: chunks of 64 tokens --------------------------------------------------------------------------------------
// With L_t the sum of log2 w over a chunk's tokens up to t (L = 0 ahead of the first), all products by channel,
//   o_t   = (r_t 2^(L_(t-1))) S + sum_(j < t) (r_t . k_j 2^(L_(t-1) - L_j)) v_j + (r_t u . k_t) v_t
//   S_out = 2^(L_end) S + sum_j (k_j 2^(L_end - L_j)) v_j^T
// in three launches: every chunk's own sum of k v^T (parallel), the scan over a sequence's chunks (elementwise), and the
// outputs (parallel). Scores are taken relative to the start of the 16 tokens that the query belongs to, so that no factor
// of earlier tokens exceeds 1; inside the 16 tokens a factor stays below 2^100, or the scores are summed up one by one. What
// is 32-bit by definition enters the bf16 products as hi + lo. A chunk's scratch entry, [h][d * d + d]: its own sum (then
// the state entering the chunk), and 2^(L_end).
constexpr int TC = 64;

__device__ __forceinline__ size_t chunk_entry(const TimeMixArgs& a, int seq_base, int b, int c) {
  return static_cast<size_t>((a.cu_q[b] - a.cu_q[seq_base]) / TC + (b - seq_base) + c);
}

template <int DP>
struct MixTile {
  static constexpr int LD = DP + 8;           // rows of bf16 tiles, four banks apart from one another
  static constexpr int BYTES = TC * LD * 2;
};

// rows of n tokens of one head (d columns) -> shared memory, the rest zeros
template <int DP>
__device__ __forceinline__ void load_tile(__nv_bfloat16* dst, const void* src, int ld, int t0, int n, int col, int d) {
  constexpr int W = DP / 8;
#pragma unroll 4
  for (int i = threadIdx.x; i < TC * W; i += 128) {
    const int t = i / W, c = i % W * 8;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (t < n && c < d)
      v = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(src) + static_cast<size_t>(t0 + t) * ld + col + c);
    *reinterpret_cast<uint4*>(dst + t * MixTile<DP>::LD + c) = v;
  }
}

// sL[0] = 0, sL[1 + t] = L_t of every channel; tot: [128] floats. Ends with a barrier.
template <int DP>
__device__ __forceinline__ void chunk_decays(const TimeMixArgs& a, int t0, int n, int head, float* sL, float* tot) {
  constexpr int PARTS = 128 / DP, SPAN = TC / PARTS;
  const int c = threadIdx.x % DP, part = threadIdx.x / DP, d = a.d;
  const float w0 = c < d ? a.w0[head * d + c] : 0.f;
  const float* z = a.z + static_cast<size_t>(t0) * a.ldz + head * d + c;
  float run = 0.f;
  for (int i0 = 0; i0 < SPAN; i0 += 8) {
    float x[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int t = part * SPAN + i0 + i;
      x[i] = t < n && c < d ? z[static_cast<size_t>(t) * a.ldz] : -INFINITY;
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      // (beyond 2^-200 a state is gone either way: sums stay small enough for differences between tokens to be exact)
      run -= x[i] == -INFINITY ? 0.f : fminf(expf(x[i] + w0) * LOG2E, 200.f);
      sL[(1 + part * SPAN + i0 + i) * DP + c] = run;
    }
  }
  if (part == 0) sL[c] = 0.f;
  tot[threadIdx.x] = run;
  __syncthreads();
  if (part > 0) {
    float off = 0.f;
    for (int p = 0; p < part; ++p) off += tot[p * DP + c];
#pragma unroll 8
    for (int i = 0; i < SPAN; ++i) sL[(1 + part * SPAN + i) * DP + c] += off;
  }
  __syncthreads();
}

// Launch 1: one (chunk, head). Channels on the rows of K^T V.
template <int DP>
__global__ void __launch_bounds__(128)
time_mix_chunk_kv_kernel(TimeMixArgs a, int seq_base, float* __restrict__ scratch) {
  using M_ = MixTile<DP>;
  constexpr int LD = M_::LD;
  const int b = blockIdx.z + seq_base, c0 = blockIdx.x, head = blockIdx.y, d = a.d;
  const int t0 = a.cu_q[b] + c0 * TC, n = min(TC, a.cu_q[b + 1] - t0);
  if (n <= 0) return;
  extern __shared__ __align__(16) uint8_t smem[];
  float* sL = reinterpret_cast<float*>(smem);  // [65][DP]
  float* tot = sL + (TC + 1) * DP;             // [128]
  __nv_bfloat16* sk = reinterpret_cast<__nv_bfloat16*>(tot + 128);
  __nv_bfloat16* sl = sk + TC * LD;
  __nv_bfloat16* sv = sl + TC * LD;
  load_tile<DP>(sk, a.k, a.ldk, t0, n, head * d, d);
  load_tile<DP>(sv, a.v, a.ldv, t0, n, head * d, d);
  chunk_decays<DP>(a, t0, n, head, sL, tot);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  float* out = scratch + (chunk_entry(a, seq_base, b, c0) * a.h + head) * (static_cast<size_t>(d) * d + d);
  {
    constexpr int PARTS = 128 / DP;
    const int c = tid % DP, part = tid / DP;
    const float end = sL[TC * DP + c];
    if (part == 0 && c < d) out[static_cast<size_t>(d) * d + c] = ex2_ftz(end);
#pragma unroll 8
    for (int t = part; t < TC; t += PARTS) {
      const float x = __bfloat162float(sk[t * LD + c]) * ex2_ftz(end - sL[(1 + t) * DP + c]);
      const __nv_bfloat16 hi = __float2bfloat16_rn(x);
      sk[t * LD + c] = hi;
      sl[t * LD + c] = __float2bfloat16_rn(x - __bfloat162float(hi));
    }
  }
  __syncthreads();
  const int a_row = (lane & 7) + ((lane >> 4) << 3), a_col = ((lane >> 3) & 1) * 8;  // A from rows of tokens, transposed
  const int b_row = (lane & 7) + (lane & 8), b_col = (lane >> 4) * 8;                // B likewise
  const int r = lane >> 2, j2 = (lane & 3) * 2;
  for (int mt = warp; mt < DP / 16; mt += 4) {
    float acc[DP / 8][4];
#pragma unroll
    for (int i = 0; i < DP / 8; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
#pragma unroll
    for (int kb = 0; kb < TC / 16; ++kb) {
      uint32_t fh[4], fl[4];
      ldmatrix_x4<true>(fh, smem_u32(sk + (kb * 16 + a_row) * LD + mt * 16 + a_col));
      ldmatrix_x4<true>(fl, smem_u32(sl + (kb * 16 + a_row) * LD + mt * 16 + a_col));
#pragma unroll
      for (int nt = 0; nt < DP / 16; ++nt) {
        uint32_t fv[4];
        ldmatrix_x4<true>(fv, smem_u32(sv + (kb * 16 + b_row) * LD + nt * 16 + b_col));
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          mma_16816(acc[nt * 2 + x], fh, fv[x * 2], fv[x * 2 + 1]);
          mma_16816(acc[nt * 2 + x], fl, fv[x * 2], fv[x * 2 + 1]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < DP / 8; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int row = mt * 16 + r + e * 8, col = i * 8 + j2;
        if (row < d && col < d)
          *reinterpret_cast<float2*>(out + static_cast<size_t>(row) * d + col) = make_float2(acc[i][e * 2], acc[i][e * 2 + 1]);
      }
  }
}

// Launch 2: turns every chunk's own sum into the state entering that chunk and leaves the final state in the slot.
__global__ void __launch_bounds__(256)
time_mix_chunk_scan_kernel(TimeMixArgs a, int seq_base, float* __restrict__ scratch) {
  const int b = blockIdx.z + seq_base, head = blockIdx.y, d = a.d, per = d * d;  // a multiple of 4
  const int e = (blockIdx.x * 256 + threadIdx.x) * 4;
  const int slot = a.slots[b], q_len = a.cu_q[b + 1] - a.cu_q[b];
  if (e >= per || q_len <= 0 || slot < 0) return;
  float4* S = reinterpret_cast<float4*>(a.state + slot * a.slot_pitch + static_cast<size_t>(head) * per + e);
  float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
  if (a.kv_lens[b] != q_len) s = *S;
  const int chunks = (q_len + TC - 1) / TC;
  const size_t step = static_cast<size_t>(a.h) * (per + d);
  float* p = scratch + (chunk_entry(a, seq_base, b, 0) * a.h + head) * (per + d);
  const float* w = p + per + e / d;
  auto at = [&](int c) { return reinterpret_cast<float4*>(p + c * step + e); };
  // the chain over the chunks is short arithmetic: what it costs is the loads, so AHEAD of them are kept in flight
  constexpr int AHEAD = 8;
  float4 ring[AHEAD];
  float wr[AHEAD];
#pragma unroll
  for (int i = 0; i < AHEAD; ++i)
    if (i < chunks) ring[i] = *at(i), wr[i] = w[i * step];
  for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      const int c = c0 + i;
      if (c < chunks) {
        const float4 v = ring[i];
        const float f = wr[i];
        if (c + AHEAD < chunks) ring[i] = *at(c + AHEAD), wr[i] = w[(c + AHEAD) * step];
        *at(c) = s;
        s.x = f * s.x + v.x; s.y = f * s.y + v.y; s.z = f * s.z + v.z; s.w = f * s.w + v.w;
      }
    }
  }
  *S = s;
}

// Launch 3: outputs of one (chunk, head); a warp has 16 tokens.
template <int DP>
__global__ void __launch_bounds__(128)
time_mix_chunk_out_kernel(TimeMixArgs a, int seq_base, const float* __restrict__ scratch) {
  using M_ = MixTile<DP>;
  constexpr int LD = M_::LD, KB = DP / 16;
  const int b = blockIdx.z + seq_base, c0 = blockIdx.x, head = blockIdx.y, d = a.d;
  const int q_len = a.cu_q[b + 1] - a.cu_q[b], t0 = a.cu_q[b] + c0 * TC, n = min(TC, q_len - c0 * TC);
  if (n <= 0) return;
  const bool has_state = c0 > 0 || a.kv_lens[b] != q_len;
  extern __shared__ __align__(16) uint8_t smem[];
  float* sL = reinterpret_cast<float*>(smem);  // [65][DP]
  float* tot = sL + (TC + 1) * DP;             // [128]
  __nv_bfloat16* sr = reinterpret_cast<__nv_bfloat16*>(tot + 128);
  __nv_bfloat16* sk = sr + TC * LD;
  __nv_bfloat16* sv = sk + TC * LD;
  __nv_bfloat16* s_hi = sv + TC * LD;  // [DP][LD]: the state entering the chunk
  __nv_bfloat16* s_lo = s_hi + DP * LD;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r = lane >> 2, j2 = (lane & 3) * 2;
  load_tile<DP>(sr, a.r, a.ldr, t0, n, head * d, d);
  load_tile<DP>(sk, a.k, a.ldk, t0, n, head * d, d);
  load_tile<DP>(sv, a.v, a.ldv, t0, n, head * d, d);
  if (has_state) {
    const float* S = scratch + (chunk_entry(a, seq_base, b, c0) * a.h + head) * (static_cast<size_t>(d) * d + d);
#pragma unroll 4
    for (int i = tid; i < DP * (DP / 4); i += 128) {
      const int row = i / (DP / 4), col = i % (DP / 4) * 4;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (row < d && col < d) v = *reinterpret_cast<const float4*>(S + static_cast<size_t>(row) * d + col);
      uint2 hi, lo;
      hi.x = split_bf16(v.x, v.y, &lo.x);
      hi.y = split_bf16(v.z, v.w, &lo.y);
      *reinterpret_cast<uint2*>(s_hi + row * LD + col) = hi;
      *reinterpret_cast<uint2*>(s_lo + row * LD + col) = lo;
    }
  }
  chunk_decays<DP>(a, t0, n, head, sL, tot);
  if (warp * 16 >= n) return;  // (no barrier below)
  auto pair_of = [](const __nv_bfloat16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); };
  const float* ref = sL + warp * 16 * DP;  // L ahead of this warp's tokens
  float acc[DP / 8][4];
#pragma unroll
  for (int i = 0; i < DP / 8; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
  const int b_row = (lane & 7) + (lane & 8), b_col = (lane >> 4) * 8;

  // r 2^(L_(t-1) - ref), the share of the entering state, and each token's own score
  uint32_t qh[KB][4], ql[KB][4];
  float own[2] = {0.f, 0.f}, range = 0.f;
#pragma unroll
  for (int kb = 0; kb < KB; ++kb) {
    uint32_t ih[4], il[4];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int c = kb * 16 + u * 8 + j2;
      const float2 f = *reinterpret_cast<const float2*>(ref + c);
      const float2 end = *reinterpret_cast<const float2*>(ref + 16 * DP + c);
      range = fmaxf(range, fmaxf(f.x - end.x, f.y - end.y));
      const float fx = ex2_ftz(f.x), fy = ex2_ftz(f.y);
      const float ux = c < d ? a.u[head * d + c] : 0.f, uy = c < d ? a.u[head * d + c + 1] : 0.f;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = warp * 16 + r + e * 8;
        const float2 x = pair_of(sr + t * LD + c), k = pair_of(sk + t * LD + c);
        const float2 l = *reinterpret_cast<const float2*>(sL + t * DP + c);
        own[e] += x.x * ux * k.x + x.y * uy * k.y;
        const float p = x.x * ex2_ftz(l.x - f.x), q = x.y * ex2_ftz(l.y - f.y);
        qh[kb][u * 2 + e] = split_bf16(p, q, &ql[kb][u * 2 + e]);
        ih[u * 2 + e] = split_bf16(p * fx, q * fy, &il[u * 2 + e]);
      }
    }
    if (has_state) {
#pragma unroll
      for (int nt = 0; nt < KB; ++nt) {
        uint32_t gh[4], gl[4];
        ldmatrix_x4<true>(gh, smem_u32(s_hi + (kb * 16 + b_row) * LD + nt * 16 + b_col));
        ldmatrix_x4<true>(gl, smem_u32(s_lo + (kb * 16 + b_row) * LD + nt * 16 + b_col));
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          mma_16816(acc[nt * 2 + x], ih, gh[x * 2], gh[x * 2 + 1]);
          mma_16816(acc[nt * 2 + x], il, gh[x * 2], gh[x * 2 + 1]);
          mma_16816(acc[nt * 2 + x], ih, gl[x * 2], gl[x * 2 + 1]);
        }
      }
    }
  }
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    own[e] += __shfl_xor_sync(0xffffffffu, own[e], 1);
    own[e] += __shfl_xor_sync(0xffffffffu, own[e], 2);
  }
  const bool steep = __any_sync(0xffffffffu, range > 100.f);

  for (int jb = 0; jb <= warp; ++jb) {
    float s[2][4];
#pragma unroll
    for (int e = 0; e < 4; ++e) s[0][e] = s[1][e] = 0.f;
    if (jb < warp || !steep) {
#pragma unroll
      for (int kb = 0; kb < KB; ++kb)
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          uint32_t kh[2], kl[2];
          const int j = jb * 16 + x * 8 + r;
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            const int c = kb * 16 + u * 8 + j2;
            const float2 k = pair_of(sk + j * LD + c), f = *reinterpret_cast<const float2*>(ref + c);
            const float2 l = *reinterpret_cast<const float2*>(sL + (1 + j) * DP + c);
            kh[u] = split_bf16(k.x * ex2_ftz(f.x - l.x), k.y * ex2_ftz(f.y - l.y), &kl[u]);
          }
          mma_16816(s[x], qh[kb], kh[0], kh[1]);
          mma_16816(s[x], ql[kb], kh[0], kh[1]);
          mma_16816(s[x], qh[kb], kl[0], kl[1]);
        }
    } else {
#pragma unroll
      for (int x = 0; x < 2; ++x)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int t = warp * 16 + r + (e >> 1) * 8, j = jb * 16 + x * 8 + j2 + (e & 1);
          float sum = 0.f;
          if (j < t)
            for (int c = 0; c < d; ++c)
              sum += __bfloat162float(sr[t * LD + c]) * __bfloat162float(sk[j * LD + c]) *
                     ex2_ftz(sL[t * DP + c] - sL[(1 + j) * DP + c]);
          s[x][e] = sum;
        }
    }
    if (jb == warp) {
#pragma unroll
      for (int x = 0; x < 2; ++x)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int t = r + (e >> 1) * 8, j = x * 8 + j2 + (e & 1);
          s[x][e] = j < t ? s[x][e] : j == t ? own[e >> 1] : 0.f;
        }
    }
    uint32_t ph[4], pl[4];
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int e = 0; e < 2; ++e) ph[x * 2 + e] = split_bf16(s[x][e * 2], s[x][e * 2 + 1], &pl[x * 2 + e]);
#pragma unroll
    for (int nt = 0; nt < KB; ++nt) {
      uint32_t fv[4];
      ldmatrix_x4<true>(fv, smem_u32(sv + (jb * 16 + b_row) * LD + nt * 16 + b_col));
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        mma_16816(acc[nt * 2 + x], ph, fv[x * 2], fv[x * 2 + 1]);
        mma_16816(acc[nt * 2 + x], pl, fv[x * 2], fv[x * 2 + 1]);
      }
    }
  }
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out);
#pragma unroll
  for (int i = 0; i < DP / 8; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = warp * 16 + r + e * 8, c = i * 8 + j2;
      if (t < n && c < d)
        *reinterpret_cast<uint32_t*>(out + (static_cast<size_t>(t0 + t) * a.h + head) * d + c) =
            pack_bf16(acc[i][e * 2], acc[i][e * 2 + 1]);
    }
}

template <int DP>
static int launch_chunked(const TimeMixArgs& a, int seq_base, int num_seqs, int max_q, float* scratch, cudaStream_t st) {
  constexpr int base = ((TC + 1) * DP + 128) * 4;
  constexpr int smem_kv = base + 3 * MixTile<DP>::BYTES, smem_out = smem_kv + 2 * DP * MixTile<DP>::LD * 2;
  static_assert(smem_out <= 227 * 1024, "does not fit");
  const dim3 grid((max_q + TC - 1) / TC, a.h, num_seqs);
  auto kv = time_mix_chunk_kv_kernel<DP>;
  auto out = time_mix_chunk_out_kernel<DP>;
  if (KSANA_SMEM_ONCE(kv, smem_kv) != 0 || KSANA_SMEM_ONCE(out, smem_out) != 0) return -4;
  kv<<<grid, 128, smem_kv, st>>>(a, seq_base, scratch);
  time_mix_chunk_scan_kernel<<<dim3((a.d * a.d + 1023) / 1024, a.h, num_seqs), 256, 0, st>>>(a, seq_base, scratch);
  out<<<grid, 128, smem_out, st>>>(a, seq_base, scratch);
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

// fp32 scratch elements that ksana_time_mix_chunked needs for `tokens` tokens in `num_seqs` sequences.
KSANA_API long long ksana_time_mix_scratch(int tokens, int num_seqs, int h, int d) {
  return (static_cast<long long>(tokens) / TC + num_seqs) * h * (static_cast<long long>(d) * d + d);
}

// bf16, chunked form for sequences [seq_base, seq_base + num_seqs), each with at most max_q new tokens. Returns -1 for
// sizes it does not take (d <= 128 in multiples of 8, 16-byte aligned rows and states).
KSANA_API int ksana_time_mix_chunked(const void* r, int ldr, const void* k, int ldk, const void* v, int ldv, const float* z,
                                     int ldz, const float* w0, const float* u, float* state, long long slot_pitch,
                                     const int* slots, const int* cu_q, const int* kv_lens, int h, int d, void* out,
                                     int seq_base, int num_seqs, int max_q, float* scratch, cudaStream_t st) {
  if (num_seqs <= 0 || max_q <= 0) return 0;
  auto rows16 = [](const void* p, long long ld) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0 && (ld & 7) == 0; };
  if (d > 128 || (d & 7) || !rows16(r, ldr) || !rows16(k, ldk) || !rows16(v, ldv) || !rows16(out, 0) || !rows16(scratch, 0) ||
      !rows16(state, 0) || (slot_pitch & 3))
    return -1;
  TimeMixArgs a{r, k, v, ldr, ldk, ldv, z, ldz, w0, u, state, slot_pitch, slots, cu_q, kv_lens, h, d, out};
  if (d <= 32) return launch_chunked<32>(a, seq_base, num_seqs, max_q, scratch, st);
  if (d <= 64) return launch_chunked<64>(a, seq_base, num_seqs, max_q, scratch, st);
  return launch_chunked<128>(a, seq_base, num_seqs, max_q, scratch, st);
}
