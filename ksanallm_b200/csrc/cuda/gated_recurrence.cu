// The core of a gated linear recurrent block: a short causal convolution, the gates' block-diagonal products, the
// recurrence per channel, and the product with the GELU branch.
//
//   u_t = conv_b + sum_j conv_w[:, j] x_(t - K + 1 + j)
//   r = sigmoid(z_r), i = sigmoid(z_i), z = W u + b per block, log a = -r rate
//   S_t = a S_(t-1) + sqrt(1 - a^2) i u,   out = S gelu(y)
//
// A sequence's memory is one slot of fp32: [K][C], row 0 the state S, rows 1 .. K - 1 the last K - 1 inputs x, oldest
// first. A sequence whose first token is among the new ones does not read it.
#include "host_common.h"
#include "mixer_common.cuh"

namespace ksana {

// a - 1 and sqrt(1 - a^2) from log a <= 0. The recurrence runs as S + (a - 1) S: over thousands of tokens the rounding of
// an a close to 1 would add up.
__device__ __forceinline__ void decay_of(float la, float* am1, float* in) {
  *am1 = expm1f(la);
  *in = sqrtf(-*am1 * (2.f + *am1));
}

struct RecurrenceArgs {
  const void* y;
  int ldy;
  const void* x;
  int ldx;
  float* state;            // [slots][K][C]
  const int* slots;
  const int* cu_q;
  const int* kv_lens;
  const float* conv_w;     // [K, C]
  const float* conv_b;
  const float* gates_b;    // [2, C]
  const float* rate;       // [C]
  void* out;
  int ldo, C, K, B;
};

// ---- any size, any storage type ---------------------------------------------------------------------------------------
// u of every new token; one thread per (token, channel).
template <typename T>
__global__ void __launch_bounds__(256)
recurrence_conv_kernel(RecurrenceArgs a, const int* __restrict__ seq_of_token, T* __restrict__ u, int tok_base) {
  const int c = blockIdx.x * 256 + threadIdx.x;
  if (c >= a.C) return;
  const int t = tok_base + blockIdx.y, b = seq_of_token[t];
  const int q0 = a.cu_q[b], n = a.cu_q[b + 1] - q0, i = t - q0;
  const bool fresh = a.kv_lens[b] == n;
  const float* mem = a.state + static_cast<size_t>(a.slots[b]) * a.K * a.C;
  const T* x = static_cast<const T*>(a.x);
  float s = a.conv_b[c];
  for (int j = 0; j < a.K; ++j) {
    const int back = i - (a.K - 1) + j;  // token of this portion, or one of the inputs before it
    float v = 0.f;
    if (back >= 0)
      v = to_f(x[static_cast<size_t>(q0 + back) * a.ldx + c]);
    else if (!fresh)
      v = mem[static_cast<size_t>(a.K + back) * a.C + c];
    s = fmaf(a.conv_w[static_cast<size_t>(j) * a.C + c], v, s);
  }
  u[static_cast<size_t>(t - tok_base) * a.C + c] = from_f<T>(s);
}

// The recurrence itself, token by token; one thread per (sequence, channel). z: [token][block][r outputs | i outputs].
template <typename T>
__global__ void __launch_bounds__(128)
recurrence_scan_kernel(RecurrenceArgs a, const T* __restrict__ u, const float* __restrict__ z, int seq_base, int tok_base) {
  const int c = blockIdx.x * 128 + threadIdx.x;
  if (c >= a.C) return;
  const int b = seq_base + blockIdx.y;
  const int q0 = a.cu_q[b], n = a.cu_q[b + 1] - q0;
  if (n <= 0) return;
  const bool fresh = a.kv_lens[b] == n;
  float* mem = a.state + static_cast<size_t>(a.slots[b]) * a.K * a.C + c;
  const int part = a.C / a.B, blk = c / part, off = c % part;
  const float rate = a.rate[c], br = a.gates_b[c], bi = a.gates_b[a.C + c];
  float S = fresh ? 0.f : mem[0];
  const T* y = static_cast<const T*>(a.y);
  T* out = static_cast<T*>(a.out);
  for (int t = q0; t < q0 + n; ++t) {
    const size_t row = t - tok_base;
    const float* zt = z + (row * a.B + blk) * 2 * part + off;
    float am1, in;
    decay_of(-sigmoid_f(zt[0] + br) * rate, &am1, &in);
    S = fmaf(am1, S, S) + in * sigmoid_f(zt[part] + bi) * to_f(u[row * a.C + c]);
    out[static_cast<size_t>(t) * a.ldo + c] = from_f<T>(S * gelu_tanh_f(to_f(y[static_cast<size_t>(t) * a.ldy + c])));
  }
  mem[0] = S;
  // the last K - 1 inputs: those of this portion, behind what stays of the earlier ones
  const T* x = static_cast<const T*>(a.x);
  for (int j = 1; j < a.K; ++j) {
    const int back = n - a.K + j;  // token of this portion that moves into row j
    float v = 0.f;
    if (back >= 0)
      v = to_f(x[static_cast<size_t>(q0 + back) * a.ldx + c]);
    else if (!fresh)
      v = mem[static_cast<size_t>(a.K + back) * a.C];  // row K + back > j: not overwritten yet
    mem[static_cast<size_t>(j) * a.C] = v;
  }
}

// ---- bf16 on the tensor cores ---------------------------------------------------------------------------------------
// One CTA = 128 output channels of one block x TC columns, 256 threads. A column is a token of a prompt, or (STEP) the
// single new token of one sequence.
//   convolution   u of the block's channels -> shared memory, bf16, K-major with 128-byte swizzle
//   products      Z_r = W_r u^T and Z_i = W_i u^T: 128 x TC x s, the channels on the MMA rows -> TMEM
//   gates         thread (g, m) owns channel m (TMEM lane m) and walks along half g of the columns
// so the recurrence over a chunk (half a tile) is a loop in registers. Prompts: every chunk of 64 tokens runs on its own
// from S = 0 and leaves S and the running sum of log2 a per token; recurrence_carry_kernel takes the states from chunk to
// chunk and recurrence_finish_kernel adds each chunk's entering state, S_t + 2^(sum log2 a) S_in, and multiplies by the
// other branch. STEP: the state is read, advanced and written here.
constexpr int RG_MAX_PART = 256;  // channels of a block

template <int TC>
struct RecurrenceSmem {
  static constexpr int U_BYTES = TC * 128;       // one 64-channel column block of u
  static constexpr int W_BYTES = 128 * 128;      // one 64-column block of a gate's rows
  __host__ __device__ static int total(int kc) { return kc * (U_BYTES + 2 * W_BYTES) + 256 + 1024; }
};

// 1 / (1 + 2^x): the sigmoid of -x ln 2
__device__ __forceinline__ float sigmoid_log2(float x) { return rcp_ftz(1.f + ex2_ftz(x)); }
// l = log2 a <= 0 -> a - 1 and sqrt(1 - a^2). a - 1 = e^(l ln 2) - 1 is its Taylor series
// where the difference would cancel.
__device__ __forceinline__ void decay_fast(float l, float* am1, float* in) {
  constexpr float c = 0.6931471805599453f;  // ln 2
  const float small = l * fmaf(l, fmaf(l, fmaf(l, c * c * c * c / 24.f, c * c * c / 6.f), c * c / 2.f), c);
  const float d = l > -0.05f ? small : ex2_ftz(l) - 1.f;
  const float w = fmaxf(-d * (2.f + d), 1e-30f);
  *am1 = d;
  *in = w * rsqrt_ftz(w);
}

template <int TC, int KT, bool STEP>
__global__ void __launch_bounds__(256)
recurrence_tile_kernel(const __grid_constant__ CUtensorMap tmW, RecurrenceArgs a, int seq_base, int num_seqs,
                       float* __restrict__ local, float* __restrict__ decay, int tok_base, unsigned int* err) {
  using L_ = RecurrenceSmem<TC>;
  const int part = a.C / a.B, groups = (part + 127) / 128;
  const int blk = blockIdx.y / groups, m0 = blockIdx.y % groups * 128;
  const int tid = threadIdx.x, warp = tid >> 5;
  constexpr int HALF = TC / 2;  // columns per thread
  const int m = m0 + (tid & 127), half0 = (tid >> 7) * HALF;
  const bool mine = m < part;
  const int ch = blk * part + (mine ? m : 0);
  // columns: tokens [q0 + i0, + n) of one sequence, or sequences [first, + n)
  int b = 0, q0 = 0, i0 = 0, n;
  bool fresh = false;
  if constexpr (STEP) {
    i0 = seq_base + blockIdx.x * TC;
    n = min(TC, seq_base + num_seqs - i0);
  } else {
    b = seq_base + blockIdx.z;
    q0 = a.cu_q[b];
    const int q_len = a.cu_q[b + 1] - q0;
    i0 = blockIdx.x * TC;
    n = min(TC, q_len - i0);
    if (n <= 0) return;
    fresh = a.kv_lens[b] == q_len;
  }
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int kc = (part + 63) / 64;
  uint8_t* sU = smem;
  uint8_t* sW = smem + kc * L_::U_BYTES;  // [gate][kc]
  uint64_t* w_full = reinterpret_cast<uint64_t*>(sW + 2 * kc * L_::W_BYTES);
  uint64_t* z_done = w_full + 1;
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(z_done + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_holder + 1);
  constexpr int TM_COLS = 2 * TC < 32 ? 32 : 2 * TC;
  if (tid == 0) {
    mbar_init(w_full, 1);
    mbar_init(z_done, 1);
    *abort_flag = 0;
    fence_mbar_init();
    mbar_expect_tx(w_full, 2 * kc * L_::W_BYTES);
    for (int g = 0; g < 2; ++g)
      for (int k = 0; k < kc; ++k)
        tma_load_2d(sW + (g * kc + k) * L_::W_BYTES, &tmW, w_full, k * 64, (g * a.B + blk) * part + m0);
  }
  if (warp == 0) {
    tmem_alloc(tmem_holder, TM_COLS);
    tmem_relinquish();
  }

  // STEP: what the gates will meet is under way while the products are made
  [[maybe_unused]] float old[STEP ? HALF : 1], yy[STEP ? HALF : 1];
  [[maybe_unused]] float* mem_at[STEP ? HALF : 1];
  [[maybe_unused]] int row_at[STEP ? HALF : 1];
  if constexpr (STEP) {
#pragma unroll
    for (int j = 0; j < HALF; ++j) {
      const int sb = i0 + min(half0 + j, n - 1);
      row_at[j] = a.cu_q[sb];
      mem_at[j] = a.state + static_cast<size_t>(a.slots[sb]) * a.K * a.C + ch;
      old[j] = a.kv_lens[sb] == 1 ? 0.f : *mem_at[j];
      yy[j] = __bfloat162float(static_cast<const __nv_bfloat16*>(a.y)[static_cast<size_t>(row_at[j]) * a.ldy + ch]);
    }
  }

  // ---- u -> shared memory
  const __nv_bfloat16* x = static_cast<const __nv_bfloat16*>(a.x) + blk * part;
  const int vecs = part / 8, strips = STEP ? TC : TC / 8;
  for (int w = tid; w < kc * 8 * strips; w += 256) {
    const int v = w % (kc * 8), strip = w / (kc * 8), c = v * 8;
    uint8_t* dst = sU + (v >> 3) * L_::U_BYTES;
    auto put = [&](int r, const float* f) {
      *reinterpret_cast<uint4*>(dst + r * 128 + (((v & 7) ^ (r & 7)) << 4)) =
          make_uint4(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]), pack_bf16(f[4], f[5]), pack_bf16(f[6], f[7]));
    };
    const float zero[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    constexpr int ROWS = STEP ? 1 : 8;
    if (v >= vecs || strip * ROWS >= n) {
      for (int r = 0; r < ROWS; ++r) put(strip * ROWS + r, zero);
      continue;
    }
    const int ch = blk * part + c;
    // STEP: the inputs before this one and this one; else the strip's and those before it, all loads in flight together
    [[maybe_unused]] uint4 raw[STEP ? 1 : ROWS + KT - 1];
    if constexpr (!STEP) {
      const float* mem = a.state + static_cast<size_t>(a.slots[b]) * a.K * a.C + ch;
#pragma unroll
      for (int j = 0; j < ROWS + KT - 1; ++j) {
        const int i = i0 + strip * ROWS + j - (KT - 1);  // token of this portion, or what came before it
        raw[j] = make_uint4(0u, 0u, 0u, 0u);
        if (i >= 0) {
          if (i < i0 + n) raw[j] = *reinterpret_cast<const uint4*>(x + static_cast<size_t>(q0 + i) * a.ldx + c);
        } else if (!fresh && i > -a.K) {
          float f[8];
          load_n<8>(mem + static_cast<size_t>(a.K + i) * a.C, f);
          raw[j] = make_uint4(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]), pack_bf16(f[4], f[5]), pack_bf16(f[6], f[7]));
        }
      }
    }
    float taps[KT][8], bias[8];  // taps[KT - 1] meets the newest input
    [[maybe_unused]] float win[STEP ? KT : 1][8];
    load_n<8>(a.conv_b + ch, bias);
#pragma unroll
    for (int j = 0; j < KT; ++j) {
      if (j >= KT - a.K) {
        load_n<8>(a.conv_w + static_cast<size_t>(j - (KT - a.K)) * a.C + ch, taps[j]);
      } else {
#pragma unroll
        for (int e = 0; e < 8; ++e) taps[j][e] = 0.f;
      }
    }
    if constexpr (STEP) {
      const int sb = i0 + strip, t = a.cu_q[sb];
      const bool first = a.kv_lens[sb] == 1;
      float* mem = a.state + static_cast<size_t>(a.slots[sb]) * a.K * a.C + ch;
#pragma unroll
      for (int j = 0; j < KT - 1; ++j) {
        const int row = a.K - (KT - 1) + j;  // the state's rows 1 .. K - 1
        if (row >= 1 && !first)
          load_n<8>(mem + static_cast<size_t>(row) * a.C, win[j]);
        else
#pragma unroll
          for (int e = 0; e < 8; ++e) win[j][e] = 0.f;
      }
      load_n<8>(x + static_cast<size_t>(t) * a.ldx + c, win[KT - 1]);
      float f[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        f[e] = bias[e];
#pragma unroll
        for (int j = 0; j < KT; ++j) f[e] = fmaf(taps[j][e], win[j][e], f[e]);
      }
      put(strip, f);
      if (groups == 1) {  // else other CTAs read these rows: recurrence_shift_kernel moves them afterwards
#pragma unroll
        for (int j = 0; j < KT - 1; ++j) {
          const int row = a.K - (KT - 1) + j;
          if (row >= 1) store_n<8>(mem + static_cast<size_t>(row) * a.C, win[j + 1]);
        }
      }
    } else {
      float in[KT][8];
#pragma unroll
      for (int j = 0; j < KT - 1; ++j) unpack8(raw[j], in[j]);
#pragma unroll
      for (int r = 0; r < ROWS; ++r) {
        unpack8(raw[r + KT - 1], in[(r + KT - 1) % KT]);
        float f[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          f[e] = bias[e];
#pragma unroll
          for (int j = 0; j < KT; ++j) f[e] = fmaf(taps[j][e], in[(r + j) % KT][e], f[e]);
          if (strip * ROWS + r >= n) f[e] = 0.f;
        }
        put(strip * ROWS + r, f);
      }
    }
  }
  fence_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_holder;
  bool ok = true;
  if (tid == 0) {
    ok = mbar_wait_bounded(w_full, 0, abort_flag, err);
    if (ok) {
      tc_fence_after();
      constexpr uint32_t idesc = umma_idesc(128, TC, 1, 1);
      for (int g = 0; g < 2; ++g)
        for (int k = 0; k < (part + 15) / 16; ++k)
          umma_f16(tmem + g * TC, umma_desc_k128(smem_u32(sW + (g * kc + (k >> 2)) * L_::W_BYTES) + (k & 3) * 32),
                   umma_desc_k128(smem_u32(sU + (k >> 2) * L_::U_BYTES) + (k & 3) * 32), idesc, k > 0 ? 1u : 0u);
      umma_commit(z_done);
    }
  }
  __syncwarp();
  ok = mbar_wait_bounded(z_done, 0, abort_flag, err);
  if (__all_sync(0xffffffffu, ok)) {
    tc_fence_after();
    const float rate2 = -a.rate[ch] * LOG2E, br2 = -a.gates_b[ch] * LOG2E, bi2 = -a.gates_b[a.C + ch] * LOG2E;
    const uint32_t tm = tmem + (static_cast<uint32_t>((warp & 3) * 32) << 16);
    const uint8_t* u_col = sU + (m >> 6) * L_::U_BYTES + (m & 7) * 2;
    const int u_vec = (m >> 3) & 7;
    float S = 0.f, sum = 0.f;
    constexpr int N = HALF < 16 ? 8 : 16;
    static_assert(HALF % N == 0, "a thread's columns come in whole loads");
    const int end = min(half0 + HALF, n);
    float* lp = nullptr;
    float* dp = nullptr;
    if constexpr (!STEP) {
      const size_t at = static_cast<size_t>(q0 - tok_base + i0 + half0) * a.C + ch;
      lp = local + at;
      dp = decay + at;
    }
#pragma unroll 1
    for (int c0 = half0; c0 < end; c0 += N) {  // uniform over the warp
      uint32_t zr[N], zi[N];
      __syncwarp();
      if constexpr (N == 8) {
        tmem_ld8(tm + c0, zr);
        tmem_ld8(tm + TC + c0, zi);
      } else {
        tmem_ld16(tm + c0, zr);
        tmem_ld16(tm + TC + c0, zi);
      }
      tmem_wait_ld();
      float dec[N], in[N], l2[N];
#pragma unroll
      for (int j = 0; j < N; ++j) {
        const int r = c0 + j;
        const float u = mine ? __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(u_col + r * 128 + ((u_vec ^ (r & 7)) << 4))) : 0.f;
        l2[j] = sigmoid_log2(fmaf(__uint_as_float(zr[j]), -LOG2E, br2)) * rate2;
        decay_fast(l2[j], &dec[j], &in[j]);
        in[j] *= sigmoid_log2(fmaf(__uint_as_float(zi[j]), -LOG2E, bi2)) * u;
      }
      if constexpr (STEP) {
#pragma unroll
        for (int j = 0; j < N; ++j)
          if (mine && c0 + j < n) {
            const float s = fmaf(dec[j], old[j], old[j]) + in[j];
            *mem_at[j] = s;
            static_cast<__nv_bfloat16*>(a.out)[static_cast<size_t>(row_at[j]) * a.ldo + ch] =
                __float2bfloat16_rn(s * gelu_tanh_as<__nv_bfloat16>(yy[j]));
          }
      } else {
#pragma unroll
        for (int j = 0; j < N; ++j) {
          S = fmaf(dec[j], S, S) + in[j];
          sum += l2[j];
          if (mine && c0 + j < n) {
            *lp = S;
            *dp = sum;
          }
          lp += a.C;
          dp += a.C;
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(tmem, TM_COLS);
  }
}

// The states that enter a sequence's chunks, its last state, and the inputs its next portion's convolution needs. One
// thread per (sequence, channel).
template <int TC>
__global__ void __launch_bounds__(128)
recurrence_carry_kernel(RecurrenceArgs a, int seq_base, const float* __restrict__ local, const float* __restrict__ decay,
                        float* __restrict__ carry, int max_chunks, int tok_base) {
  const int c = blockIdx.x * 128 + threadIdx.x;
  if (c >= a.C) return;
  const int b = seq_base + blockIdx.y;
  const int q0 = a.cu_q[b], n = a.cu_q[b + 1] - q0;
  if (n <= 0) return;
  const bool fresh = a.kv_lens[b] == n;
  float* mem = a.state + static_cast<size_t>(a.slots[b]) * a.K * a.C + c;
  float S = fresh ? 0.f : mem[0];
  const int chunks = (n + TC - 1) / TC;
  constexpr int U = 16;
  for (int j0 = 0; j0 < chunks; j0 += U) {
    float s[U], d[U];
#pragma unroll
    for (int j = 0; j < U; ++j)
      if (j0 + j < chunks) {
        const size_t at = static_cast<size_t>(q0 - tok_base + min((j0 + j + 1) * TC, n) - 1) * a.C + c;
        s[j] = local[at];
        d[j] = decay[at];
      }
#pragma unroll
    for (int j = 0; j < U; ++j)
      if (j0 + j < chunks) {
        carry[(static_cast<size_t>(blockIdx.y) * max_chunks + j0 + j) * a.C + c] = S;
        S = fmaf(exp2f(d[j]), S, s[j]);
      }
  }
  mem[0] = S;
  const __nv_bfloat16* x = static_cast<const __nv_bfloat16*>(a.x);
  for (int j = 1; j < a.K; ++j) {
    const int back = n - a.K + j;  // as in recurrence_scan_kernel
    float v = 0.f;
    if (back >= 0)
      v = __bfloat162float(x[static_cast<size_t>(q0 + back) * a.ldx + c]);
    else if (!fresh)
      v = mem[static_cast<size_t>(a.K + back) * a.C];
    mem[static_cast<size_t>(j) * a.C] = v;
  }
}

// out = (S of the chunk alone + a's product so far * entering state) * gelu(y); 4 channels per thread
template <int TC>
__global__ void __launch_bounds__(256)
recurrence_finish_kernel(RecurrenceArgs a, const int* __restrict__ seq_of_token, int seq_base,
                         const float* __restrict__ local, const float* __restrict__ decay,
                         const float* __restrict__ carry, int max_chunks, int tok_base) {
  const int c = (blockIdx.y * 256 + threadIdx.x) * 4;
  if (c >= a.C) return;
  const int t = tok_base + blockIdx.x, b = seq_of_token[t];
  const int chunk = (t - a.cu_q[b]) / TC;
  float s[4], d[4], in[4], y[4];
  load_n<4>(local + static_cast<size_t>(blockIdx.x) * a.C + c, s);
  load_n<4>(decay + static_cast<size_t>(blockIdx.x) * a.C + c, d);
  load_n<4>(carry + (static_cast<size_t>(b - seq_base) * max_chunks + chunk) * a.C + c, in);
  load_n<4>(static_cast<const __nv_bfloat16*>(a.y) + static_cast<size_t>(t) * a.ldy + c, y);
#pragma unroll
  for (int j = 0; j < 4; ++j) s[j] = fmaf(ex2_ftz(d[j]), in[j], s[j]) * gelu_tanh_as<__nv_bfloat16>(y[j]);
  store_n<4>(static_cast<__nv_bfloat16*>(a.out) + static_cast<size_t>(t) * a.ldo + c, s);
}

// One step's inputs move into the last rows of the memory, where recurrence_tile_kernel could not do it.
__global__ void __launch_bounds__(256)
recurrence_shift_kernel(RecurrenceArgs a, int seq_base) {
  const int c = blockIdx.x * 256 + threadIdx.x, b = seq_base + blockIdx.y;
  if (c >= a.C) return;
  float* mem = a.state + static_cast<size_t>(a.slots[b]) * a.K * a.C + c;
  const bool first = a.kv_lens[b] == 1;
  for (int j = 1; j < a.K; ++j)
    mem[static_cast<size_t>(j) * a.C] =
        j == a.K - 1 ? __bfloat162float(static_cast<const __nv_bfloat16*>(a.x)[static_cast<size_t>(a.cu_q[b]) * a.ldx + c])
        : first      ? 0.f
                     : mem[static_cast<size_t>(j + 1) * a.C];
}

static bool tile_sizes(const RecurrenceArgs& a, const void* gates) {
  auto rows16 = [](const void* p, int ld) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0 && (ld & 7) == 0; };
  const int part = a.C / a.B;
  return part % 8 == 0 && part <= RG_MAX_PART && a.K >= 1 && a.K <= 8 && rows16(a.x, a.ldx) && rows16(a.y, a.ldy) &&
         rows16(a.out, a.ldo) && rows16(gates, 0) && rows16(a.state, 0) &&
         rows16(a.conv_w, 0) && rows16(a.conv_b, 0);
}

template <int TC, int KT, bool STEP>
static int launch_tile(const RecurrenceArgs& a, const void* gates, int seq_base, int num_seqs, int columns, float* local,
                       float* decay, int tok_base, cudaStream_t st) {
  const int part = a.C / a.B, kc = (part + 63) / 64, smem = RecurrenceSmem<TC>::total(kc);
  CUtensorMap tw;
  if (make_tmap_2d(&tw, gates, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, static_cast<uint64_t>(2) * a.C, part, part, 128, 64,
                   CU_TENSOR_MAP_SWIZZLE_128B))
    return -3;
  auto kern = recurrence_tile_kernel<TC, KT, STEP>;
  if (KSANA_SMEM_ONCE(kern, RecurrenceSmem<TC>::total(RG_MAX_PART / 64)) != 0) return -4;
  const dim3 grid((columns + TC - 1) / TC, a.B * ((part + 127) / 128), STEP ? 1 : num_seqs);
  kern<<<grid, 256, smem, st>>>(tw, a, seq_base, num_seqs, local, decay, tok_base, error_word());
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

constexpr int RG_TILE = 128, RG_CHUNK = RG_TILE / 2, RG_STEP = 16;

}  // namespace ksana

using namespace ksana;

// Floats of scratch that ksana_recurrence_prompts needs.
KSANA_API long long ksana_recurrence_scratch(int tokens, int num_seqs, int max_q, int C) {
  return (2LL * tokens + static_cast<long long>(num_seqs) * ((max_q + RG_CHUNK - 1) / RG_CHUNK)) * C;
}

// bf16. Sequences [seq_base, seq_base + num_seqs), whose tokens are [tok_base, tok_base + tokens), at most max_q each.
// conv_w: [K, C], gates: [2, B, C / B, C / B]. -1: sizes it does not take.
KSANA_API int ksana_recurrence_prompts(const void* y, int ldy, const void* x, int ldx, float* state, const int* slots,
                                       const int* cu_q, const int* kv_lens, const int* seq_of_token, const float* conv_w,
                                       const float* conv_b, const void* gates, const float* gates_b, const float* rate,
                                       int C, int K, int B, void* out, int ldo, int seq_base, int num_seqs, int tok_base,
                                       int tokens, int max_q, float* scratch, cudaStream_t st) {
  if (num_seqs <= 0 || tokens <= 0) return 0;
  if (B < 1 || C % B || K < 1) return -2;
  RecurrenceArgs a{y, ldy, x, ldx, state, slots, cu_q, kv_lens, conv_w, conv_b, gates_b, rate, out, ldo, C, K, B};
  if (!tile_sizes(a, gates)) return -1;
  const int max_chunks = (max_q + RG_CHUNK - 1) / RG_CHUNK;
  float *local = scratch, *decay = local + static_cast<size_t>(tokens) * C, *carry = decay + static_cast<size_t>(tokens) * C;
  const int rc = K <= 4 ? launch_tile<RG_TILE, 4, false>(a, gates, seq_base, num_seqs, max_q, local, decay, tok_base, st)
                        : launch_tile<RG_TILE, 8, false>(a, gates, seq_base, num_seqs, max_q, local, decay, tok_base, st);
  if (rc) return rc;
  recurrence_carry_kernel<RG_CHUNK><<<dim3((C + 127) / 128, num_seqs), 128, 0, st>>>(a, seq_base, local, decay, carry,
                                                                                     max_chunks, tok_base);
  recurrence_finish_kernel<RG_CHUNK><<<dim3(tokens, (C + 1023) / 1024), 256, 0, st>>>(a, seq_of_token, seq_base, local,
                                                                                      decay, carry, max_chunks, tok_base);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

// bf16. Sequences [seq_base, seq_base + num_seqs) with exactly one new token each. -1: sizes it does not take.
KSANA_API int ksana_recurrence_step(const void* y, int ldy, const void* x, int ldx, float* state, const int* slots,
                                    const int* cu_q, const int* kv_lens, const float* conv_w, const float* conv_b,
                                    const void* gates, const float* gates_b, const float* rate, int C, int K, int B,
                                    void* out, int ldo, int seq_base, int num_seqs, cudaStream_t st) {
  if (num_seqs <= 0) return 0;
  if (B < 1 || C % B || K < 1) return -2;
  RecurrenceArgs a{y, ldy, x, ldx, state, slots, cu_q, kv_lens, conv_w, conv_b, gates_b, rate, out, ldo, C, K, B};
  if (!tile_sizes(a, gates)) return -1;
#define KSANA_RS(TC, KT) launch_tile<TC, KT, true>(a, gates, seq_base, num_seqs, num_seqs, nullptr, nullptr, 0, st)
  // wide blocks: fewer CTAs load their gates (one CTA fills an SM's shared memory with them)
  const int rc = K > 4 ? KSANA_RS(RG_STEP, 8) : C / B > 128 ? KSANA_RS(2 * RG_STEP, 4) : KSANA_RS(RG_STEP, 4);
#undef KSANA_RS
  if (rc || C / B <= 128 || K == 1) return rc;
  recurrence_shift_kernel<<<dim3((C + 255) / 256, num_seqs), 256, 0, st>>>(a, seq_base);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

KSANA_API int ksana_recurrence_conv(const void* x, int ldx, const float* state, const int* slots, const int* cu_q,
                                    const int* kv_lens, const int* seq_of_token, const float* conv_w, const float* conv_b,
                                    int C, int K, void* u, int tok_base, int tokens, int kind, cudaStream_t st) {
  if (tokens <= 0) return 0;
  RecurrenceArgs a{nullptr, 0, x, ldx, const_cast<float*>(state), slots, cu_q, kv_lens, conv_w, conv_b, nullptr, nullptr,
                   nullptr, 0, C, K, 1};
  const dim3 grid((C + 255) / 256, tokens);
  if (kind)
    recurrence_conv_kernel<__nv_bfloat16><<<grid, 256, 0, st>>>(a, seq_of_token, static_cast<__nv_bfloat16*>(u), tok_base);
  else
    recurrence_conv_kernel<float><<<grid, 256, 0, st>>>(a, seq_of_token, static_cast<float*>(u), tok_base);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

// Sequences [seq_base, seq_base + num_seqs); u and z begin with token tok_base.
KSANA_API int ksana_recurrence_scan(const void* y, int ldy, const void* x, int ldx, float* state, const int* slots,
                                    const int* cu_q, const int* kv_lens, const void* u, const float* z,
                                    const float* gates_b, const float* rate, int C, int K, int B, void* out, int ldo,
                                    int seq_base, int num_seqs, int tok_base, int kind, cudaStream_t st) {
  if (num_seqs <= 0) return 0;
  if (B < 1 || C % B || K < 1) return -2;
  RecurrenceArgs a{y, ldy, x, ldx, state, slots, cu_q, kv_lens, nullptr, nullptr, gates_b, rate, out, ldo, C, K, B};
  const dim3 grid((C + 127) / 128, num_seqs);
  if (kind)
    recurrence_scan_kernel<__nv_bfloat16><<<grid, 128, 0, st>>>(a, static_cast<const __nv_bfloat16*>(u), z, seq_base, tok_base);
  else
    recurrence_scan_kernel<float><<<grid, 128, 0, st>>>(a, static_cast<const float*>(u), z, seq_base, tok_base);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}
