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

// sqrt(1 - a^2) and a itself from log a <= 0
__device__ __forceinline__ void decay_of(float la, float* a, float* in) {
  *a = expf(la);
  *in = sqrtf(-expm1f(2.f * la));
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
  const float* conv_w;     // [C, K]
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
    s = fmaf(a.conv_w[static_cast<size_t>(c) * a.K + j], v, s);
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
    float dec, in;
    decay_of(-sigmoid_f(zt[0] + br) * rate, &dec, &in);
    S = fmaf(dec, S, in * sigmoid_f(zt[part] + bi) * to_f(u[row * a.C + c]));
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

}  // namespace ksana

using namespace ksana;

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
