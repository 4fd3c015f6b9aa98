// Attention over the paged cache of layers with sizes of their own: a sliding window, a learned bias per distance, and
// key / value heads of different sizes. Scores, softmax and the accumulation are 32-bit.
//
// Cache of a layer: [block][keys hk x bs x d | values hk x bs x dv]. bias: [h][bias_len] fp32 (null: none), indexed by
// the distance between query and key.
#include "host_common.h"
#include "mixer_common.cuh"

namespace ksana {

struct WindowAttnArgs {
  const void* q;
  int ldq;
  const void* cache;
  const int* block_tables;
  int max_blocks;
  const int* cu_q;
  const int* kv_lens;
  const int* seq_of_token;
  int h, hk, d, dv, bs, window;
  float scale;
  const float* bias;
  int bias_len;
  float out_scale;
  void* out;
  int ldo;
};

// ---- any size, any storage type ---------------------------------------------------------------------------------
// One warp per (new token, head). Keys are taken 32 at a time, one per lane for the scores; for the weighted sum the
// lanes share out the value's columns (NV per lane).
template <typename T, int NV>
__global__ void __launch_bounds__(128)
window_attention_any_kernel(WindowAttnArgs a, int tok_base, int tokens) {
  extern __shared__ float sm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long unit = static_cast<long long>(blockIdx.x) * 4 + warp;
  if (unit >= static_cast<long long>(tokens) * a.h) return;
  const int t = tok_base + static_cast<int>(unit / a.h), head = static_cast<int>(unit % a.h);
  const int b = a.seq_of_token[t];
  const int pos = a.kv_lens[b] - a.cu_q[b + 1] + t;
  const int kh = head / (a.h / a.hk);
  float* sq = sm + warp * a.d;
  const T* q = static_cast<const T*>(a.q) + static_cast<size_t>(t) * a.ldq + head * a.d;
  for (int c = lane; c < a.d; c += 32) sq[c] = to_f(q[c]);
  __syncwarp();
  const int* bt = a.block_tables + static_cast<size_t>(b) * a.max_blocks;
  const T* cache = static_cast<const T*>(a.cache);
  const size_t block_elems = static_cast<size_t>(a.hk) * a.bs * (a.d + a.dv);
  const size_t v_off = static_cast<size_t>(a.hk) * a.bs * a.d;
  const float* bias = a.bias ? a.bias + static_cast<size_t>(head) * a.bias_len : nullptr;
  const int lo = a.window > 0 && pos - a.window + 1 > 0 ? pos - a.window + 1 : 0;
  float m = -INFINITY, l = 0.f, acc[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) acc[i] = 0.f;
  for (int j0 = lo; j0 <= pos; j0 += 32) {
    const int j = j0 + lane;
    float s = -INFINITY;
    if (j <= pos) {
      const T* kp = cache + bt[j / a.bs] * block_elems + (static_cast<size_t>(kh) * a.bs + j % a.bs) * a.d;
      float dot = 0.f;
      for (int c = 0; c < a.d; ++c) dot += sq[c] * to_f(kp[c]);
      s = dot * a.scale;
      if (bias) s += bias[min(pos - j, a.bias_len - 1)];
    }
    const float m_new = fmaxf(m, warp_max(s));
    const float f = expf(m - m_new);
    const float p = j <= pos ? expf(s - m_new) : 0.f;
    l = l * f + warp_sum(p);
    m = m_new;
#pragma unroll
    for (int i = 0; i < NV; ++i) acc[i] *= f;
    const int n = min(32, pos - j0 + 1);
    for (int u = 0; u < n; ++u) {
      const float pu = __shfl_sync(0xffffffffu, p, u);
      const int ju = j0 + u;
      const T* vp = cache + bt[ju / a.bs] * block_elems + v_off + (static_cast<size_t>(kh) * a.bs + ju % a.bs) * a.dv;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = i * 32 + lane;
        if (c < a.dv) acc[i] += pu * to_f(vp[c]);
      }
    }
  }
  T* o = static_cast<T*>(a.out) + static_cast<size_t>(t) * a.ldo + head * a.dv;
  const float inv = a.out_scale / l;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = i * 32 + lane;
    if (c < a.dv) o[c] = from_f<T>(acc[i] * inv);
  }
}

template <typename T>
static int launch_any(const WindowAttnArgs& a, int tok_base, int tokens, cudaStream_t st) {
  const long long units = static_cast<long long>(tokens) * a.h;
  const unsigned grid = static_cast<unsigned>((units + 3) / 4);
  const int smem = 4 * a.d * static_cast<int>(sizeof(float));
  if (smem > 48 * 1024) return -1;
  if (a.dv <= 64)
    window_attention_any_kernel<T, 2><<<grid, 128, smem, st>>>(a, tok_base, tokens);
  else if (a.dv <= 128)
    window_attention_any_kernel<T, 4><<<grid, 128, smem, st>>>(a, tok_base, tokens);
  else if (a.dv <= 256)
    window_attention_any_kernel<T, 8><<<grid, 128, smem, st>>>(a, tok_base, tokens);
  else if (a.dv <= 1024)
    window_attention_any_kernel<T, 32><<<grid, 128, smem, st>>>(a, tok_base, tokens);
  else
    return -1;
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

}  // namespace ksana

using namespace ksana;

// Tokens [tok_base, tok_base + tokens) of the step, whatever sequences they belong to. kind: 0 fp32, 1 bf16.
KSANA_API int ksana_window_attention_any(const void* q, int ldq, const void* cache, const int* block_tables,
                                         int max_blocks, const int* cu_q, const int* kv_lens, const int* seq_of_token,
                                         int h, int hk, int d, int dv, int bs, int window, float scale,
                                         const float* bias, int bias_len, float out_scale, void* out, int ldo,
                                         int tok_base, int tokens, int kind, cudaStream_t st) {
  if (tokens <= 0) return 0;
  if (h % hk) return -1;
  WindowAttnArgs a{q, ldq, cache, block_tables, max_blocks, cu_q, kv_lens, seq_of_token, h, hk, d, dv, bs, window, scale,
                   bias, bias_len, out_scale, out, ldo};
  return kind ? launch_any<__nv_bfloat16>(a, tok_base, tokens, st) : launch_any<float>(a, tok_base, tokens, st);
}
