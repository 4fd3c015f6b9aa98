// Attention over the paged cache whose softmax weights are mixed across heads before the values are summed up:
//   p_g(i, j) = exp(q_ig . k_j scale) / (sum over keys of the same + exp(sink_g)),
//   o_ih = sum_j (sum_g talk[h][g] p_g(i, j)) v_j,
// each head with the keys and values of its own key / value head, times the sigmoid of a gate per output. Scores, softmax,
// mix and sums are 32-bit. Cache of a layer: [block][keys hk x bs x d | values hk x bs x dv]. Query i sees every j <= i.
#include "talking.cuh"

namespace ksana {

// ---- any size, any storage type -----------------------------------------------------------------------------------------
// One CTA per new token, in two passes over its keys, 32 at a time: every head's maximum and sum, then the weights again,
// mixed, and the values. A warp scores one head at a time, a key per lane. With gridDim.y > 1 the output heads are shared out.
template <typename T>
__global__ void __launch_bounds__(256)
talking_any_kernel(TalkArgs a, int tok_base, int heads_per) {
  extern __shared__ float sm[];
  const int t = tok_base + blockIdx.x, h = a.h, d = a.d, dv = a.dv;
  const int h0 = blockIdx.y * heads_per, hn = min(heads_per, h - h0);
  float* sq = sm;                 // [h][d]
  float* sm_m = sq + h * d;       // [h]: maximum, then the logarithm of the whole sum
  float* sm_l = sm_m + h;         // [h]
  float* sp = sm_l + h;           // [h][33]
  float* sw = sp + h * 33;        // [hn][33]
  float* so = sw + heads_per * 33;  // [hn][dv]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int b = a.seq_of_token[t];
  const int n = a.kv_lens[b] - a.cu_q[b + 1] + t + 1;  // visible keys
  const int group = h / a.hk;
  const int* bt = a.block_tables + static_cast<size_t>(b) * a.max_blocks;
  const T* cache = static_cast<const T*>(a.cache);
  const T* q = static_cast<const T*>(a.q) + static_cast<size_t>(t) * a.ldq;
  for (int c = tid; c < h * d; c += 256) sq[c] = to_f(q[c]);
  for (int c = tid; c < hn * dv; c += 256) so[c] = 0.f;
  for (int c = tid; c < h; c += 256) {
    sm_m[c] = a.sink[c];
    sm_l[c] = 1.f;
  }
  __syncthreads();
  auto score = [&](int g, int j) {
    const T* kp = cache + bt[j / a.bs] * a.block_elems() + (static_cast<size_t>(g / group) * a.bs + j % a.bs) * d;
    const float* x = sq + g * d;
    float dot[4] = {0.f, 0.f, 0.f, 0.f};
    int c = 0;
    for (; c + 4 <= d; c += 4)
#pragma unroll
      for (int u = 0; u < 4; ++u) dot[u] = fmaf(x[c + u], to_f(kp[c + u]), dot[u]);
    for (; c < d; ++c) dot[0] = fmaf(x[c], to_f(kp[c]), dot[0]);
    return ((dot[0] + dot[1]) + (dot[2] + dot[3])) * a.scale;
  };
  for (int g = warp; g < h; g += 8) {
    float m = sm_m[g], l = 1.f;
    for (int j0 = 0; j0 < n; j0 += 32) {
      const float s = j0 + lane < n ? score(g, j0 + lane) : -INFINITY;
      const float m_new = fmaxf(m, warp_max(s));
      l = l * expf(m - m_new) + warp_sum(j0 + lane < n ? expf(s - m_new) : 0.f);
      m = m_new;
    }
    __syncwarp();
    if (lane == 0) {
      sm_m[g] = m;
      sm_l[g] = 1.f / l;
    }
  }
  __syncthreads();
  for (int j0 = 0; j0 < n; j0 += 32) {
    for (int g = warp; g < h; g += 8)
      sp[g * 33 + lane] = j0 + lane < n ? expf(score(g, j0 + lane) - sm_m[g]) * sm_l[g] : 0.f;
    __syncthreads();
    for (int i = tid; i < hn * 32; i += 256) {
      const int to = i >> 5, key = i & 31;
      const float* row = a.talk + static_cast<size_t>(h0 + to) * h;
      float w = 0.f;
      for (int g = 0; g < h; ++g) w = fmaf(row[g], sp[g * 33 + key], w);
      sw[to * 33 + key] = w;
    }
    __syncthreads();
    const int count = min(32, n - j0);
    for (int i = tid; i < hn * dv; i += 256) {
      const int to = i / dv, c = i % dv;
      float part = 0.f;
      for (int u = 0; u < count; ++u) {
        const int j = j0 + u;
        const T* vp = cache + bt[j / a.bs] * a.block_elems() + a.v_off() +
                      (static_cast<size_t>((h0 + to) / group) * a.bs + j % a.bs) * dv;
        part = fmaf(sw[to * 33 + u], to_f(vp[c]), part);
      }
      so[i] += part;
    }
    // (the next round writes sp, which nobody reads any more, and sw only behind its first barrier)
  }
  __syncthreads();
  T* o = static_cast<T*>(a.out) + static_cast<size_t>(t) * a.ldo + h0 * dv;
  const T* gate = a.gate ? static_cast<const T*>(a.gate) + static_cast<size_t>(t) * a.ldg + h0 * dv : nullptr;
  for (int i = tid; i < hn * dv; i += 256)
    o[i] = from_f<T>(so[i] * a.out_scale * (gate ? sigmoid_f(to_f(gate[i])) : 1.f));
}

template <typename T>
static int launch_any(const TalkArgs& a, int tok_base, int tokens, cudaStream_t st) {
  auto bytes = [&](int per) { return 4 * (a.h * (a.d + 2 + 33) + per * (33 + a.dv)); };
  int parts = 1;
  while (parts < a.h && bytes((a.h + parts - 1) / parts) > 200 * 1024) ++parts;
  const int per = (a.h + parts - 1) / parts;
  if (bytes(per) > 227 * 1024) return -1;
  auto kern = talking_any_kernel<T>;
  if (bytes(per) > 48 * 1024 && KSANA_SMEM_ONCE(kern, 227 * 1024) != 0) return -4;
  kern<<<dim3(tokens, (a.h + per - 1) / per), 256, bytes(per), st>>>(a, tok_base, per);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

}  // namespace ksana

using namespace ksana;

// Tokens [tok_base, tok_base + tokens) of the step, whatever sequences they belong to. kind: 0 fp32, 1 bf16.
KSANA_API int ksana_talking_any(const void* q, int ldq, const void* cache, const int* block_tables, int max_blocks,
                                const int* cu_q, const int* kv_lens, const int* seq_of_token, int h, int hk, int d, int dv,
                                int bs, float scale, const float* sink, const float* talk, float out_scale,
                                const void* gate, int ldg, void* out, int ldo, int tok_base, int tokens, int kind,
                                cudaStream_t st) {
  if (tokens <= 0) return 0;
  if (h % hk) return -2;
  TalkArgs a{q, ldq, cache, block_tables, max_blocks, cu_q, kv_lens, seq_of_token, h, hk, d, dv, bs, scale, sink, talk,
             out_scale, gate, ldg, out, ldo};
  return kind ? launch_any<__nv_bfloat16>(a, tok_base, tokens, st) : launch_any<float>(a, tok_base, tokens, st);
}
