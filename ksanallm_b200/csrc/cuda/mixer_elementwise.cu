// Bandwidth-bound steps of layers with mixers of their own sizes: LayerNorm over a 32-bit residual stream, embedding
// into that stream, GELU(gate) * up, per-head QK norm with the paged cache append, the gated RMS norm behind linear
// attention, and the logit soft cap. Everything is computed in 32-bit floats; T is the storage type of activations.
#include "host_common.h"
#include "mixer_common.cuh"

namespace ksana {

// ---- LayerNorm (+ residual add) -----------------------------------------------------------------------------
// residual (fp32 or T, may be null) += x; out = (r - mean) / sqrt(var + eps) * w (+ b). The row stays in registers:
// VPT groups of 4 per thread.
template <typename X, typename R, typename W, typename O, int VPT>
__global__ void __launch_bounds__(256)
layer_norm_kernel(const X* __restrict__ x, int ldx, R* __restrict__ residual, int ldr, const W* __restrict__ w,
                  const W* __restrict__ b, O* __restrict__ out, int ldo, int H, float eps) {
  __shared__ float red[32];
  const size_t row = blockIdx.x;
  float v[VPT][4];
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (i * 256 + threadIdx.x) * 4;
    if (c < H) {
      load_n<4>(x + row * ldx + c, v[i]);
      if (residual) {
        float r[4];
        load_n<4>(residual + row * ldr + c, r);
#pragma unroll
        for (int j = 0; j < 4; ++j) v[i][j] += r[j];
        store_n<4>(residual + row * ldr + c, v[i]);
        if constexpr (sizeof(R) == 2) {  // the norm sees what the stream keeps
#pragma unroll
          for (int j = 0; j < 4; ++j) v[i][j] = to_f(from_f<R>(v[i][j]));
        }
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) s += v[i][j];
    }
  }
  const float mean = block_sum(s, red) / static_cast<float>(H);
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    if ((i * 256 + threadIdx.x) * 4 < H) {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        v[i][j] -= mean;
        ss += v[i][j] * v[i][j];
      }
    }
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / static_cast<float>(H) + eps);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (i * 256 + threadIdx.x) * 4;
    if (c < H) {
      float g[4], o[4];
      load_n<4>(w + c, g);
#pragma unroll
      for (int j = 0; j < 4; ++j) o[j] = v[i][j] * inv * g[j];
      if (b) {
        load_n<4>(b + c, g);
#pragma unroll
        for (int j = 0; j < 4; ++j) o[j] += g[j];
      }
      store_n<4>(out + row * ldo + c, o);
    }
  }
}

// Any width and alignment: the row is read again for each of the three passes.
template <typename X, typename R, typename W, typename O>
__global__ void __launch_bounds__(256)
layer_norm_any_kernel(const X* __restrict__ x, int ldx, R* residual, int ldr, const W* __restrict__ w,
                      const W* __restrict__ b, O* __restrict__ out, int ldo, int H, float eps) {
  __shared__ float red[32];
  const size_t row = blockIdx.x;
  auto value = [&](int c) { return residual ? to_f(residual[row * ldr + c]) : to_f(x[row * ldx + c]); };
  float s = 0.f;
  for (int c = threadIdx.x; c < H; c += 256) {
    if (residual) residual[row * ldr + c] = from_f<R>(to_f(residual[row * ldr + c]) + to_f(x[row * ldx + c]));
    s += value(c);
  }
  const float mean = block_sum(s, red) / static_cast<float>(H);
  float ss = 0.f;
  for (int c = threadIdx.x; c < H; c += 256) {
    const float d = value(c) - mean;
    ss += d * d;
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / static_cast<float>(H) + eps);
  for (int c = threadIdx.x; c < H; c += 256) {
    float o = (value(c) - mean) * inv * to_f(w[c]);
    if (b) o += to_f(b[c]);
    out[row * ldo + c] = from_f<O>(o);
  }
}

template <typename X, typename R, typename W, typename O>
static int launch_layer_norm(const void* x, int ldx, void* residual, int ldr, const void* w, const void* b, void* out,
                             int ldo, int rows, int H, float eps, cudaStream_t st) {
  auto px = static_cast<const X*>(x);
  auto pr = static_cast<R*>(residual);
  auto pw = static_cast<const W*>(w), pb = static_cast<const W*>(b);
  auto po = static_cast<O*>(out);
  const bool vec = !((H | ldx | ldr | ldo) & 3) && H <= 8192;
#define KSANA_LN(V) layer_norm_kernel<X, R, W, O, V><<<rows, 256, 0, st>>>(px, ldx, pr, ldr, pw, pb, po, ldo, H, eps)
  if (!vec)
    layer_norm_any_kernel<X, R, W, O><<<rows, 256, 0, st>>>(px, ldx, pr, ldr, pw, pb, po, ldo, H, eps);
  else if (H <= 1024)
    KSANA_LN(1);
  else if (H <= 2048)
    KSANA_LN(2);
  else if (H <= 4096)
    KSANA_LN(4);
  else
    KSANA_LN(8);
#undef KSANA_LN
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

// ---- embedding into a 32-bit stream ---------------------------------------------------------------------------
template <typename T>
__global__ void embedding_f32_kernel(const int* __restrict__ ids, const T* __restrict__ table, float* __restrict__ out,
                                     int H, int vocab, float scale) {
  const size_t row = blockIdx.y;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= H) return;
  int id = ids[row];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  out[row * H + c] = to_f(table[static_cast<size_t>(id) * H + c]) * scale;
}

// ---- GELU(gate) * up --------------------------------------------------------------------------------------------
template <typename T, int N>
__global__ void gelu_mul_kernel(const T* __restrict__ x, int ldx, T* __restrict__ out, int ldo, int I) {
  const size_t row = blockIdx.y;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * N;
  if (c >= I) return;
  float g[N], u[N];
  load_n<N>(x + row * ldx + c, g);
  load_n<N>(x + row * ldx + I + c, u);
#pragma unroll
  for (int j = 0; j < N; ++j) g[j] = gelu_tanh_f(g[j]) * u[j];
  store_n<N>(out + row * ldo + c, g);
}

// ---- per-head QK norm + cache append ------------------------------------------------------------------------------
// One warp per (token, head): heads [0, h) are queries (normalised in place), the next hk keys (normalised into the
// cache), the last hk values (copied into the cache). Cache: [block][keys hk x bs x d | values hk x bs x dv].
template <typename T, int N>
__global__ void __launch_bounds__(256)
qk_norm_cache_kernel(T* __restrict__ q, int ldq, const T* __restrict__ k, int ldk, const T* __restrict__ v, int ldv,
                     const int* __restrict__ slots, T* __restrict__ cache, const float* __restrict__ qw,
                     const float* __restrict__ kw, float eps, int tokens, int h, int hk, int d, int dv, int bs) {
  const int heads = h + 2 * hk;
  const long long unit = static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (unit >= static_cast<long long>(tokens) * heads) return;
  const int t = static_cast<int>(unit / heads), hd = static_cast<int>(unit % heads);
  const T* src;
  T* dst;
  const float* w = nullptr;
  int n = d;
  if (hd < h) {
    dst = q + static_cast<size_t>(t) * ldq + hd * d;
    src = dst;
    w = qw;
    if (w == nullptr) return;
  } else {
    const int slot = slots[t];
    if (slot < 0) return;
    T* block = cache + static_cast<size_t>(slot / bs) * (static_cast<size_t>(hk) * bs * (d + dv));
    const int off = slot % bs;
    if (hd < h + hk) {
      const int kh = hd - h;
      src = k + static_cast<size_t>(t) * ldk + kh * d;
      dst = block + (static_cast<size_t>(kh) * bs + off) * d;
      w = kw;
    } else {
      const int kh = hd - h - hk;
      src = v + static_cast<size_t>(t) * ldv + kh * dv;
      dst = block + static_cast<size_t>(hk) * bs * d + (static_cast<size_t>(kh) * bs + off) * dv;
      n = dv;
    }
  }
  float f[N], inv = 1.f;
  if (w) {
    float ss = 0.f;
    for (int c = lane * N; c < n; c += 32 * N) {
      load_n<N>(src + c, f);
#pragma unroll
      for (int j = 0; j < N; ++j) ss += f[j] * f[j];
    }
    inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(n) + eps);
  }
  for (int c = lane * N; c < n; c += 32 * N) {
    load_n<N>(src + c, f);
    if (w) {
#pragma unroll
      for (int j = 0; j < N; ++j) f[j] = f[j] * inv * w[c + j];
    }
    store_n<N>(dst + c, f);
  }
}

// ---- gated RMS norm behind linear attention -------------------------------------------------------------------------
template <typename T>
__device__ __forceinline__ float gate_f(float g, int kind) {
  if (sizeof(T) == 2) {
    const float s = __fdividef(1.f, 1.f + __expf(-g));
    return kind == 0 ? g * s : s;
  }
  return kind == 0 ? silu_f(g) : sigmoid_f(g);
}

// per head, no weight: a warp takes HEADS heads of a token at a time, up to 32 N columns each in registers
template <typename T, int N, int HEADS>
__global__ void __launch_bounds__(256)
gated_head_norm_kernel(const T* __restrict__ o, const T* __restrict__ g, int ldg, T* __restrict__ out, int ldo,
                       int tokens, int h, int dv, float eps, int gate, float out_scale) {
  const int groups = (h + HEADS - 1) / HEADS;
  const long long unit = static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (unit >= static_cast<long long>(tokens) * groups) return;
  const size_t t = unit / groups;
  const int h0 = static_cast<int>(unit % groups) * HEADS;
  if (dv <= 32 * N) {
    float f[HEADS][N], gg[HEADS][N];
    const int c = lane * N;
#pragma unroll
    for (int i = 0; i < HEADS; ++i) {
#pragma unroll
      for (int j = 0; j < N; ++j) f[i][j] = gg[i][j] = 0.f;
      if (h0 + i < h && c < dv) {
        load_n<N>(o + (t * h + h0 + i) * dv + c, f[i]);
        load_n<N>(g + t * ldg + (h0 + i) * dv + c, gg[i]);
      }
    }
#pragma unroll
    for (int i = 0; i < HEADS; ++i) {
      float ss = 0.f;
#pragma unroll
      for (int j = 0; j < N; ++j) ss += f[i][j] * f[i][j];
      const float inv = out_scale / sqrtf(warp_sum(ss) / static_cast<float>(dv) + eps);
#pragma unroll
      for (int j = 0; j < N; ++j) f[i][j] *= inv * gate_f<T>(gg[i][j], gate);
      if (h0 + i < h && c < dv) store_n<N>(out + t * ldo + (h0 + i) * dv + c, f[i]);
    }
    return;
  }
  for (int hd = h0; hd < min(h0 + HEADS, h); ++hd) {
    const T* src = o + (t * h + hd) * dv;
    float f[N], gg[N], ss = 0.f;
    for (int c = lane * N; c < dv; c += 32 * N) {
      load_n<N>(src + c, f);
#pragma unroll
      for (int j = 0; j < N; ++j) ss += f[j] * f[j];
    }
    const float inv = out_scale / sqrtf(warp_sum(ss) / static_cast<float>(dv) + eps);
    for (int c = lane * N; c < dv; c += 32 * N) {
      load_n<N>(src + c, f);
      load_n<N>(g + t * ldg + hd * dv + c, gg);
#pragma unroll
      for (int j = 0; j < N; ++j) f[j] *= inv * gate_f<T>(gg[j], gate);
      store_n<N>(out + t * ldo + hd * dv + c, f);
    }
  }
}

// over all heads of a token, with a weight: one CTA per token
template <typename T, int N>
__global__ void __launch_bounds__(256)
gated_row_norm_kernel(const T* __restrict__ o, const T* __restrict__ g, int ldg, const float* __restrict__ w,
                      T* __restrict__ out, int ldo, int width, float eps, int gate, float out_scale) {
  __shared__ float red[32];
  const size_t t = blockIdx.x;
  float f[N], gg[N], ss = 0.f;
  for (int c = threadIdx.x * N; c < width; c += 256 * N) {
    load_n<N>(o + t * width + c, f);
#pragma unroll
    for (int j = 0; j < N; ++j) ss += f[j] * f[j];
  }
  const float inv = out_scale / sqrtf(block_sum(ss, red) / static_cast<float>(width) + eps);
  for (int c = threadIdx.x * N; c < width; c += 256 * N) {
    load_n<N>(o + t * width + c, f);
    load_n<N>(g + t * ldg + c, gg);
#pragma unroll
    for (int j = 0; j < N; ++j) f[j] = f[j] * inv * w[c + j] * gate_f<T>(gg[j], gate);
    store_n<N>(out + t * ldo + c, f);
  }
}

// ---- logit soft cap ---------------------------------------------------------------------------------------------------
__global__ void softcap_kernel(const float* __restrict__ x, int ldx, float* __restrict__ out, int n, float cap) {
  const size_t row = blockIdx.y;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c < n) out[row * n + c] = cap * tanhf(x[row * ldx + c] / cap);
}

static bool aligned(const void* p, int bytes) { return (reinterpret_cast<uintptr_t>(p) & (bytes - 1)) == 0; }
static int done() { return cudaGetLastError() == cudaSuccess ? 0 : -5; }

}  // namespace ksana

using namespace ksana;
using bf16 = __nv_bfloat16;

// Storage types: 0 = fp32, 1 = bf16. `kinds` = x | residual << 1 | weight << 2 | out << 3. Row pitches in elements.
KSANA_API int ksana_layer_norm(const void* x, int ldx, void* residual, int ldr, const void* w, const void* b, void* out,
                               int ldo, int rows, int H, float eps, int kinds, cudaStream_t st) {
  if (rows <= 0 || H <= 0) return 0;
#define KSANA_LN_CASE(K, X, R, W, O) \
  case K: return launch_layer_norm<X, R, W, O>(x, ldx, residual, ldr, w, b, out, ldo, rows, H, eps, st)
  switch (kinds) {
    KSANA_LN_CASE(0, float, float, float, float);
    KSANA_LN_CASE(12, float, float, bf16, bf16);  // first norm of a bf16 model over its 32-bit stream
    KSANA_LN_CASE(13, bf16, float, bf16, bf16);   // sublayer output into the 32-bit stream
    KSANA_LN_CASE(15, bf16, bf16, bf16, bf16);
    default: return -1;
  }
#undef KSANA_LN_CASE
}

KSANA_API int ksana_embedding_f32(const int* ids, const void* table, float* out, int rows, int H, int vocab, float scale,
                                  int kind, cudaStream_t st) {
  if (rows <= 0) return 0;
  dim3 grid((H + 255) / 256, rows);
  if (kind)
    embedding_f32_kernel<<<grid, 256, 0, st>>>(ids, static_cast<const bf16*>(table), out, H, vocab, scale);
  else
    embedding_f32_kernel<<<grid, 256, 0, st>>>(ids, static_cast<const float*>(table), out, H, vocab, scale);
  return done();
}

KSANA_API int ksana_gelu_mul(const void* x, int ldx, void* out, int ldo, int rows, int I, int kind, cudaStream_t st) {
  if (rows <= 0) return 0;
  const bool vec = !((I | ldx | ldo) & 7) && aligned(x, 16) && aligned(out, 16);
#define KSANA_GELU(T, N)                                                                                   \
  gelu_mul_kernel<T, N><<<dim3((I / N + 255) / 256 + (I % N ? 1 : 0), rows), 256, 0, st>>>(                \
      static_cast<const T*>(x), ldx, static_cast<T*>(out), ldo, I)
  if (kind) {
    if (vec) KSANA_GELU(bf16, 8); else KSANA_GELU(bf16, 1);
  } else {
    if (vec) KSANA_GELU(float, 8); else KSANA_GELU(float, 1);
  }
#undef KSANA_GELU
  return done();
}

KSANA_API int ksana_qk_norm_cache(void* q, int ldq, const void* k, int ldk, const void* v, int ldv, const int* slots,
                                  void* cache, const float* qw, const float* kw, float eps, int tokens, int h, int hk,
                                  int d, int dv, int bs, int kind, cudaStream_t st) {
  if (tokens <= 0) return 0;
  const int esz = kind ? 2 : 4;
  const bool vec = !((ldq | ldk | ldv | d | dv) & 3) && aligned(q, 4 * esz) && aligned(k, 4 * esz) &&
                   aligned(v, 4 * esz) && aligned(cache, 4 * esz);
  const long long units = static_cast<long long>(tokens) * (h + 2 * hk);
  const unsigned grid = static_cast<unsigned>((units + 7) / 8);
#define KSANA_QK(T, N)                                                                                              \
  qk_norm_cache_kernel<T, N><<<grid, 256, 0, st>>>(static_cast<T*>(q), ldq, static_cast<const T*>(k), ldk,          \
                                                   static_cast<const T*>(v), ldv, slots, static_cast<T*>(cache), qw, \
                                                   kw, eps, tokens, h, hk, d, dv, bs)
  if (kind) {
    if (vec) KSANA_QK(bf16, 4); else KSANA_QK(bf16, 1);
  } else {
    if (vec) KSANA_QK(float, 4); else KSANA_QK(float, 1);
  }
#undef KSANA_QK
  return done();
}

// gate: 0 silu, 1 sigmoid. w == nullptr: per head, no weight. o is [tokens, h, dv] contiguous.
KSANA_API int ksana_gated_norm(const void* o, const void* g, int ldg, const float* w, void* out, int ldo, int tokens,
                               int h, int dv, float eps, int gate, float out_scale, int kind, cudaStream_t st) {
  if (tokens <= 0) return 0;
  const int esz = kind ? 2 : 4;
  const int width = h * dv;
  const bool vec = !((dv | ldg | ldo) & 3) && aligned(o, 4 * esz) && aligned(g, 4 * esz) && aligned(out, 4 * esz);
  const bool wide = kind && !w && dv > 128 && !((dv | ldg | ldo) & 7) && aligned(o, 16) && aligned(g, 16) && aligned(out, 16);
  const unsigned grid = static_cast<unsigned>((static_cast<long long>(tokens) * ((h + 3) / 4) + 7) / 8);
#define KSANA_GN(T, N)                                                                                               \
  do {                                                                                                               \
    if (w)                                                                                                           \
      gated_row_norm_kernel<T, N><<<tokens, 256, 0, st>>>(static_cast<const T*>(o), static_cast<const T*>(g), ldg, w, \
                                                          static_cast<T*>(out), ldo, width, eps, gate, out_scale);   \
    else                                                                                                             \
      gated_head_norm_kernel<T, N, 4><<<grid, 256, 0, st>>>(static_cast<const T*>(o), static_cast<const T*>(g), ldg,    \
                                                         static_cast<T*>(out), ldo, tokens, h, dv, eps, gate,        \
                                                         out_scale);                                                 \
  } while (0)
  if (kind) {
    if (wide) KSANA_GN(bf16, 8); else if (vec) KSANA_GN(bf16, 4); else KSANA_GN(bf16, 1);
  } else {
    if (vec) KSANA_GN(float, 4); else KSANA_GN(float, 1);
  }
#undef KSANA_GN
  return done();
}

KSANA_API int ksana_softcap(const float* x, int ldx, float* out, int rows, int n, float cap, cudaStream_t st) {
  if (rows <= 0) return 0;
  softcap_kernel<<<dim3((n + 255) / 256, rows), 256, 0, st>>>(x, ldx, out, n, cap);
  return done();
}
