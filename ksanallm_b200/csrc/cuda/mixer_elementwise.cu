// Bandwidth-bound steps of layers with mixers of their own sizes: norms over a 32-bit residual stream (which may take gated
// sublayers), embedding into that stream, GELU (gated or not), squared ReLU and clamped gates, the paged cache append (with
// QK norm per head or per row and rotation, or beside the activation), the gated RMS norm behind linear attention, and the
// logit soft cap. Everything is computed in 32-bit floats; T is the storage type of activations.
#include "host_common.h"
#include "mixer_common.cuh"

namespace ksana {

// ---- the stream and its norms -----------------------------------------------------------------------------------
// A row of the stream (R) takes what a sublayer hands over and is normalised for the next one:
//   v = res_in + (x + sum_j weights[t, j] y[pos[t, j]]) + add_rows + add_vec;  res_out = v
//   out = v / sqrt(mean(v^2) + eps) * w                        (center 0)
//   out = (v - mean(v)) / sqrt(var(v) + eps) * w (+ b)         (center 1)
// Every term may be absent (null). y holds the rows of routed experts in sorted order (pos -1: another rank's expert).
template <typename X, typename R, typename W, typename O>
struct StreamNormArgs {
  const X* x;
  int ldx;
  const R* res_in;
  R* res_out;
  int ldr;
  const W* w;
  const W* b;
  O* out;
  int ldo, H;
  float eps;
  int center;
  const float* add_rows;  // [rows, H]
  const float* add_vec;   // [H]
  const X* y;             // [n, H]
  const int* pos;
  const float* weights;
  int k;

  // V groups of N columns of the new stream value of `row`, `step` columns apart. Each term is loaded for all groups at
  // once, so that its loads are in flight together.
  template <int N, int V>
  __device__ void value(size_t row, int c0, int step, float (*v)[N]) const {
#pragma unroll
    for (int i = 0; i < V; ++i)
#pragma unroll
      for (int j = 0; j < N; ++j) v[i][j] = 0.f;
    auto add = [&](const auto* p, float w) {
      float f[V][N];
#pragma unroll
      for (int i = 0; i < V; ++i)
        if (c0 + i * step < H) load_n<N>(p + c0 + i * step, f[i]);
#pragma unroll
      for (int i = 0; i < V; ++i)
        if (c0 + i * step < H)
#pragma unroll
          for (int j = 0; j < N; ++j) v[i][j] = fmaf(w, f[i][j], v[i][j]);
    };
    if (x) add(x + row * ldx, 1.f);
    for (int e = 0; e < k; ++e) {
      const int p = pos[row * k + e];
      if (p >= 0) add(y + static_cast<size_t>(p) * H, weights[row * k + e]);
    }
    if (res_in) add(res_in + row * ldr, 1.f);
    if (add_rows) add(add_rows + row * H, 1.f);
    if (add_vec) add(add_vec, 1.f);
  }
  template <int N>
  __device__ void keep(size_t row, int c, float* v) const {
    if (res_out) {
      store_n<N>(res_out + row * ldr + c, v);
      if constexpr (sizeof(R) == 2) {  // the norm sees what the stream keeps
#pragma unroll
        for (int j = 0; j < N; ++j) v[j] = to_f(from_f<R>(v[j]));
      }
    }
  }
};

// The row stays in registers: VPT groups of 4 per thread.
template <typename X, typename R, typename W, typename O, int VPT>
__global__ void __launch_bounds__(256)
stream_norm_kernel(const StreamNormArgs<X, R, W, O> a) {
  __shared__ float red[32];
  const size_t row = blockIdx.x;
  const int H = a.H;
  float v[VPT][4];
  float s = 0.f;
  a.template value<4, VPT>(row, threadIdx.x * 4, 1024, v);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (i * 256 + threadIdx.x) * 4;
    if (c < H) {
      a.template keep<4>(row, c, v[i]);
#pragma unroll
      for (int j = 0; j < 4; ++j) s += v[i][j];
    }
  }
  const float mean = a.center ? block_sum(s, red) / static_cast<float>(H) : 0.f;
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
  const float inv = 1.f / sqrtf(block_sum(ss, red) / static_cast<float>(H) + a.eps);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (i * 256 + threadIdx.x) * 4;
    if (c < H) {
      float g[4], o[4];
      load_n<4>(a.w + c, g);
#pragma unroll
      for (int j = 0; j < 4; ++j) o[j] = v[i][j] * inv * g[j];
      if (a.b) {
        load_n<4>(a.b + c, g);
#pragma unroll
        for (int j = 0; j < 4; ++j) o[j] += g[j];
      }
      store_n<4>(a.out + row * a.ldo + c, o);
    }
  }
}

// Any width and alignment: the row's new value stays in shared memory.
template <typename X, typename R, typename W, typename O>
__global__ void __launch_bounds__(256)
stream_norm_any_kernel(const StreamNormArgs<X, R, W, O> a) {
  extern __shared__ float row_v[];
  __shared__ float red[32];
  const size_t row = blockIdx.x;
  const int H = a.H;
  float s = 0.f;
  for (int c = threadIdx.x; c < H; c += 256) {
    float v[1][1];
    a.template value<1, 1>(row, c, 0, v);
    a.template keep<1>(row, c, v[0]);
    row_v[c] = v[0][0];  // only this thread reads it back
    s += v[0][0];
  }
  const float mean = a.center ? block_sum(s, red) / static_cast<float>(H) : 0.f;
  float ss = 0.f;
  for (int c = threadIdx.x; c < H; c += 256) {
    const float d = row_v[c] - mean;
    ss += d * d;
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / static_cast<float>(H) + a.eps);
  for (int c = threadIdx.x; c < H; c += 256) {
    float o = (row_v[c] - mean) * inv * to_f(a.w[c]);
    if (a.b) o += to_f(a.b[c]);
    a.out[row * a.ldo + c] = from_f<O>(o);
  }
}

template <typename X, typename R, typename W, typename O>
static int launch_stream_norm(const void* x, int ldx, const void* res_in, void* res_out, int ldr, const void* w,
                              const void* b, void* out, int ldo, int rows, int H, float eps, int center,
                              const float* add_rows, const float* add_vec, const void* y, const int* pos,
                              const float* weights, int k, cudaStream_t st) {
  const StreamNormArgs<X, R, W, O> a{static_cast<const X*>(x), ldx, static_cast<const R*>(res_in),
                                     static_cast<R*>(res_out), ldr, static_cast<const W*>(w), static_cast<const W*>(b),
                                     static_cast<O*>(out), ldo, H, eps, center, add_rows, add_vec,
                                     static_cast<const X*>(y), pos, weights, y ? k : 0};
  const bool vec = !((H | ldx | ldr | ldo) & 3) && H <= 8192;
#define KSANA_SN(V) stream_norm_kernel<X, R, W, O, V><<<rows, 256, 0, st>>>(a)
  if (!vec) {
    if (H > 50 * 1024) return -1;
    auto kern = stream_norm_any_kernel<X, R, W, O>;
    if (H * 4 > 47 * 1024 && KSANA_SMEM_ONCE(kern, 200 * 1024) != 0) return -4;
    kern<<<rows, 256, H * 4, st>>>(a);
  } else if (H <= 1024) {
    KSANA_SN(1);
  } else if (H <= 2048) {
    KSANA_SN(2);
  } else if (H <= 4096) {
    KSANA_SN(4);
  } else {
    KSANA_SN(8);
  }
#undef KSANA_SN
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

// ---- gated sublayers into the stream ------------------------------------------------------------------------------
// v = in + scale (x sig(xg) + (sum_j weights[t, j] rows[pos[t, j]] + y sig(ys[t])) sig(yg));  stream = v
// out[n] = v / sqrt(mean(v^2) + eps) * w[n] for up to two weights. Every term may be absent (null).
template <typename T>
__device__ __forceinline__ float sigmoid_as(float x) {
  if constexpr (sizeof(T) == 2) return __fdividef(1.f, 1.f + __expf(-x));
  return sigmoid_f(x);
}

template <typename T>
struct GatedNormArgs {
  const T *x, *xg, *rows, *y, *yg;
  int ldx, ldxg, ldy, ldyg, ldys, k, H, norms;
  const int* pos;
  const float *weights, *ys;
  float scale, eps;
  const float* in;  // [rows, H]
  float* stream;    // [rows, H] (in itself is fine; null: nowhere)
  const T* w[2];
  T* out;           // [norms][tokens][H]
  size_t plane;     // tokens * H

  template <int N, int V>
  __device__ void value(size_t row, int c0, int step, float (*v)[N]) const {
    auto load = [&](const auto* p, float (*f)[N]) {
#pragma unroll
      for (int i = 0; i < V; ++i)
        if (c0 + i * step < H) load_n<N>(p + c0 + i * step, f[i]);
    };
    float a[V][N], b[V][N];
#pragma unroll
    for (int i = 0; i < V; ++i)
#pragma unroll
      for (int j = 0; j < N; ++j) v[i][j] = a[i][j] = b[i][j] = 0.f;
    if (y) {
      load(y + row * ldy, a);
      load(yg + row * ldyg, b);
      const float s = sigmoid_as<T>(ys[row * ldys]);
#pragma unroll
      for (int i = 0; i < V; ++i)
#pragma unroll
        for (int j = 0; j < N; ++j) v[i][j] = a[i][j] * s;
      for (int e = 0; e < k; ++e) {
        const int p = pos[row * k + e];
        if (p < 0) continue;
        const float we = weights[row * k + e];
        load(rows + static_cast<size_t>(p) * H, a);
#pragma unroll
        for (int i = 0; i < V; ++i)
#pragma unroll
          for (int j = 0; j < N; ++j) v[i][j] = fmaf(we, a[i][j], v[i][j]);
      }
#pragma unroll
      for (int i = 0; i < V; ++i)
#pragma unroll
        for (int j = 0; j < N; ++j) v[i][j] *= sigmoid_as<T>(b[i][j]);
    }
    if (x) {
      load(x + row * ldx, a);
      load(xg + row * ldxg, b);
#pragma unroll
      for (int i = 0; i < V; ++i)
#pragma unroll
        for (int j = 0; j < N; ++j) v[i][j] = fmaf(a[i][j], sigmoid_as<T>(b[i][j]), v[i][j]);
    }
    load(in + row * H, a);
#pragma unroll
    for (int i = 0; i < V; ++i)
#pragma unroll
      for (int j = 0; j < N; ++j) v[i][j] = fmaf(scale, v[i][j], a[i][j]);
  }
};

template <typename T, int VPT>
__global__ void __launch_bounds__(256)
gated_stream_norm_kernel(const GatedNormArgs<T> a) {
  __shared__ float red[32];
  const size_t row = blockIdx.x;
  const int H = a.H;
  float v[VPT][4], ss = 0.f;
  a.template value<4, VPT>(row, threadIdx.x * 4, 1024, v);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (i * 256 + threadIdx.x) * 4;
    if (c < H) {
      if (a.stream) store_n<4>(a.stream + row * H + c, v[i]);
#pragma unroll
      for (int j = 0; j < 4; ++j) ss += v[i][j] * v[i][j];
    }
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / static_cast<float>(H) + a.eps);
  for (int n = 0; n < a.norms; ++n) {
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (i * 256 + threadIdx.x) * 4;
      if (c < H) {
        float g[4];
        load_n<4>(a.w[n] + c, g);
#pragma unroll
        for (int j = 0; j < 4; ++j) g[j] *= v[i][j] * inv;
        store_n<4>(a.out + n * a.plane + row * H + c, g);
      }
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
gated_stream_norm_any_kernel(const GatedNormArgs<T> a) {
  extern __shared__ float row_v[];
  __shared__ float red[32];
  const size_t row = blockIdx.x;
  const int H = a.H;
  float ss = 0.f;
  for (int c = threadIdx.x; c < H; c += 256) {
    float v[1][1];
    a.template value<1, 1>(row, c, 0, v);
    if (a.stream) a.stream[row * H + c] = v[0][0];
    row_v[c] = v[0][0];  // only this thread reads it back
    ss += v[0][0] * v[0][0];
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / static_cast<float>(H) + a.eps);
  for (int n = 0; n < a.norms; ++n)
    for (int c = threadIdx.x; c < H; c += 256)
      a.out[n * a.plane + row * H + c] = from_f<T>(row_v[c] * inv * to_f(a.w[n][c]));
}

template <typename T>
static int launch_gated_norm(const GatedNormArgs<T>& a, int rows, cudaStream_t st) {
  auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & (4 * sizeof(T) - 1)) == 0; };
  const int H = a.H;
  const bool vec = !((H | a.ldx | a.ldxg | a.ldy | a.ldyg) & 3) && H <= 8192 && al(a.x) && al(a.xg) && al(a.y) && al(a.yg) &&
                   al(a.rows) && al(a.out) && al(a.w[0]) && al(a.w[1]);
#define KSANA_GSN(V) gated_stream_norm_kernel<T, V><<<rows, 256, 0, st>>>(a)
  if (!vec) {
    if (H > 50 * 1024) return -1;
    auto kern = gated_stream_norm_any_kernel<T>;
    if (H * 4 > 47 * 1024 && KSANA_SMEM_ONCE(kern, 200 * 1024) != 0) return -4;
    kern<<<rows, 256, H * 4, st>>>(a);
  } else if (H <= 1024) {
    KSANA_GSN(1);
  } else if (H <= 2048) {
    KSANA_GSN(2);
  } else if (H <= 4096) {
    KSANA_GSN(4);
  } else {
    KSANA_GSN(8);
  }
#undef KSANA_GSN
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

// ---- embedding into a 32-bit stream ---------------------------------------------------------------------------
// out = table[id] * scale (+ pos_table[position], unscaled)
template <typename T>
__global__ void embedding_f32_kernel(const int* __restrict__ ids, const T* __restrict__ table, float* __restrict__ out,
                                     int H, int vocab, float scale, const int* __restrict__ positions,
                                     const T* __restrict__ pos_table, int pos_rows) {
  const size_t row = blockIdx.y;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= H) return;
  const int id = min(max(ids[row], 0), vocab - 1);
  float v = to_f(table[static_cast<size_t>(id) * H + c]) * scale;
  if (pos_table) v += to_f(pos_table[static_cast<size_t>(min(max(positions[row], 0), pos_rows - 1)) * H + c]);
  out[row * H + c] = v;
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
  for (int j = 0; j < N; ++j) g[j] = gelu_tanh_as<T>(g[j]) * u[j];
  store_n<N>(out + row * ldo + c, g);
}

// ---- squared ReLU; gate and up clamped -------------------------------------------------------------------------------
template <typename T, int N>
__global__ void relu2_kernel(const T* __restrict__ x, int ldx, T* __restrict__ out, int cols, size_t n) {
  const size_t i = (static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x) * N;
  if (i >= n) return;
  float f[N];
  load_n<N>(ldx == cols ? x + i : x + i / cols * ldx + i % cols, f);
#pragma unroll
  for (int j = 0; j < N; ++j) f[j] = fmaxf(f[j], 0.f) * fmaxf(f[j], 0.f);
  store_n<N>(out + i, f);
}

// out = g sigmoid(alpha g) (u + 1) with g = min(gate, limit), u = up clamped to +-limit, over rows [gate | up]
template <typename T, int N>
__global__ void clamped_gate_mul_kernel(const T* __restrict__ x, T* __restrict__ out, int I, float limit, float alpha) {
  const size_t row = blockIdx.x;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * N;
  if (c >= I) return;
  float g[N], u[N];
  load_n<N>(x + row * 2 * I + c, g);
  load_n<N>(x + row * 2 * I + I + c, u);
#pragma unroll
  for (int j = 0; j < N; ++j) {
    g[j] = fminf(g[j], limit);
    const float s = sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(-alpha * g[j])) : sigmoid_f(alpha * g[j]);
    g[j] *= s * (fminf(fmaxf(u[j], -limit), limit) + 1.f);
  }
  store_n<N>(out + row * I + c, g);
}

// ---- per-head QK norm, rotation, cache append -----------------------------------------------------------------------
// One warp per (token, head): heads [0, h) are queries (in place; h is 0 when nothing happens to them), the next hk keys
// (into the cache), the last hk values (copied into the cache). Queries and keys are normalised where there is a weight,
// then the pairs (2i, 2i + 1) of their first rd dimensions are rotated where there is a table. Cache: [block][keys hk x bs
// x d | values hk x bs x dv].
template <typename T, int N>
__global__ void __launch_bounds__(256)
qk_norm_cache_kernel(T* __restrict__ q, int ldq, const T* __restrict__ k, int ldk, const T* __restrict__ v, int ldv,
                     const int* __restrict__ slots, T* __restrict__ cache, const float* __restrict__ qw,
                     const float* __restrict__ kw, float eps, const int* __restrict__ positions,
                     const float* __restrict__ rotary, int rd, int tokens, int h, int hk, int d, int dv, int bs) {
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
  const bool turn = rotary != nullptr && hd < h + hk;
  const float* cs = turn ? rotary + static_cast<size_t>(positions[t]) * rd : nullptr;
  for (int c0 = 0; c0 < n; c0 += 32 * N) {
    const int c = c0 + lane * N;
    if (c < n) load_n<N>(src + c, f);
    if (w && c < n) {
#pragma unroll
      for (int j = 0; j < N; ++j) f[j] = f[j] * inv * w[c + j];
    }
    if (turn) {
      if constexpr (N == 1) {
        const float other = __shfl_xor_sync(0xffffffffu, f[0], 1);
        if (c < rd) {
          const float co = cs[c >> 1], si = cs[rd / 2 + (c >> 1)];
          f[0] = c & 1 ? f[0] * co + other * si : f[0] * co - other * si;
        }
      } else {
#pragma unroll
        for (int j = 0; j < N; j += 2)
          if (c + j < rd) {
            const int i = (c + j) >> 1;
            const float co = cs[i], si = cs[rd / 2 + i], a = f[j], b = f[j + 1];
            f[j] = a * co - b * si;
            f[j + 1] = b * co + a * si;
          }
      }
    }
    if (c < n) store_n<N>(dst + c, f);
  }
}

// ---- QK norm over whole rows, rotation of halves, cache append -------------------------------------------------------
// One CTA per token. All heads of q are normalised together, then all of k; then entries i and i + rd / 2 of every head
// turn; q stays in place, k and v go to their cache slots. N consecutive columns per thread.
template <typename T, int N>
__global__ void __launch_bounds__(256)
qk_row_norm_cache_kernel(T* __restrict__ q, int ldq, const T* __restrict__ k, int ldk, const T* __restrict__ v, int ldv,
                         const int* __restrict__ slots, T* __restrict__ cache, const float* __restrict__ qw,
                         const float* __restrict__ kw, float eps, const int* __restrict__ positions,
                         const float* __restrict__ rotary, int rd, int h, int hk, int d, int dv, int bs) {
  extern __shared__ float row_qk[];  // [h * d] queries, [hk * d] keys
  __shared__ float red[32];
  const int t = blockIdx.x, nq = h * d, nk = hk * d;
  q += static_cast<size_t>(t) * ldq;
  k += static_cast<size_t>(t) * ldk;
  v += static_cast<size_t>(t) * ldv;
  float f[N], sq = 0.f, sk = 0.f;
  for (int c = threadIdx.x * N; c < nq + nk; c += 256 * N) {
    const bool is_q = c < nq;
    load_n<N>(is_q ? q + c : k + c - nq, f);
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < N; ++j) {
      row_qk[c + j] = f[j];
      s += f[j] * f[j];
    }
    if (is_q) sq += s; else sk += s;
  }
  const float iq = 1.f / sqrtf(block_sum(sq, red) / static_cast<float>(nq) + eps);
  const float ik = 1.f / sqrtf(block_sum(sk, red) / static_cast<float>(nk) + eps);  // (its barriers: the row is complete)
  const float* cs = rotary ? rotary + static_cast<size_t>(positions[t]) * rd : nullptr;
  const int slot = slots[t], half = rd >> 1;
  T* block = cache + static_cast<size_t>(max(slot, 0) / bs) * (static_cast<size_t>(hk) * bs * (d + dv));
  const int off = max(slot, 0) % bs;
  for (int c = threadIdx.x * N; c < nq + nk; c += 256 * N) {
    const bool is_q = c < nq;
    const float inv = is_q ? iq : ik;
    const float* w = is_q ? qw : kw - nq;
    const int hd = (is_q ? c : c - nq) / d, i0 = (is_q ? c : c - nq) % d;
#pragma unroll
    for (int j = 0; j < N; ++j) {
      const int i = i0 + j;
      float x = row_qk[c + j] * inv * w[c + j];
      if (i < rd && cs) {
        const bool low = i < half;
        const int p = low ? c + j + half : c + j - half, a = low ? i : i - half;
        const float y = row_qk[p] * inv * w[p];
        x = low ? x * cs[a] - y * cs[half + a] : x * cs[a] + y * cs[half + a];
      }
      f[j] = x;
    }
    if (is_q)
      store_n<N>(q + c, f);
    else if (slot >= 0)
      store_n<N>(block + (static_cast<size_t>(hd) * bs + off) * d + i0, f);
  }
  if (slot < 0) return;
  for (int c = threadIdx.x * N; c < hk * dv; c += 256 * N) {
    load_n<N>(v + c, f);
    store_n<N>(block + static_cast<size_t>(hk) * bs * d + (static_cast<size_t>(c / dv) * bs + off) * dv + c % dv, f);
  }
}

// ---- cache append beside an activation -----------------------------------------------------------------------------
// A row of x holds new keys (nk columns, to the cache of keys alone: [block][hk x bs x d]) and, behind them, the input of
// a feed-forward's activation: out = gelu(up), or gelu(gate) * up over 2 I columns. N columns per thread.
template <typename T, int N>
__global__ void __launch_bounds__(256)
append_act_kernel(const T* __restrict__ k, const T* __restrict__ u, int ldx, const int* __restrict__ slots,
                  T* __restrict__ cache, int nk, int d, int bs, T* __restrict__ out, int ldo, int I, int gated) {
  const size_t row = blockIdx.x;
  int c = (blockIdx.y * 256 + threadIdx.x) * N;
  float f[N];
  if (c < nk) {
    const int slot = slots[row];
    if (slot < 0) return;
    load_n<N>(k + row * ldx + c, f);
    store_n<N>(cache + static_cast<size_t>(slot / bs) * bs * nk + (static_cast<size_t>(c / d) * bs + slot % bs) * d + c % d,
               f);
    return;
  }
  c -= nk;
  if (c >= I) return;
  load_n<N>(u + row * ldx + c, f);
  float g[N];
  if (gated) load_n<N>(u + row * ldx + I + c, g);
#pragma unroll
  for (int j = 0; j < N; ++j) f[j] = gelu_tanh_as<T>(f[j]) * (gated ? g[j] : 1.f);
  store_n<N>(out + row * ldo + c, f);
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

// per head (w: null, or a factor per column of all heads): a warp takes HEADS heads of a token at a time, up to 32 N columns each in registers
template <typename T, int N, int HEADS>
__global__ void __launch_bounds__(256)
gated_head_norm_kernel(const T* __restrict__ o, const T* __restrict__ g, int ldg, const float* __restrict__ w,
                       T* __restrict__ out, int ldo, int tokens, int h, int dv, float eps, int gate, float out_scale) {
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
      if (w && h0 + i < h && c < dv) {
        float ww[N];
        load_n<N>(w + (h0 + i) * dv + c, ww);
#pragma unroll
        for (int j = 0; j < N; ++j) f[i][j] *= ww[j];
      }
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
      for (int j = 0; j < N; ++j) f[j] *= inv * gate_f<T>(gg[j], gate) * (w ? w[hd * dv + c + j] : 1.f);
      store_n<N>(out + t * ldo + hd * dv + c, f);
    }
  }
}

// The same for heads of exactly 8 LANES columns (16-bit): LANES lanes take a head, and every lane two heads at a time.
template <int LANES>
__global__ void __launch_bounds__(256)
gated_head_norm_packed_kernel(const __nv_bfloat16* __restrict__ o, const __nv_bfloat16* __restrict__ g, int ldg,
                              const float* __restrict__ w, __nv_bfloat16* __restrict__ out, int ldo, long long units, int h,
                              float eps, int gate, float out_scale) {
  const int l = threadIdx.x % LANES, c = l * 8;
  const long long stride = static_cast<long long>(gridDim.x) * (256 / LANES);  // (both heads of a lane are far apart: no matter)
  const long long u0 = static_cast<long long>(blockIdx.x) * (256 / LANES) + threadIdx.x / LANES;
  float f[2][8], gg[2][8];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const long long u = u0 + i * stride;  // (token, head)
#pragma unroll
    for (int j = 0; j < 8; ++j) f[i][j] = gg[i][j] = 0.f;
    if (u < units) {
      load_n<8>(o + u * (8 * LANES) + c, f[i]);
      load_n<8>(g + (u / h) * ldg + (u % h) * (8 * LANES) + c, gg[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const long long u = u0 + i * stride;
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += f[i][j] * f[i][j];
#pragma unroll
    for (int x = LANES / 2; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);
    const float inv = out_scale / sqrtf(ss / static_cast<float>(8 * LANES) + eps);
    if (u >= units) continue;
    const int col = static_cast<int>(u % h) * (8 * LANES) + c;
#pragma unroll
    for (int j = 0; j < 8; ++j) f[i][j] *= inv * gate_f<__nv_bfloat16>(gg[i][j], gate);
    if (w) {
      load_n<8>(w + col, gg[i]);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[i][j] *= gg[i][j];
    }
    store_n<8>(out + (u / h) * ldo + col, f[i]);
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

// Storage types: 0 = fp32, 1 = bf16. `kinds` = x (and y) | stream << 1 | weight << 2 | out << 3. Row pitches in elements.
KSANA_API int ksana_stream_norm(const void* x, int ldx, const void* res_in, void* res_out, int ldr, const void* w,
                                const void* b, void* out, int ldo, int rows, int H, float eps, int kinds, int center,
                                const float* add_rows, const float* add_vec, const void* y, const int* pos,
                                const float* weights, int k, cudaStream_t st) {
  if (rows <= 0 || H <= 0) return 0;
#define KSANA_SN_CASE(K, X, R, W, O)                                                                             \
  case K:                                                                                                        \
    return launch_stream_norm<X, R, W, O>(x, ldx, res_in, res_out, ldr, w, b, out, ldo, rows, H, eps, center,    \
                                          add_rows, add_vec, y, pos, weights, k, st)
  switch (kinds) {
    KSANA_SN_CASE(0, float, float, float, float);
    KSANA_SN_CASE(12, float, float, bf16, bf16);  // first norm of a bf16 model over its 32-bit stream
    KSANA_SN_CASE(13, bf16, float, bf16, bf16);   // sublayer output into the 32-bit stream
    KSANA_SN_CASE(15, bf16, bf16, bf16, bf16);
    default: return -1;
  }
#undef KSANA_SN_CASE
}

// residual (may be null) += x, and its LayerNorm
KSANA_API int ksana_layer_norm(const void* x, int ldx, void* residual, int ldr, const void* w, const void* b, void* out,
                               int ldo, int rows, int H, float eps, int kinds, cudaStream_t st) {
  return ksana_stream_norm(x, ldx, residual, residual, ldr, w, b, out, ldo, rows, H, eps, kinds, 1, nullptr, nullptr,
                           nullptr, nullptr, nullptr, 0, st);
}

// pos_table may be null (no learned positions); both tables have storage type `kind`.
KSANA_API int ksana_embedding_f32(const int* ids, const void* table, float* out, int rows, int H, int vocab, float scale,
                                  const int* positions, const void* pos_table, int pos_rows, int kind,
                                  cudaStream_t st) {
  if (rows <= 0) return 0;
  dim3 grid((H + 255) / 256, rows);
  if (kind)
    embedding_f32_kernel<<<grid, 256, 0, st>>>(ids, static_cast<const bf16*>(table), out, H, vocab, scale, positions,
                                               static_cast<const bf16*>(pos_table), pos_rows);
  else
    embedding_f32_kernel<<<grid, 256, 0, st>>>(ids, static_cast<const float*>(table), out, H, vocab, scale, positions,
                                               static_cast<const float*>(pos_table), pos_rows);
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

// x: [rows, cols] with pitch ldx, out: contiguous.
KSANA_API int ksana_relu2(const void* x, int ldx, void* out, int rows, int cols, int kind, cudaStream_t st) {
  if (rows <= 0 || cols <= 0) return 0;
  const size_t n = static_cast<size_t>(rows) * cols;
  const bool vec = !(n & 7) && (ldx == cols || !((ldx | cols) & 7)) && aligned(x, 16) && aligned(out, 16);
#define KSANA_R2(T, N)                                                                                        \
  relu2_kernel<T, N><<<static_cast<unsigned>((n / N + (n % N ? 1 : 0) + 255) / 256), 256, 0, st>>>(           \
      static_cast<const T*>(x), ldx, static_cast<T*>(out), cols, n)
  if (kind) {
    if (vec) KSANA_R2(bf16, 8); else KSANA_R2(bf16, 1);
  } else {
    if (vec) KSANA_R2(float, 8); else KSANA_R2(float, 1);
  }
#undef KSANA_R2
  return done();
}

// x: [rows, 2 I] contiguous, out: [rows, I].
KSANA_API int ksana_clamped_gate_mul(const void* x, void* out, int rows, int I, float limit, float alpha, int kind,
                                     cudaStream_t st) {
  if (rows <= 0 || I <= 0) return 0;
  const bool vec = !(I & 7) && aligned(x, 16) && aligned(out, 16);
  const int n = vec ? 8 : 1;
  const dim3 grid(rows, (I + n * 256 - 1) / (n * 256));
#define KSANA_CG(T, N) \
  clamped_gate_mul_kernel<T, N><<<grid, 256, 0, st>>>(static_cast<const T*>(x), static_cast<T*>(out), I, limit, alpha)
  if (kind) {
    if (vec) KSANA_CG(bf16, 8); else KSANA_CG(bf16, 1);
  } else {
    if (vec) KSANA_CG(float, 8); else KSANA_CG(float, 1);
  }
#undef KSANA_CG
  return done();
}

KSANA_API int ksana_qk_norm_cache(void* q, int ldq, const void* k, int ldk, const void* v, int ldv, const int* slots,
                                  void* cache, const float* qw, const float* kw, float eps, const int* positions,
                                  const float* rotary, int rd, int tokens, int h, int hk, int d, int dv, int bs, int kind,
                                  cudaStream_t st) {
  if (tokens <= 0) return 0;
  if (rotary && (rd < 0 || rd > d || (rd & 1))) return -2;
  const int esz = kind ? 2 : 4;
  const bool vec = !((ldq | ldk | ldv | d | dv) & 3) && aligned(q, 4 * esz) && aligned(k, 4 * esz) &&
                   aligned(v, 4 * esz) && aligned(cache, 4 * esz);
  if (!qw && !rotary) h = 0;
  if (h + hk <= 0) return 0;
  const long long units = static_cast<long long>(tokens) * (h + 2 * hk);
  const unsigned grid = static_cast<unsigned>((units + 7) / 8);
#define KSANA_QK(T, N)                                                                                              \
  qk_norm_cache_kernel<T, N><<<grid, 256, 0, st>>>(static_cast<T*>(q), ldq, static_cast<const T*>(k), ldk,          \
                                                   static_cast<const T*>(v), ldv, slots, static_cast<T*>(cache), qw, \
                                                   kw, eps, positions, rotary, rd, tokens, h, hk, d, dv, bs)
  if (kind) {
    if (vec) KSANA_QK(bf16, 4); else KSANA_QK(bf16, 1);
  } else {
    if (vec) KSANA_QK(float, 4); else KSANA_QK(float, 1);
  }
#undef KSANA_QK
  return done();
}

// k: [tokens, hk * d] or null (hk 0: nothing to append); u: [tokens, I or 2 I] or null (I 0: no activation), both inside
// rows of pitch ldx. The cache holds keys alone.
KSANA_API int ksana_append_act(const void* k, const void* u, int ldx, const int* slots, void* cache, int tokens, int hk,
                               int d, int bs, void* out, int ldo, int I, int gated, int kind, cudaStream_t st) {
  const int nk = hk * d;
  if (tokens <= 0 || nk + I <= 0) return 0;
  const bool vec = !((ldx | d | I | ldo) & 7) && aligned(k, 16) && aligned(u, 16) &&
                   aligned(cache, 16) && aligned(out, 16);
  const int n = vec ? 8 : 1;
  const dim3 grid(tokens, (nk + I + n * 256 - 1) / (n * 256));
#define KSANA_AA(T, N)                                                                                             \
  append_act_kernel<T, N><<<grid, 256, 0, st>>>(static_cast<const T*>(k), static_cast<const T*>(u), ldx, slots,    \
                                                static_cast<T*>(cache), nk, d, bs, static_cast<T*>(out), ldo, I, gated)
  if (kind) {
    if (vec) KSANA_AA(bf16, 8); else KSANA_AA(bf16, 1);
  } else {
    if (vec) KSANA_AA(float, 8); else KSANA_AA(float, 1);
  }
#undef KSANA_AA
  return done();
}

// The stream takes two gated sublayers, see GatedNormArgs. All activations have storage type `kind` (0 fp32, 1 bf16);
// norms 1 or 2.
KSANA_API int ksana_gated_stream_norm(const void* x, int ldx, const void* xg, int ldxg, const void* rows, const int* pos,
                                      const float* weights, int k, const void* y, int ldy, const float* ys, int ldys,
                                      const void* yg, int ldyg, float scale, const float* in, float* stream,
                                      const void* w0, const void* w1, void* out, int tokens, int H, float eps, int kind,
                                      cudaStream_t st) {
  if (tokens <= 0 || H <= 0) return 0;
#define KSANA_GSN_ARGS(T)                                                                                                 \
  GatedNormArgs<T>{static_cast<const T*>(x), static_cast<const T*>(xg), static_cast<const T*>(rows),                      \
                   static_cast<const T*>(y), static_cast<const T*>(yg), ldx, ldxg, ldy, ldyg, ldys, rows ? k : 0, H,       \
                   w1 ? 2 : 1, pos, weights, ys, scale, eps, in, stream,                                                   \
                   {static_cast<const T*>(w0), static_cast<const T*>(w1)}, static_cast<T*>(out),                           \
                   static_cast<size_t>(tokens) * H}
  return kind ? launch_gated_norm<bf16>(KSANA_GSN_ARGS(bf16), tokens, st)
              : launch_gated_norm<float>(KSANA_GSN_ARGS(float), tokens, st);
#undef KSANA_GSN_ARGS
}

KSANA_API int ksana_qk_row_norm_cache(void* q, int ldq, const void* k, int ldk, const void* v, int ldv, const int* slots,
                                      void* cache, const float* qw, const float* kw, float eps, const int* positions,
                                      const float* rotary, int rd, int tokens, int h, int hk, int d, int dv, int bs,
                                      int kind, cudaStream_t st) {
  if (tokens <= 0) return 0;
  if (rotary && (rd < 0 || rd > d || (rd & 1))) return -2;
  const int esz = kind ? 2 : 4, smem = (h + hk) * d * 4;
  if (smem > 200 * 1024) return -1;
  const bool vec = !((ldq | ldk | ldv | d | dv) & 3) && aligned(q, 4 * esz) && aligned(k, 4 * esz) &&
                   aligned(v, 4 * esz) && aligned(cache, 4 * esz);
#define KSANA_QR(T, N)                                                                                                  \
  do {                                                                                                                  \
    auto kern = qk_row_norm_cache_kernel<T, N>;                                                                         \
    if (smem > 47 * 1024 && KSANA_SMEM_ONCE(kern, 200 * 1024) != 0) return -4;                                          \
    kern<<<tokens, 256, smem, st>>>(static_cast<T*>(q), ldq, static_cast<const T*>(k), ldk, static_cast<const T*>(v),   \
                                    ldv, slots, static_cast<T*>(cache), qw, kw, eps, positions, rotary, rd, h, hk, d,   \
                                    dv, bs);                                                                            \
  } while (0)
  if (kind) {
    if (vec) KSANA_QR(bf16, 4); else KSANA_QR(bf16, 1);
  } else {
    if (vec) KSANA_QR(float, 4); else KSANA_QR(float, 1);
  }
#undef KSANA_QR
  return done();
}

// gate: 0 silu, 1 sigmoid. w == nullptr: per head, no weight; per_head: per head, then w over all columns. o is [tokens, h, dv] contiguous.
KSANA_API int ksana_gated_norm(const void* o, const void* g, int ldg, const float* w, void* out, int ldo, int tokens,
                               int h, int dv, float eps, int gate, float out_scale, int per_head, int kind,
                               cudaStream_t st) {
  if (tokens <= 0) return 0;
  const int esz = kind ? 2 : 4;
  const int width = h * dv;
  const bool vec = !((dv | ldg | ldo) & 3) && aligned(o, 4 * esz) && aligned(g, 4 * esz) && aligned(out, 4 * esz);
  if (kind && (!w || per_head) && (dv == 32 || dv == 64 || dv == 128) && !((ldg | ldo) & 7) && aligned(o, 16) && aligned(g, 16) &&
      aligned(out, 16) && aligned(w, 16)) {
    const long long units = static_cast<long long>(tokens) * h;
#define KSANA_GHP(L)                                                                                                     \
  gated_head_norm_packed_kernel<L><<<static_cast<unsigned>((units + 2 * (256 / L) - 1) / (2 * (256 / L))), 256, 0, st>>>(  \
      static_cast<const bf16*>(o), static_cast<const bf16*>(g), ldg, w, static_cast<bf16*>(out), ldo, units, h, eps, gate,  \
      out_scale)
    if (dv == 32) KSANA_GHP(4); else if (dv == 64) KSANA_GHP(8); else KSANA_GHP(16);
#undef KSANA_GHP
    return done();
  }
  const bool wide = kind && (!w || per_head) && dv > 128 && !((dv | ldg | ldo) & 7) && aligned(o, 16) && aligned(g, 16) && aligned(out, 16);
  const unsigned grid = static_cast<unsigned>((static_cast<long long>(tokens) * ((h + 3) / 4) + 7) / 8);
#define KSANA_GN(T, N)                                                                                               \
  do {                                                                                                               \
    if (w && !per_head)                                                                                              \
      gated_row_norm_kernel<T, N><<<tokens, 256, 0, st>>>(static_cast<const T*>(o), static_cast<const T*>(g), ldg, w, \
                                                          static_cast<T*>(out), ldo, width, eps, gate, out_scale);   \
    else                                                                                                             \
      gated_head_norm_kernel<T, N, 4><<<grid, 256, 0, st>>>(static_cast<const T*>(o), static_cast<const T*>(g), ldg, w, \
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
