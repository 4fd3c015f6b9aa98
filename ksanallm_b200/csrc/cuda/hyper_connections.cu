// Hyper-connected residual streams: S rows of 32-bit floats per token instead of one. Between two sublayers one launch
// takes the last one's result into every stream, mixes the streams, reads the next one's input out of them and normalises
// it:
//   y    = (x + sum_j weights[t, j] rows[pos[t, j]]) * scale          (every term may be absent)
//   v_t  = sum_s mix[s, t] in_s + out_w[t] y                          (mix null: v = in)
//   out  = u / sqrt(mean(u^2) + eps) * w   with   u = sum_t in_w[t] v_t
// All of it is computed in 32-bit floats; T is the storage type of activations. The streams are the traffic: 8 S bytes
// per token and column, read and written once.
#include "host_common.h"
#include "mixer_common.cuh"

namespace ksana {

template <typename T>
struct HyperArgs {
  const T* x;
  int ldx;
  const float* scale;    // [H]
  const T* rows;         // [n, H] in sorted order, pos -1: another rank's
  const int* pos;
  const float* weights;
  int k;
  const float* in;       // stream s of token t at in + t * in_row + s * in_stream (0: all streams are one row)
  long long in_row, in_stream;
  const float* mix;      // [S, S], from x to
  const float* out_w;    // [S]
  float* res;            // [tokens, S, H] (null: not kept)
  const float* in_w;     // [S]
  const T* w;
  T* out;
  int H, S;
  float eps;
};

// NT threads hold a row: VPT groups of 4 columns each. All loads of a thread are in flight together.
template <typename T, int S, int VPT, int NT>
__global__ void __launch_bounds__(NT)
hyper_norm_kernel(const HyperArgs<T> a) {
  __shared__ float red[32];
  __shared__ float cf[S * S + 2 * S];
  const size_t row = blockIdx.x;
  const int tid = threadIdx.x, H = a.H;
  float v[S][VPT][4], y[VPT][4];
  const float* in = a.in + row * a.in_row;
#pragma unroll
  for (int s = 0; s < S; ++s)
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (i * NT + tid) * 4;
      if (c < H) load_n<4>(in + s * a.in_stream + c, v[s][i]);
    }
  if (a.mix) {
    if (tid < S * S) cf[tid] = a.mix[tid];
    if (tid < S) cf[S * S + tid] = a.out_w[tid];
  }
  if (tid < S) cf[S * S + S + tid] = a.in_w[tid];
#pragma unroll
  for (int i = 0; i < VPT; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) y[i][j] = 0.f;
  auto add = [&](const T* p, float wt) {
    float f[VPT][4];
#pragma unroll
    for (int i = 0; i < VPT; ++i)
      if ((i * NT + tid) * 4 < H) load_n<4>(p + (i * NT + tid) * 4, f[i]);
#pragma unroll
    for (int i = 0; i < VPT; ++i)
      if ((i * NT + tid) * 4 < H)
#pragma unroll
        for (int j = 0; j < 4; ++j) y[i][j] = fmaf(wt, f[i][j], y[i][j]);
  };
  if (a.x) add(a.x + row * a.ldx, 1.f);
  for (int e = 0; e < a.k; ++e) {
    const int p = a.pos[row * a.k + e];
    if (p >= 0) add(a.rows + static_cast<size_t>(p) * H, a.weights[row * a.k + e]);
  }
  __syncthreads();
  float u[VPT][4], ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (i * NT + tid) * 4;
    if (c < H) {
      if (a.scale) {
        float f[4];
        load_n<4>(a.scale + c, f);
#pragma unroll
        for (int j = 0; j < 4; ++j) y[i][j] *= f[j];
      }
      if (a.mix) {
        float n[S][4];
#pragma unroll
        for (int t = 0; t < S; ++t)
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            float z = cf[S * S + t] * y[i][j];
#pragma unroll
            for (int s = 0; s < S; ++s) z = fmaf(cf[s * S + t], v[s][i][j], z);
            n[t][j] = z;
          }
#pragma unroll
        for (int t = 0; t < S; ++t) {
          if (a.res) store_n<4>(a.res + (row * S + t) * H + c, n[t]);
#pragma unroll
          for (int j = 0; j < 4; ++j) v[t][i][j] = n[t][j];
        }
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        float z = 0.f;
#pragma unroll
        for (int t = 0; t < S; ++t) z = fmaf(cf[S * S + S + t], v[t][i][j], z);
        u[i][j] = z;
        ss = fmaf(z, z, ss);
      }
    }
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / static_cast<float>(H) + a.eps);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (i * NT + tid) * 4;
    if (c < H) {
      float g[4];
      load_n<4>(a.w + c, g);
#pragma unroll
      for (int j = 0; j < 4; ++j) g[j] *= u[i][j] * inv;
      store_n<4>(a.out + row * H + c, g);
    }
  }
}

// Any width and up to 16 streams: the row's next input stays in shared memory.
constexpr int HYPER_MAX = 16;
template <typename T>
__global__ void __launch_bounds__(256)
hyper_norm_any_kernel(const HyperArgs<T> a) {
  extern __shared__ float row_u[];
  __shared__ float red[32];
  __shared__ float cf[HYPER_MAX * HYPER_MAX + 2 * HYPER_MAX];
  const size_t row = blockIdx.x;
  const int tid = threadIdx.x, H = a.H, S = a.S;
  float* out_w = cf + S * S;
  float* in_w = out_w + S;
  if (a.mix)
    for (int i = tid; i < S * S; i += 256) cf[i] = a.mix[i];
  if (tid < S) {
    out_w[tid] = a.mix ? a.out_w[tid] : 0.f;
    in_w[tid] = a.in_w[tid];
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = tid; c < H; c += 256) {
    float v[HYPER_MAX];
#pragma unroll
    for (int s = 0; s < HYPER_MAX; ++s)
      if (s < S) v[s] = a.in[row * a.in_row + s * a.in_stream + c];
    float u = 0.f;
    if (a.mix) {
      float y = a.x ? to_f(a.x[row * a.ldx + c]) : 0.f;
      for (int e = 0; e < a.k; ++e) {
        const int p = a.pos[row * a.k + e];
        if (p >= 0) y = fmaf(a.weights[row * a.k + e], to_f(a.rows[static_cast<size_t>(p) * H + c]), y);
      }
      if (a.scale) y *= a.scale[c];
      for (int t = 0; t < S; ++t) {
        float z = out_w[t] * y;
#pragma unroll
        for (int s = 0; s < HYPER_MAX; ++s)
          if (s < S) z = fmaf(cf[s * S + t], v[s], z);
        if (a.res) a.res[(row * S + t) * H + c] = z;
        u = fmaf(in_w[t], z, u);
      }
    } else {
#pragma unroll
      for (int s = 0; s < HYPER_MAX; ++s)
        if (s < S) u = fmaf(in_w[s], v[s], u);
    }
    row_u[c] = u;  // only this thread reads it back
    ss = fmaf(u, u, ss);
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / static_cast<float>(H) + a.eps);
  for (int c = tid; c < H; c += 256) a.out[row * H + c] = from_f<T>(row_u[c] * inv * to_f(a.w[c]));
}

template <typename T>
static int launch_any(const HyperArgs<T>& a, int tokens, cudaStream_t st) {
  if (a.H > 50 * 1024 || a.S > HYPER_MAX) return -1;
  auto kern = hyper_norm_any_kernel<T>;
  if (a.H * 4 > 40 * 1024 && KSANA_SMEM_ONCE(kern, 200 * 1024) != 0) return -4;
  kern<<<tokens, 256, a.H * 4, st>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

template <int S>
static int launch_rows(const HyperArgs<__nv_bfloat16>& a, int tokens, cudaStream_t st) {
#define KSANA_HN(V, NT) hyper_norm_kernel<__nv_bfloat16, S, V, NT><<<tokens, NT, 0, st>>>(a)
  if (a.H <= 1024) {
    KSANA_HN(1, 256);
  } else if (a.H <= 2048) {
    KSANA_HN(2, 256);
  } else if (a.H <= 4096) {
    KSANA_HN(4, 256);
  } else {
    KSANA_HN(4, 512);
  }
#undef KSANA_HN
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

}  // namespace ksana

using namespace ksana;

// streams: [tokens, S, H] fp32, or [tokens, H] (one != 0) while all streams are still equal. kind: 0 fp32, 1 bf16.
KSANA_API int ksana_hyper_norm(const void* x, int ldx, const float* scale, const void* rows, const int* pos,
                               const float* weights, int k, const float* streams, int one, const float* mix,
                               const float* out_w, float* res, const float* in_w, const void* w, void* out, int tokens,
                               int H, int S, float eps, int kind, cudaStream_t st) {
  if (tokens <= 0) return 0;
  if (S < 1 || H < 1) return -2;
  auto args = [&](auto* type) {
    using T = std::remove_pointer_t<decltype(type)>;
    const long long hh = H;
    return HyperArgs<T>{static_cast<const T*>(x), ldx, scale, static_cast<const T*>(rows), pos, weights, rows ? k : 0,
                        streams, one ? hh : hh * S, one ? 0 : hh, mix, out_w, res, in_w, static_cast<const T*>(w),
                        static_cast<T*>(out), H, S, eps};
  };
  if (!kind) return launch_any(args(static_cast<float*>(nullptr)), tokens, st);
  const auto a = args(static_cast<__nv_bfloat16*>(nullptr));
  auto aligned = [](const void* p, int bytes) { return (reinterpret_cast<uintptr_t>(p) & (bytes - 1)) == 0; };
  const bool vec = !((H | ldx) & 3) && H <= 8192 && aligned(x, 8) && aligned(rows, 8) && aligned(w, 8) &&
                   aligned(out, 8) && aligned(streams, 16) && aligned(res, 16) && aligned(scale, 16);
  if (vec) {
    if (S == 1) return launch_rows<1>(a, tokens, st);
    if (S == 2) return launch_rows<2>(a, tokens, st);
    if (S == 3) return launch_rows<3>(a, tokens, st);
    if (S == 4) return launch_rows<4>(a, tokens, st);
  }
  return launch_any(a, tokens, st);
}
