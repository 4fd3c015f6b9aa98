// Attention over the paged cache of layers with sizes of their own: a sliding window, first tokens that stay visible
// behind it, a learned bias per distance, key / value heads of different sizes, or values that are the keys. Scores,
// softmax and the accumulation are 32-bit.
//
// Cache of a layer: [block][keys hk x bs x d | values hk x bs x dv], the second part only where values are not the keys.
// bias: [h][bias_len] fp32 (null: none), indexed by the distance between query and key.
//
// Query i sees key j when j <= i and (i - j < window or j < keep); window 0: every j <= i.
//
// softcap > 0: a score becomes cap * tanh(score / cap) before anything else. sink: the softmax's denominator has one more
// term exp(0). gate: each head's result is multiplied by the sigmoid of gate[token][head] (the storage type of q). Where
// the cache holds keys alone, a key's first dv numbers are its value.
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
  int h, hk, d, dv, bs, window, keep, shared;  // shared: values are the keys (their first dv numbers)
  float scale;
  const float* bias;
  int bias_len;
  float out_scale;
  void* out;
  int ldo;
  float softcap;
  int sink;
  const void* gate;
  int ldg;
  __host__ __device__ size_t v_off() const { return shared ? 0 : static_cast<size_t>(hk) * bs * d; }
  __host__ __device__ size_t block_elems() const { return static_cast<size_t>(hk) * bs * (d + (shared ? 0 : dv)); }
  // oldest key inside the window of the query at `pos`
  __device__ int window_start(int pos) const { return window > 0 && pos - window + 1 > 0 ? pos - window + 1 : 0; }
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
  const size_t block_elems = a.block_elems(), v_off = a.v_off();
  const float* bias = a.bias ? a.bias + static_cast<size_t>(head) * a.bias_len : nullptr;
  const int lo = a.window_start(pos);
  const int kept = min(a.keep, lo), n = kept + pos - lo + 1;  // the visible keys: [0, kept) and [lo, pos]
  float m = -INFINITY, l = 0.f, acc[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) acc[i] = 0.f;
  for (int i0 = 0; i0 < n; i0 += 32) {
    const int i = i0 + lane, j = i < kept ? i : lo + i - kept;
    float s = -INFINITY;
    if (i < n) {
      const T* kp = cache + bt[j / a.bs] * block_elems + (static_cast<size_t>(kh) * a.bs + j % a.bs) * a.d;
      float dot[4] = {0.f, 0.f, 0.f, 0.f};
      int c = 0;
      for (; c + 4 <= a.d; c += 4)
#pragma unroll
        for (int u = 0; u < 4; ++u) dot[u] = fmaf(sq[c + u], to_f(kp[c + u]), dot[u]);
      for (; c < a.d; ++c) dot[0] = fmaf(sq[c], to_f(kp[c]), dot[0]);
      s = ((dot[0] + dot[1]) + (dot[2] + dot[3])) * a.scale;
      if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
      if (bias) s += bias[min(pos - j, a.bias_len - 1)];
    }
    const float m_new = fmaxf(m, warp_max(s));
    const float f = expf(m - m_new);
    const float p = i < n ? expf(s - m_new) : 0.f;
    l = l * f + warp_sum(p);
    m = m_new;
    float part[NV];  // of these 32 keys: long sums in two steps keep their rounding small
#pragma unroll
    for (int i = 0; i < NV; ++i) part[i] = 0.f;
    const int count = min(32, n - i0);
    for (int u = 0; u < count; ++u) {
      const float pu = __shfl_sync(0xffffffffu, p, u);
      const int ju = i0 + u < kept ? i0 + u : lo + i0 + u - kept;
      const T* vp = cache + bt[ju / a.bs] * block_elems + v_off +
                    (static_cast<size_t>(kh) * a.bs + ju % a.bs) * (a.shared ? a.d : a.dv);
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = i * 32 + lane;
        if (c < a.dv) part[i] = fmaf(pu, to_f(vp[c]), part[i]);
      }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) acc[i] = fmaf(acc[i], f, part[i]);
  }
  T* o = static_cast<T*>(a.out) + static_cast<size_t>(t) * a.ldo + head * a.dv;
  if (a.sink) {  // relative to the larger of the running maximum and the sink's own score
    const float top = fmaxf(m, 0.f), f = expf(m - top);
    l = l * f + expf(-top);
#pragma unroll
    for (int i = 0; i < NV; ++i) acc[i] *= f;
  }
  float inv = a.out_scale / l;
  if (a.gate) inv *= sigmoid_f(to_f(static_cast<const T*>(a.gate)[static_cast<size_t>(t) * a.ldg + head]));
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

// ---- prompts: tcgen05 ------------------------------------------------------------------------------------------------
// One CTA = 128 query rows of one (sequence, head), 160 threads. Thread r of warps 0-3 owns query row r (TMEM lane r);
// one lane of warp 4 issues the TMA loads and the MMAs, so that Q K^T of the next tile runs under the softmax of this
// one. Per 128-key tile:
//   S = Q K^T       128 x 128 x DP -> TMEM, two buffers
//   softmax         scores + bias in registers; the mask is part of the tile's bias table (one entry per distance,
//                   -inf outside the window); running max with a lazy rescale of O
//   O += P V        A = P from TMEM, written over S as two bf16 matrices hi + lo (the weights keep 16 mantissa bits)
// Tiles start at the block of 128 keys that holds the first row's oldest key in the window; the blocks of the kept first
// tokens ahead of it come first. Where a block holds kept tokens its table has no window cut, and the scores are masked
// one by one. Head sizes below DP / DVP are filled up with zeros by TMA.
//
// LATENT: keys and values of every head have been written out of the latents, [row][h x d keys | h x dv values] with the
// contexts of the sequences behind one another; the last 64 columns of a key are the rotated part all heads share.
//
// SHARED: the values are the keys. Both products read the same tile in shared memory - rows of keys are K-major for
// Q K^T and MN-major for P V - and the values' room holds a third tile in flight.
constexpr int WP_PAGE = 16;

template <int DP, int DVP, bool SHARED>
struct WindowPrefillSmem {
  static constexpr int STAGES = SHARED ? 3 : 2;
  static constexpr int Q_BYTES = 128 * DP * 2;
  static constexpr int K_BYTES = 128 * DP * 2;
  static constexpr int V_BYTES = 128 * DVP * 2;
  static constexpr int OFF_K = Q_BYTES;
  static constexpr int OFF_V = OFF_K + STAGES * K_BYTES;
  static constexpr int OFF_TAB = OFF_V + (SHARED ? 0 : 2) * V_BYTES;
  static constexpr int OFF_BAR = OFF_TAB + 2 * 256 * 4;
  static constexpr int USED = OFF_BAR + 256 + 1024;
  // at least half of the SM's shared memory: two CTAs would compete for the 512 TMEM columns each of them takes
  static constexpr int TOTAL = USED > 120 * 1024 ? USED : 120 * 1024;
};

// The cap of a score, in units where exp2 is the exponential: s -> c tanh(s / c) with c in those units. Tiles whose scores
// are small against the cap take the Taylor series of tanh to degree 11 (error below 1e-7 of the cap up to |s / c| = 0.4); others
// the exponential form.
constexpr float CAP_POLY = 0.4f;
// two 32-bit floats in one register pair; FMAs on them issue as one
__device__ __forceinline__ uint64_t pair(float a, float b) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ void cap_small2(float* s, float inv_c) {
  const uint64_t v = pair(s[0], s[1]), x = mul2(v, pair(inv_c, inv_c)), z = mul2(x, x);
  uint64_t p = fma2(z, pair(-1382.f / 155925.f, -1382.f / 155925.f), pair(62.f / 2835.f, 62.f / 2835.f));
  p = fma2(p, z, pair(-17.f / 315.f, -17.f / 315.f));
  p = fma2(p, z, pair(2.f / 15.f, 2.f / 15.f));
  p = fma2(p, z, pair(-1.f / 3.f, -1.f / 3.f));
  p = fma2(mul2(p, z), v, v);
  asm("mov.b64 {%0, %1}, %2;" : "=f"(s[0]), "=f"(s[1]) : "l"(p));
}
__device__ __forceinline__ float cap_any(float s, float c, float inv_c) {
  const float x = fminf(fmaxf(s * inv_c, -20.f), 20.f);
  return c - __fdividef(2.f * c, 1.f + __expf(2.f * x));
}

template <int DP, int DVP, bool SHARED, bool KEEP, bool CAP, bool LATENT = false>
__global__ void __launch_bounds__(160, 1)
window_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                      const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmR,
                      WindowAttnArgs a, int seq_base, unsigned int* err) {
  constexpr int DN = LATENT ? DP - 64 : DP;  // columns of a key's own
  using L_ = WindowPrefillSmem<DP, DVP, SHARED>;
  constexpr int STAGES = L_::STAGES;
  const int b = blockIdx.y + seq_base, head = blockIdx.z, qt = blockIdx.x;
  const int q0 = a.cu_q[b];
  const int q_len = a.cu_q[b + 1] - q0;
  if (qt * 128 >= q_len) return;
  const int L = a.kv_lens[b];
  const int row_pos = L - q_len + qt * 128;  // position of query row 0
  const int kh = head / (a.h / a.hk);
  const int tid = threadIdx.x, warp = tid >> 5;

  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;
  uint8_t* sK = smem + L_::OFF_K;
  uint8_t* sV = smem + L_::OFF_V;
  float* tab = reinterpret_cast<float*>(smem + L_::OFF_TAB);  // [2][256]
  uint64_t* q_bar = reinterpret_cast<uint64_t*>(smem + L_::OFF_BAR);
  uint64_t* k_full = q_bar + 1;        // [STAGES]
  uint64_t* v_full = k_full + STAGES;  // [2]
  uint64_t* s_done = v_full + 2;  // [2]
  uint64_t* p_ready = s_done + 2;
  uint64_t* o_done = p_ready + 1;
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(o_done + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_holder + 1);

  if (tid == 0) {
    mbar_init(q_bar, 1);
    for (int s = 0; s < STAGES; ++s) mbar_init(&k_full[s], 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(&v_full[s], 1);
      mbar_init(&s_done[s], 1);
    }
    mbar_init(p_ready, 128);
    mbar_init(o_done, 1);
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 0) {
    tmem_alloc(tmem_holder, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_S = *tmem_holder;       // two buffers of 128 columns
  const uint32_t tmem_O = tmem_S + 256;

  const int kt0 = a.window_start(row_pos) / 128;
  const int kv_end = min(L, row_pos + 128);
  // tiles of kept tokens ahead of the window's
  const int n_kept = KEEP ? min(a.keep / 128 + (a.keep % 128 != 0), kt0) : 0;
  const int n = n_kept + (kv_end + 127) / 128 - kt0;  // >= 1
  auto tile = [&](int i) { return i < n_kept ? i : kt0 + i - n_kept; };
  const int n_pages = (L + WP_PAGE - 1) / WP_PAGE;
  const int* bt = a.block_tables + static_cast<size_t>(b) * a.max_blocks;

  if (warp == 4) {
    if ((tid & 31) == 0) {
      int k_loads = 0, v_loads = 0;
      // the pages of tile i of one operand; pages past the sequence repeat its last one (masked keys)
      auto load = [&](const CUtensorMap& tm, uint8_t* base, int bytes, int halves, uint64_t* bar, int i, int st) {
        mbar_expect_tx(&bar[st], bytes);
        for (int p = 0; p < 128 / WP_PAGE; ++p) {
          const int blk = bt[min(tile(i) * (128 / WP_PAGE) + p, n_pages - 1)];
          for (int hf = 0; hf < halves; ++hf)
            tma_load_3d(base + st * bytes + hf * (128 * 128) + p * (WP_PAGE * 128), &tm, &bar[st], hf * 64,
                        kh * WP_PAGE, blk);
        }
      };
      int ctx0 = 0;  // LATENT: the sequence's first row
      if constexpr (LATENT)
        for (int i = seq_base; i < b; ++i) ctx0 += a.kv_lens[i];
      auto load_k = [&](int i) {
        if constexpr (LATENT) {
          uint8_t* dst = sK + (i % STAGES) * L_::K_BYTES;
          uint64_t* bar = &k_full[i % STAGES];
          mbar_expect_tx(bar, L_::K_BYTES);
          for (int hf = 0; hf < DN / 64; ++hf) tma_load_3d(dst + hf * (128 * 128), &tmK, bar, hf * 64, head, ctx0 + i * 128);
          tma_load_2d(dst + (DN / 64) * (128 * 128), &tmR, bar, 0, ctx0 + i * 128);
        } else {
          load(tmK, sK, L_::K_BYTES, DP / 64, k_full, i, i % STAGES);
        }
        k_loads = i + 1;
      };
      auto load_v = [&](int i) {
        if constexpr (LATENT) {
          mbar_expect_tx(&v_full[i & 1], L_::V_BYTES);
          for (int hf = 0; hf < DVP / 64; ++hf)
            tma_load_3d(sV + (i & 1) * L_::V_BYTES + hf * (128 * 128), &tmV, &v_full[i & 1], hf * 64, head, ctx0 + i * 128);
        } else {
          load(tmV, sV, L_::V_BYTES, DVP / 64, v_full, i, i & 1);
        }
        v_loads = i + 1;
      };
      auto issue_qk = [&](int i) {
        tc_fence_after();
        constexpr uint32_t idesc = umma_idesc(128, 128, 1, 1);
        const uint32_t kb = smem_u32(sK + (i % STAGES) * L_::K_BYTES), qb = smem_u32(sQ);
#pragma unroll
        for (int k = 0; k < DP / 16; ++k) {
          const uint32_t off = (k >> 2) * (128 * 128) + (k & 3) * 32;
          umma_f16(tmem_S + (i & 1) * 128, umma_desc_k128(qb + off), umma_desc_k128(kb + off), idesc, k > 0 ? 1u : 0u);
        }
        umma_commit(&s_done[i & 1]);
      };
      mbar_expect_tx(q_bar, L_::Q_BYTES);
      for (int hf = 0; hf < DP / 64; ++hf)
        tma_load_3d(sQ + hf * (128 * 128), &tmQ, q_bar, LATENT && hf == DN / 64 ? a.d : hf * 64, head, q0 + qt * 128);
      load_k(0);
      if constexpr (!SHARED) load_v(0);
      for (int i = 1; i < STAGES && i < n; ++i) load_k(i);
      bool ok = mbar_wait_bounded(q_bar, 0, abort_flag, err) && mbar_wait_bounded(&k_full[0], 0, abort_flag, err);
      if (ok) issue_qk(0);
      for (int i = 0; ok && i < n; ++i) {
        if (i > 0) ok = mbar_wait_bounded(o_done, (i - 1) & 1, abort_flag, err);
        if (!ok) break;
        if (SHARED && i > 0 && i + 2 < n) load_k(i + 2);  // tile i - 1 has been multiplied twice
        if (i + 1 < n) {
          if constexpr (!SHARED) load_v(i + 1);
          ok = mbar_wait_bounded(&k_full[(i + 1) % STAGES], ((i + 1) / STAGES) & 1, abort_flag, err);
          if (!ok) break;
          issue_qk(i + 1);
        }
        ok = mbar_wait_bounded(p_ready, i & 1, abort_flag, err);
        if (!ok) break;
        if constexpr (!SHARED) {
          if (i + 2 < n) load_k(i + 2);  // the keys of tile i have been multiplied
          ok = mbar_wait_bounded(&v_full[i & 1], (i >> 1) & 1, abort_flag, err);
          if (!ok) break;
        }
        tc_fence_after();
        constexpr uint32_t idesc = umma_idesc_major(128, DVP, false, true);
        const uint32_t vb = smem_u32(SHARED ? sK + (i % STAGES) * L_::K_BYTES : sV + (i & 1) * L_::V_BYTES), pb = tmem_S + (i & 1) * 128;
#pragma unroll
        for (int k = 0; k < 16; ++k)  // hi, then lo
          umma_f16_ts(tmem_O, pb + k * 8, umma_desc_mn128(vb + (k & 7) * (16 * 128), 128 * 128), idesc,
                      (i > 0 || k > 0) ? 1u : 0u);
        umma_commit(o_done);
      }
      if (!ok) {
        // copies in flight still write to this CTA's memory: give them their (bounded) time before leaving
        auto drain = [](uint64_t* bar, int stages, int loads) {
          for (int i = max(loads - stages, 0); i < loads; ++i)
            for (int it = 0; it < (1 << 20) && !mbar_try_wait(&bar[i % stages], (i / stages) & 1); ++it) {}
        };
        drain(k_full, STAGES, k_loads);
        drain(v_full, 2, v_loads);
      }
    }
    __syncwarp();
  } else {
    const uint32_t lane_off = static_cast<uint32_t>(warp * 32) << 16;
    const float scale2 = a.scale * 1.4426950408889634f;
    const float cap2 = CAP ? a.softcap * 1.4426950408889634f : 0.f, inv_cap2 = CAP ? 1.f / cap2 : 0.f;
    const float* bias = a.bias ? a.bias + static_cast<size_t>(head) * a.bias_len : nullptr;
    const int reach = a.window > 0 ? min(a.window, 1 << 30) : 1 << 30;
    float m_ref = -INFINITY, l = 0.f;
    bool ok = true;
    for (int i = 0; i < n; ++i) {
      float* tb = tab + (i & 1) * 256;
      const int key0 = tile(i) * 128;
      const int d0 = row_pos - key0 - 127;        // distance of entry 0
      const int kept = KEEP ? a.keep - key0 : 0;  // columns below this one are kept tokens
      const int cut = kept > 0 ? 1 << 30 : reach;
#pragma unroll
      for (int e = tid; e < 256; e += 128) {
        const int dist = d0 + e;
        float v = -INFINITY;
        if (dist >= 0 && dist < cut) v = bias ? bias[min(dist, a.bias_len - 1)] * 1.4426950408889634f : 0.f;
        tb[e] = v;
      }
      asm volatile("bar.sync 1, 128;" ::: "memory");
      if (ok) ok = mbar_wait_bounded(&s_done[i & 1], (i >> 1) & 1, abort_flag, err);
      if (!__all_sync(0xffffffffu, ok)) {
        ok = false;
        continue;  // keep meeting the other warps at the barrier
      }
      tc_fence_after();
      const uint32_t S = tmem_S + (i & 1) * 128 + lane_off;
      float s[128];
#pragma unroll
      for (int c = 0; c < 4; ++c) tmem_ld32(S + c * 32, reinterpret_cast<uint32_t*>(s) + c * 32);
      tmem_wait_ld();
      float m_tile = -INFINITY;
      if constexpr (CAP) {
        float big = 0.f;
#pragma unroll
        for (int j = 0; j < 128; j += 2) {
          const uint64_t v = mul2(pair(s[j], s[j + 1]), pair(scale2, scale2));
          asm("mov.b64 {%0, %1}, %2;" : "=f"(s[j]), "=f"(s[j + 1]) : "l"(v));
          big = fmaxf(big, fmaxf(fabsf(s[j]), fabsf(s[j + 1])));
        }
        if (__any_sync(0xffffffffu, big > CAP_POLY * cap2)) {
#pragma unroll
          for (int j = 0; j < 128; ++j) s[j] = cap_any(s[j], cap2, inv_cap2);
        } else {
#pragma unroll
          for (int j = 0; j < 128; j += 2) cap_small2(s + j, inv_cap2);
        }
      }
      if (KEEP && kept > 0) {
        const int behind = row_pos + tid - key0 - reach;  // columns up to this one are behind the window
#pragma unroll
        for (int j = 0; j < 128; ++j)
          if (j >= kept && j <= behind) s[j] = -INFINITY;
      }
#pragma unroll
      for (int j = 0; j < 128; ++j) {
        s[j] = CAP ? s[j] + tb[tid - j + 127] : fmaf(s[j], scale2, tb[tid - j + 127]);
        m_tile = fmaxf(m_tile, s[j]);
      }
      const float m_new = fmaxf(m_ref, m_tile);
      if (i == 0) {
        m_ref = m_new;
      } else if (__any_sync(0xffffffffu, m_new > m_ref + 8.f)) {
        // exponents stay relative to m_ref until some row's maximum has grown by more than 8 (x 256)
        ok = mbar_wait_bounded(o_done, (i - 1) & 1, abort_flag, err);
        if (!__all_sync(0xffffffffu, ok)) {
          ok = false;
          continue;
        }
        tc_fence_after();
        const float f = m_new > m_ref ? exp2f(m_ref - m_new) : 1.f;
        m_ref = m_new;
        l *= f;
#pragma unroll 1
        for (int c = 0; c < DVP / 32; ++c) {
          uint32_t r[32];
          tmem_ld32(tmem_O + lane_off + c * 32, r);
          tmem_wait_ld();
#pragma unroll
          for (int j = 0; j < 32; ++j) r[j] = __float_as_uint(__uint_as_float(r[j]) * f);
          tmem_st32(tmem_O + lane_off + c * 32, r);
        }
        tmem_wait_st();
      }
      const float m_safe = m_ref == -INFINITY ? 0.f : m_ref;
      uint32_t hi[32], lo[32];
#pragma unroll
      for (int c = 0; c < 2; ++c) {
#pragma unroll
        for (int j = 0; j < 32; ++j) {
          const float p0 = exp2f(s[c * 64 + 2 * j] - m_safe), p1 = exp2f(s[c * 64 + 2 * j + 1] - m_safe);
          l += p0 + p1;
          hi[j] = split_bf16(p0, p1, &lo[j]);
        }
        tmem_st32(S + c * 32, hi);
        tmem_st32(S + 64 + c * 32, lo);
      }
      tmem_wait_st();
      tc_fence_before();
      mbar_arrive(p_ready);
    }
    if (ok) ok = mbar_wait_bounded(o_done, (n - 1) & 1, abort_flag, err);
    if (__all_sync(0xffffffffu, ok)) {
      tc_fence_after();
      const bool valid = qt * 128 + tid < q_len;
      if (a.sink && m_ref != -INFINITY) l += exp2f(-m_ref);
      float inv = l > 0.f ? a.out_scale / l : 0.f;
      if (a.gate && valid)
        inv *= sigmoid_f(__bfloat162float(static_cast<const __nv_bfloat16*>(a.gate)[static_cast<size_t>(q0 + qt * 128 + tid) * a.ldg + head]));
      __nv_bfloat16* orow = static_cast<__nv_bfloat16*>(a.out) + static_cast<size_t>(q0 + qt * 128 + tid) * a.ldo +
                            head * a.dv;
#pragma unroll 1
      for (int c = 0; c < DVP / 32; ++c) {
        uint32_t r[32];
        tmem_ld32(tmem_O + lane_off + c * 32, r);
        tmem_wait_ld();
#pragma unroll
        for (int j = 0; j < 32; j += 8) {
          float f[8];
#pragma unroll
          for (int u = 0; u < 8; ++u) f[u] = __uint_as_float(r[j + u]) * inv;
          if (valid && c * 32 + j < a.dv) store_n<8>(orow + c * 32 + j, f);
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(tmem_S, 512);
  }
}

// The tensor maps of a layer's cache: pages of 16 keys (values) of one head, 64 columns at a time.
static int cache_maps(const WindowAttnArgs& a, int num_blocks, CUtensorMap* tk, CUtensorMap* tv) {
  const uint32_t box[3] = {64, WP_PAGE, 1};
  const uint64_t rows = static_cast<uint64_t>(a.hk) * a.bs, blk = a.block_elems() * 2;
  for (int which = 0; which < (a.shared ? 1 : 2); ++which) {
    const uint64_t cols = which ? a.dv : a.d;
    const uint64_t dims[3] = {cols, rows, static_cast<uint64_t>(num_blocks)};
    const uint64_t str[2] = {cols * 2, blk};
    const void* base = static_cast<const char*>(a.cache) + (which ? a.v_off() * 2 : 0);
    if (make_tmap_nd(which ? tv : tk, base, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, dims, str, box, CU_TENSOR_MAP_SWIZZLE_128B))
      return -3;
  }
  if (a.shared) *tv = *tk;
  return 0;
}

template <int DP, int DVP, bool SHARED, bool KEEP, bool CAP>
static int launch_prefill(const WindowAttnArgs& a, int total_tokens, int num_blocks, int seq_base, int num_seqs,
                          int max_q, cudaStream_t st) {
  using L_ = WindowPrefillSmem<DP, DVP, SHARED>;
  CUtensorMap tq, tk, tv;
  {
    const uint64_t dims[3] = {static_cast<uint64_t>(a.d), static_cast<uint64_t>(a.h), static_cast<uint64_t>(total_tokens)};
    const uint64_t str[2] = {static_cast<uint64_t>(a.d) * 2, static_cast<uint64_t>(a.ldq) * 2};
    const uint32_t box[3] = {64, 1, 128};
    if (make_tmap_nd(&tq, a.q, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, dims, str, box, CU_TENSOR_MAP_SWIZZLE_128B)) return -2;
  }
  if (int rc = cache_maps(a, num_blocks, &tk, &tv)) return rc;
  auto kern = window_prefill_kernel<DP, DVP, SHARED, KEEP, CAP>;
  if (KSANA_SMEM_ONCE(kern, L_::TOTAL) != 0) return -4;
  kern<<<dim3((max_q + 127) / 128, num_seqs, a.h), 160, L_::TOTAL, st>>>(tq, tk, tv, tk, a, seq_base, error_word());
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

// d, dv: a head's unrotated key and value sizes; kv: [rows][h * d | h * dv] (pitch ldkv); rot: [rows][rd] (pitch ldr)
template <int DP, int DVP>
static int launch_latent(const WindowAttnArgs& a, int total_tokens, const void* kv, int ldkv, const void* rot, int ldr,
                         int rd, int rows, int seq_base, int num_seqs, int max_q, cudaStream_t st) {
  using L_ = WindowPrefillSmem<DP, DVP, false>;
  CUtensorMap tq, tk, tv, tr;
  auto heads_map = [&](CUtensorMap* m, const void* base, int cols, int pitch, int count) {
    const uint64_t dims[3] = {static_cast<uint64_t>(cols), static_cast<uint64_t>(a.h), static_cast<uint64_t>(count)};
    const uint64_t str[2] = {static_cast<uint64_t>(cols) * 2, static_cast<uint64_t>(pitch) * 2};
    const uint32_t box[3] = {64, 1, 128};
    return make_tmap_nd(m, base, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, dims, str, box, CU_TENSOR_MAP_SWIZZLE_128B);
  };
  if (heads_map(&tq, a.q, a.d + rd, a.ldq, total_tokens) || heads_map(&tk, kv, a.d, ldkv, rows) ||
      heads_map(&tv, static_cast<const char*>(kv) + static_cast<size_t>(a.h) * a.d * 2, a.dv, ldkv, rows))
    return -2;
  if (make_tmap_2d(&tr, rot, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, rows, rd, ldr, 128, 64, CU_TENSOR_MAP_SWIZZLE_128B))
    return -3;
  auto kern = window_prefill_kernel<DP, DVP, false, false, false, true>;
  if (KSANA_SMEM_ONCE(kern, L_::TOTAL) != 0) return -4;
  kern<<<dim3((max_q + 127) / 128, num_seqs, a.h), 160, L_::TOTAL, st>>>(tq, tk, tv, tr, a, seq_base, error_word());
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

// ---- one new token: mma.sync over pages streamed through shared memory --------------------------------------------------
// One CTA of 4 warps = (sequence, key / value head, split of the visible pages); the splits of a head form a cluster
// and merge through distributed shared memory. Every warp streams its own 16-key pages: one lane keeps a ring of them
// in flight with TMA, the warp multiplies. Keys are the rows of the products and the (up to 8 NT) query heads that share
// the key head their columns:
//   S^T = K Q^T     16 keys x 8 NT heads, K by ldmatrix
//   O^T += V^T P^T  V^T by ldmatrix.trans, P^T = P transposed in registers, as two bf16 matrices hi + lo
// so nothing is computed for more than 8 NT - heads columns of padding. SHARED: values are keys, both products read the
// same page. Head sizes below DP / DVP are filled up with zeros by TMA. The kernel is a stream over the cache; the tensor
// instructions only keep the arithmetic out of its way.
template <int DP, int DVP, bool SHARED>
struct WindowDecodeSmem {
  static constexpr int K_BYTES = 16 * DP * 2;
  static constexpr int PAGE = K_BYTES + (SHARED ? 0 : 16 * DVP * 2);
  static constexpr int STAGES = PAGE <= 2048 ? 4 : PAGE <= 4096 ? 3 : 2;
  static constexpr int RING = 4 * STAGES * PAGE;
  static constexpr int LDO = DVP + 4;
  static constexpr int MERGE = 4 * 16 * LDO * 4;  // over the ring, once every page has been multiplied
  static constexpr int TOTAL = (RING > MERGE ? RING : MERGE) + 1024;
};

template <int DP, int DVP, int NT, bool SHARED>
__global__ void __launch_bounds__(128)
window_decode_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV, WindowAttnArgs a,
                     int seq_base, int groups, unsigned int* err) {
  using L_ = WindowDecodeSmem<DP, DVP, SHARED>;
  constexpr int STAGES = L_::STAGES, LDO = L_::LDO;
  extern __shared__ uint8_t smem_raw[];
  __shared__ uint64_t full[4][STAGES];
  __shared__ float sM[4][16], sL[4][16], cM[16], cL[16];
  __shared__ int abort_word;
  volatile int* abort_flag = &abort_word;
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int splits = gridDim.x, split = blockIdx.x;
  const int kh = blockIdx.y / groups, hpart = blockIdx.y % groups;
  const int b = blockIdx.z + seq_base;
  const int gq = a.h / a.hk;
  const int head0 = kh * gq + hpart * 8 * NT;
  const int g = min(8 * NT, gq - hpart * 8 * NT);  // query heads of this CTA
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int r = lane >> 2, j2 = (lane & 3) * 2;

  const int t = a.cu_q[b];
  const int pos = a.kv_lens[b] - 1;
  const int lo = a.window_start(pos);
  const int p0 = lo >> 4;
  const int n_kept = min((a.keep >> 4) + ((a.keep & 15) != 0), p0);  // pages of kept tokens ahead of the window's
  const int pages = n_kept + (pos >> 4) - p0 + 1;
  const int per = (pages + splits - 1) / splits;
  const int first = split * per + warp, last = min(split * per + per, pages);
  const int count = first < last ? (last - first + 3) / 4 : 0;  // of this warp
  const int* bt = a.block_tables + static_cast<size_t>(b) * a.max_blocks;
  auto page = [&](int n) {
    const int i = first + 4 * n;
    return i < n_kept ? i : p0 + i - n_kept;
  };

  if (tid == 0) {
    for (int w = 0; w < 4; ++w)
      for (int s = 0; s < STAGES; ++s) mbar_init(&full[w][s], 1);
    abort_word = 0;
    fence_mbar_init();
  }
  __syncthreads();

  uint8_t* ring = smem + warp * STAGES * L_::PAGE;
  int my_block = 0, issued = 0;  // lane l holds the block of this warp's page 32 c + l
  auto issue = [&](int n) {
    if ((n & 31) == 0) my_block = n + lane < count ? bt[page(n + lane)] : 0;
    const int blk = __shfl_sync(0xffffffffu, my_block, n & 31);
    if (lane == 0) {
      uint8_t* dst = ring + (n % STAGES) * L_::PAGE;
      uint64_t* bar = &full[warp][n % STAGES];
      mbar_expect_tx(bar, L_::PAGE);
#pragma unroll
      for (int hf = 0; hf < DP / 64; ++hf) tma_load_3d(dst + hf * 2048, &tmK, bar, hf * 64, kh * 16, blk);
      if constexpr (!SHARED) {
#pragma unroll
        for (int hf = 0; hf < DVP / 64; ++hf)
          tma_load_3d(dst + L_::K_BYTES + hf * 2048, &tmV, bar, hf * 64, kh * 16, blk);
      }
    }
    issued = n + 1;
  };
  for (int n = 0; n < STAGES && n < count; ++n) issue(n);

  uint32_t qf[DP / 16][NT][2];
#pragma unroll
  for (int nt = 0; nt < NT; ++nt) {
    const int hd = nt * 8 + r;
    const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q) + static_cast<size_t>(t) * a.ldq + (head0 + hd) * a.d;
#pragma unroll
    for (int kb = 0; kb < DP / 16; ++kb)
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int c = kb * 16 + u * 8 + j2;
        qf[kb][nt][u] = hd < g && c < a.d ? *reinterpret_cast<const uint32_t*>(q + c) : 0u;
      }
  }
  const float scale2 = a.scale * 1.4426950408889634f;
  const float cap2 = a.softcap * 1.4426950408889634f, inv_cap2 = a.softcap > 0.f ? 1.f / cap2 : 0.f;
  float acc[DVP / 16][NT][4];
#pragma unroll
  for (int i = 0; i < DVP / 16; ++i)
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int u = 0; u < 4; ++u) acc[i][nt][u] = 0.f;
  float m[NT][2], l[NT][2];  // of heads nt * 8 + j2 + {0, 1}; l: this thread's keys only
#pragma unroll
  for (int nt = 0; nt < NT; ++nt) m[nt][0] = m[nt][1] = -INFINITY, l[nt][0] = l[nt][1] = 0.f;

  // this lane's row and 16-byte column of the four 8 x 8 matrices of an ldmatrix
  const int k_row = (lane & 7) + (lane & 8), k_col = lane >> 4;
  const int v_row = (lane & 7) + ((lane >> 4) << 3), v_col = (lane >> 3) & 1;
  bool ok = true;
  for (int n = 0; n < count; ++n) {
    ok = mbar_wait_bounded(&full[warp][n % STAGES], (n / STAGES) & 1, abort_flag, err);
    if (!__all_sync(0xffffffffu, ok)) {
      ok = false;
      // copies in flight still write to this CTA's memory: give them their (bounded) time before leaving
      for (int i = n; i < issued; ++i)
        for (int it = 0; it < (1 << 20) && !mbar_try_wait(&full[warp][i % STAGES], (i / STAGES) & 1); ++it) {}
      break;
    }
    const uint32_t kb0 = smem_u32(ring + (n % STAGES) * L_::PAGE), vb0 = kb0 + (SHARED ? 0 : L_::K_BYTES);
    float c[NT][4];
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int u = 0; u < 4; ++u) c[nt][u] = 0.f;
#pragma unroll
    for (int kb = 0; kb < DP / 16; ++kb) {
      uint32_t f[4];
      const int ch = kb * 2 + k_col;
      ldmatrix_x4<false>(f, kb0 + (ch >> 3) * 2048 + k_row * 128 + (((ch & 7) ^ (k_row & 7)) << 4));
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) mma_16816(c[nt], f, qf[kb][nt][0], qf[kb][nt][1]);
    }
    const int key0 = page(n) * 16 + r;
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int key = key0 + u * 8;
      const bool seen = (key >= lo || key < a.keep) && key <= pos;
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float s = c[nt][u * 2 + e] * scale2;
          if (a.softcap > 0.f) s = cap_any(s, cap2, inv_cap2);
          if (a.bias) {
            const int hd = min(nt * 8 + j2 + e, g - 1);
            const float* bias = a.bias + static_cast<size_t>(head0 + hd) * a.bias_len;
            if (seen) s = fmaf(bias[min(pos - key, a.bias_len - 1)], 1.4426950408889634f, s);
          }
          c[nt][u * 2 + e] = seen ? s : -INFINITY;
        }
    }
    float mx[NT][2];
    bool grown = false;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        float v = fmaxf(c[nt][e], c[nt][2 + e]);
        v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 4));
        v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 8));
        v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 16));
        mx[nt][e] = fmaxf(v, m[nt][e]);  // finite: every page of the range holds a visible key
        grown = grown || mx[nt][e] > m[nt][e] + 8.f;
      }
    if (__any_sync(0xffffffffu, grown)) {
      // exponents stay relative to m until some head's maximum has grown by more than 8 (x 256)
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float f = exp2f(m[nt][e] - mx[nt][e]);
          m[nt][e] = mx[nt][e];
          l[nt][e] *= f;
#pragma unroll
          for (int i = 0; i < DVP / 16; ++i) {
            acc[i][nt][e] *= f;
            acc[i][nt][2 + e] *= f;
          }
        }
    }
    uint32_t ph[NT][2], pl[NT][2];
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const float x = exp2f(c[nt][u * 2] - m[nt][0]), y = exp2f(c[nt][u * 2 + 1] - m[nt][1]);
        l[nt][0] += x;
        l[nt][1] += y;
        uint32_t low;
        ph[nt][u] = transpose_8x8(split_bf16(x, y, &low));
        pl[nt][u] = transpose_8x8(low);
      }
#pragma unroll
    for (int i = 0; i < DVP / 16; ++i) {
      uint32_t f[4];
      const int ch = i * 2 + v_col;
      ldmatrix_x4<true>(f, vb0 + (ch >> 3) * 2048 + v_row * 128 + (((ch & 7) ^ (v_row & 7)) << 4));
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        mma_16816(acc[i][nt], f, ph[nt][0], ph[nt][1]);
        mma_16816(acc[i][nt], f, pl[nt][0], pl[nt][1]);
      }
    }
    __syncwarp();  // every lane has read this page
    if (n + STAGES < count) issue(n + STAGES);
  }
  __syncthreads();  // the ring is free: the warps' parts go over it
  float* sO = reinterpret_cast<float*>(smem);  // [4][g][LDO]
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      float s = l[nt][e];
      s += __shfl_xor_sync(0xffffffffu, s, 4);
      s += __shfl_xor_sync(0xffffffffu, s, 8);
      s += __shfl_xor_sync(0xffffffffu, s, 16);
      const int hd = nt * 8 + j2 + e;
      if (hd < g) {
        if (r == 0) {
          sM[warp][hd] = m[nt][e];
          sL[warp][hd] = s;
        }
        float* dst = sO + (warp * g + hd) * LDO + r;
#pragma unroll
        for (int i = 0; i < DVP / 16; ++i) {
          dst[i * 16] = acc[i][nt][e];
          dst[i * 16 + 8] = acc[i][nt][2 + e];
        }
      }
    }
  __syncthreads();
  // the four warps' parts -> one per CTA, in place of warp 0's
  if (tid < g) {
    float M = -INFINITY, S = 0.f;
    for (int w = 0; w < 4; ++w) M = fmaxf(M, sM[w][tid]);
    for (int w = 0; w < 4; ++w) {
      const float f = M == -INFINITY ? 0.f : exp2f(sM[w][tid] - M);
      S += sL[w][tid] * f;
      sL[w][tid] = f;  // from here on the warp's weight
    }
    cM[tid] = M;
    cL[tid] = S;
  }
  __syncthreads();
  const int quads = a.dv / 4;
  for (int e = tid; e < g * quads; e += 128) {
    const int hd = e / quads, col = e % quads * 4;
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int w = 0; w < 4; ++w) {
      const float f = sL[w][hd];
      const float4 v = *reinterpret_cast<const float4*>(sO + (w * g + hd) * LDO + col);
      s.x += f * v.x; s.y += f * v.y; s.z += f * v.z; s.w += f * v.w;
    }
    *reinterpret_cast<float4*>(sO + hd * LDO + col) = s;  // only this thread reads or writes these elements of warp 0's part
  }
  __syncwarp();
  if (splits > 1)
    cluster_sync_all();
  else
    __syncthreads();
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + static_cast<size_t>(t) * a.ldo + head0 * a.dv;
  for (int e = split * 128 + tid; e < g * quads; e += splits * 128) {
    const int hd = e / quads, col = e % quads * 4;
    float M = -INFINITY, S = 0.f, o[4] = {0.f, 0.f, 0.f, 0.f};
    if (splits == 1) {
      M = cM[hd];
      S = cL[hd];
      const float4 v = *reinterpret_cast<const float4*>(sO + hd * LDO + col);
      o[0] = v.x; o[1] = v.y; o[2] = v.z; o[3] = v.w;
    } else {
      for (int s = 0; s < splits; ++s) M = fmaxf(M, ld_cluster_f1(mapa_u32(smem_u32(cM + hd), s)));
      for (int s = 0; s < splits; ++s) {
        const float f = exp2f(ld_cluster_f1(mapa_u32(smem_u32(cM + hd), s)) - M);
        S += f * ld_cluster_f1(mapa_u32(smem_u32(cL + hd), s));
        const float4 v = ld_cluster_f4(mapa_u32(smem_u32(sO + hd * LDO + col), s));
        o[0] += f * v.x; o[1] += f * v.y; o[2] += f * v.z; o[3] += f * v.w;
      }
    }
    if (a.sink) S += exp2f(-M);
    float inv = a.out_scale / S;
    if (a.gate) inv *= sigmoid_f(__bfloat162float(static_cast<const __nv_bfloat16*>(a.gate)[static_cast<size_t>(t) * a.ldg + head0 + hd]));
#pragma unroll
    for (int u = 0; u < 4; ++u) o[u] *= inv;
    store_n<4>(out + hd * a.dv + col, o);
  }
  __syncwarp();
  if (splits > 1) cluster_sync_all();  // nobody leaves while its memory is still read
}

template <int DP, int DVP, int NT, bool SHARED>
static int launch_decode(const WindowAttnArgs& a, int num_blocks, int seq_base, int num_seqs, int max_kv,
                         cudaStream_t st) {
  using L_ = WindowDecodeSmem<DP, DVP, SHARED>;
  const int gq = a.h / a.hk, groups = (gq + 8 * NT - 1) / (8 * NT);
  CUtensorMap tk, tv;
  if (int rc = cache_maps(a, num_blocks, &tk, &tv)) return rc;
  auto kern = window_decode_kernel<DP, DVP, NT, SHARED>;
  if (KSANA_SMEM_ONCE(kern, L_::TOTAL) != 0) return -4;
  const int keys = a.window > 0 && a.window < max_kv - a.keep ? a.window + a.keep : max_kv;
  const int pages = keys / 16 + 1;
  const long long base = static_cast<long long>(num_seqs) * a.hk * groups;
  // enough CTAs for a few waves of what the SMs hold (whose last one is then short), as long as a warp gets some pages
  int splits = 1;
  while (splits < 8 && base * splits < 8 * sm_count() && pages / (splits * 2) >= 8) splits *= 2;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(splits, a.hk * groups, num_seqs);
  cfg.blockDim = dim3(128);
  cfg.dynamicSmemBytes = L_::TOTAL;
  cfg.stream = st;
  cudaLaunchAttribute at[1];
  at[0].id = cudaLaunchAttributeClusterDimension;
  at[0].val.clusterDim.x = splits;
  at[0].val.clusterDim.y = at[0].val.clusterDim.z = 1;
  cfg.attrs = at;
  cfg.numAttrs = 1;
  return cudaLaunchKernelEx(&cfg, kern, tk, tv, a, seq_base, groups, error_word()) == cudaSuccess ? 0 : -5;
}

static bool rows16(const void* p, int ld) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0 && (ld & 7) == 0; }

}  // namespace ksana

using namespace ksana;

// bf16. Sequences [seq_base, seq_base + num_seqs), each with at most max_q new tokens. Returns -1 for sizes it does not
// take (heads of at most 128 dimensions in multiples of 8, pages of 16 tokens, 16-byte aligned rows).
KSANA_API int ksana_window_prefill(const void* q, int ldq, int total_tokens, const void* cache, int num_blocks,
                                   const int* block_tables, int max_blocks, const int* cu_q, const int* kv_lens, int h,
                                   int hk, int d, int dv, int bs, int window, int keep, int shared, float scale,
                                   const float* bias, int bias_len, float out_scale, float softcap, int sink,
                                   const void* gate, int ldg, void* out, int ldo, int seq_base, int num_seqs, int max_q,
                                   cudaStream_t st) {
  if (num_seqs <= 0 || max_q <= 0) return 0;
  if (keep < 0 || (shared && d != dv)) return -2;
  if (h % hk || bs != WP_PAGE || d > 128 || dv > 128 || (d & 7) || (dv & 7) || !rows16(q, ldq) || !rows16(cache, 0) ||
      !rows16(out, ldo))
    return -1;
  WindowAttnArgs a{q, ldq, cache, block_tables, max_blocks, cu_q, kv_lens, nullptr, h, hk, d, dv, bs, window, keep,
                   shared, scale, bias, bias_len, out_scale, out, ldo, softcap, sink, gate, ldg};
  if (softcap > 0.f && (keep || shared)) return -1;
#define KSANA_WP(DP, DVP, SHARED)                                                                                      \
  return keep ? launch_prefill<DP, DVP, SHARED, true, false>(a, total_tokens, num_blocks, seq_base, num_seqs, max_q, st) \
         : softcap > 0.f                                                                                               \
             ? launch_prefill<DP, DVP, SHARED, false, !SHARED>(a, total_tokens, num_blocks, seq_base, num_seqs, max_q, st) \
             : launch_prefill<DP, DVP, SHARED, false, false>(a, total_tokens, num_blocks, seq_base, num_seqs, max_q, st)
  if (shared) {
    if (d <= 64) KSANA_WP(64, 64, true);
    KSANA_WP(128, 128, true);
  }
  if (d <= 64 && dv <= 64) KSANA_WP(64, 64, false);
  if (d <= 64) KSANA_WP(64, 128, false);
  if (dv <= 64) KSANA_WP(128, 64, false);
  KSANA_WP(128, 128, false);
#undef KSANA_WP
}

// bf16. Sequences [seq_base, seq_base + num_seqs) with exactly one new token each. Returns -1 for sizes it does not
// take (heads of at most 128 dimensions in multiples of 8, pages of 16 tokens, 16-byte aligned rows).
KSANA_API int ksana_window_decode(const void* q, int ldq, const void* cache, int num_blocks, const int* block_tables,
                                  int max_blocks, const int* cu_q, const int* kv_lens, int h, int hk, int d, int dv,
                                  int bs, int window, int keep, int shared, float scale, const float* bias, int bias_len,
                                  float out_scale, float softcap, int sink, const void* gate, int ldg, void* out,
                                  int ldo, int seq_base, int num_seqs, int max_kv, cudaStream_t st) {
  if (num_seqs <= 0) return 0;
  if (keep < 0 || (shared && d < dv)) return -2;
  if (h % hk || bs != WP_PAGE || d > 128 || dv > 128 || (shared && d != dv) || (d & 7) || (dv & 7) || !rows16(q, ldq) || !rows16(cache, 0) ||
      !rows16(out, ldo))
    return -1;
  WindowAttnArgs a{q, ldq, cache, block_tables, max_blocks, cu_q, kv_lens, nullptr, h, hk, d, dv, bs, window, keep,
                   shared, scale, bias, bias_len, out_scale, out, ldo, softcap, sink, gate, ldg};
#define KSANA_WD(DP, DVP, SHARED)                                                                             \
  return h / hk <= 8 ? launch_decode<DP, DVP, 1, SHARED>(a, num_blocks, seq_base, num_seqs, max_kv, st)       \
                     : launch_decode<DP, DVP, 2, SHARED>(a, num_blocks, seq_base, num_seqs, max_kv, st)
  if (shared) {
    if (d <= 64) KSANA_WD(64, 64, true);
    KSANA_WD(128, 128, true);
  }
  if (d <= 64 && dv <= 64) KSANA_WD(64, 64, false);
  if (d <= 64) KSANA_WD(64, 128, false);
  if (dv <= 64) KSANA_WD(128, 64, false);
  KSANA_WD(128, 128, false);
#undef KSANA_WD
}

// Prompts over keys and values that were written out of latents (see launch_latent). bf16; -1 for sizes it does not take.
KSANA_API int ksana_latent_prefill(const void* q, int ldq, int total_tokens, const void* kv, int ldkv, const void* rot,
                                   int ldr, int rows, const int* cu_q, const int* kv_lens, int h, int d, int rd, int dv,
                                   float scale, const void* gate, int ldg, void* out, int ldo, int seq_base, int num_seqs,
                                   int max_q, cudaStream_t st) {
  if (num_seqs <= 0 || max_q <= 0) return 0;
  if (d > 128 || dv > 128 || rd > 64 || (d & 7) || (dv & 7) || (rd & 7) || !rows16(q, ldq) || !rows16(kv, ldkv) ||
      !rows16(rot, ldr) || !rows16(out, ldo))
    return -1;
  WindowAttnArgs a{q, ldq, nullptr, nullptr, 0, cu_q, kv_lens, nullptr, h, h, d, dv, WP_PAGE, 0, 0, 0, scale, nullptr, 0,
                   1.f, out, ldo, 0.f, 0, gate, ldg};
#define KSANA_LP(DP, DVP) \
  return launch_latent<DP, DVP>(a, total_tokens, kv, ldkv, rot, ldr, rd, rows, seq_base, num_seqs, max_q, st)
  if (d <= 64 && dv <= 64) KSANA_LP(128, 64);
  if (d <= 64) KSANA_LP(128, 128);
  if (dv <= 64) KSANA_LP(192, 64);
  KSANA_LP(192, 128);
#undef KSANA_LP
}

// Tokens [tok_base, tok_base + tokens) of the step, whatever sequences they belong to. kind: 0 fp32, 1 bf16.
KSANA_API int ksana_window_attention_any(const void* q, int ldq, const void* cache, const int* block_tables,
                                         int max_blocks, const int* cu_q, const int* kv_lens, const int* seq_of_token,
                                         int h, int hk, int d, int dv, int bs, int window, int keep, int shared,
                                         float scale, const float* bias, int bias_len, float out_scale, float softcap,
                                         int sink, const void* gate, int ldg, void* out, int ldo, int tok_base,
                                         int tokens, int kind, cudaStream_t st) {
  if (tokens <= 0) return 0;
  if (h % hk || keep < 0 || (shared && d < dv)) return -2;
  WindowAttnArgs a{q, ldq, cache, block_tables, max_blocks, cu_q, kv_lens, seq_of_token, h, hk, d, dv, bs, window, keep,
                   shared, scale, bias, bias_len, out_scale, out, ldo, softcap, sink, gate, ldg};
  return kind ? launch_any<__nv_bfloat16>(a, tok_base, tokens, st) : launch_any<float>(a, tok_base, tokens, st);
}
