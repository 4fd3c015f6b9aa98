// Attention over the paged cache of layers with sizes of their own: a sliding window, first tokens that stay visible
// behind it, a learned bias per distance, key / value heads of different sizes, or values that are the keys. Scores,
// softmax and the accumulation are 32-bit.
//
// Cache of a layer: [block][keys hk x bs x d | values hk x bs x dv], the second part only where values are not the keys.
// bias: [h][bias_len] fp32 (null: none), indexed by the distance between query and key.
//
// Query i sees key j when j <= i and (i - j < window or j < keep); window 0: every j <= i.
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
  int h, hk, d, dv, bs, window, keep, shared;  // shared: values are the keys (dv == d)
  float scale;
  const float* bias;
  int bias_len;
  float out_scale;
  void* out;
  int ldo;
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
      float dot = 0.f;
      for (int c = 0; c < a.d; ++c) dot += sq[c] * to_f(kp[c]);
      s = dot * a.scale;
      if (bias) s += bias[min(pos - j, a.bias_len - 1)];
    }
    const float m_new = fmaxf(m, warp_max(s));
    const float f = expf(m - m_new);
    const float p = i < n ? expf(s - m_new) : 0.f;
    l = l * f + warp_sum(p);
    m = m_new;
#pragma unroll
    for (int i = 0; i < NV; ++i) acc[i] *= f;
    const int count = min(32, n - i0);
    for (int u = 0; u < count; ++u) {
      const float pu = __shfl_sync(0xffffffffu, p, u);
      const int ju = i0 + u < kept ? i0 + u : lo + i0 + u - kept;
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

template <int DP, int DVP, bool SHARED>
__global__ void __launch_bounds__(160, 1)
window_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                      const __grid_constant__ CUtensorMap tmV, WindowAttnArgs a, int seq_base, unsigned int* err) {
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
  const int n_kept = min(a.keep / 128 + (a.keep % 128 != 0), kt0);  // tiles of kept tokens ahead of the window's
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
      auto load_k = [&](int i) { load(tmK, sK, L_::K_BYTES, DP / 64, k_full, i, i % STAGES); k_loads = i + 1; };
      auto load_v = [&](int i) { load(tmV, sV, L_::V_BYTES, DVP / 64, v_full, i, i & 1); v_loads = i + 1; };
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
      for (int hf = 0; hf < DP / 64; ++hf) tma_load_3d(sQ + hf * (128 * 128), &tmQ, q_bar, hf * 64, head, q0 + qt * 128);
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
    const float* bias = a.bias ? a.bias + static_cast<size_t>(head) * a.bias_len : nullptr;
    const int reach = a.window > 0 ? min(a.window, 1 << 30) : 1 << 30;
    float m_ref = -INFINITY, l = 0.f;
    bool ok = true;
    for (int i = 0; i < n; ++i) {
      float* tb = tab + (i & 1) * 256;
      const int key0 = tile(i) * 128;
      const int d0 = row_pos - key0 - 127;   // distance of entry 0
      const int kept = a.keep - key0;        // columns below this one are kept tokens
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
      if (kept > 0) {
        const int behind = row_pos + tid - key0 - reach;  // columns up to this one are behind the window
#pragma unroll
        for (int j = 0; j < 128; ++j)
          if (j >= kept && j <= behind) s[j] = -INFINITY;
      }
#pragma unroll
      for (int j = 0; j < 128; ++j) {
        s[j] = fmaf(s[j], scale2, tb[tid - j + 127]);
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
      const float inv = l > 0.f ? a.out_scale / l : 0.f;
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

template <int DP, int DVP, bool SHARED = false>
static int launch_prefill(const WindowAttnArgs& a, int total_tokens, int num_blocks, int seq_base, int num_seqs,
                          int max_q, cudaStream_t st) {
  using L_ = WindowPrefillSmem<DP, DVP, SHARED>;
  CUtensorMap tq, tk, tv;
  const uint64_t blk = a.block_elems() * 2;
  const uint64_t d = a.d, dv = a.dv;
  {
    const uint64_t dims[3] = {d, static_cast<uint64_t>(a.h), static_cast<uint64_t>(total_tokens)};
    const uint64_t str[2] = {d * 2, static_cast<uint64_t>(a.ldq) * 2};
    const uint32_t box[3] = {64, 1, 128};
    if (make_tmap_nd(&tq, a.q, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, dims, str, box, CU_TENSOR_MAP_SWIZZLE_128B)) return -2;
  }
  const uint32_t box[3] = {64, WP_PAGE, 1};
  const uint64_t rows = static_cast<uint64_t>(a.hk) * a.bs;
  {
    const uint64_t dims[3] = {d, rows, static_cast<uint64_t>(num_blocks)};
    const uint64_t str[2] = {d * 2, blk};
    if (make_tmap_nd(&tk, a.cache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, dims, str, box, CU_TENSOR_MAP_SWIZZLE_128B)) return -3;
  }
  if (SHARED) {
    tv = tk;
  } else {
    const uint64_t dims[3] = {dv, rows, static_cast<uint64_t>(num_blocks)};
    const uint64_t str[2] = {dv * 2, blk};
    const void* base = static_cast<const char*>(a.cache) + a.v_off() * 2;
    if (make_tmap_nd(&tv, base, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, dims, str, box, CU_TENSOR_MAP_SWIZZLE_128B)) return -3;
  }
  auto kern = window_prefill_kernel<DP, DVP, SHARED>;
  if (KSANA_SMEM_ONCE(kern, L_::TOTAL) != 0) return -4;
  kern<<<dim3((max_q + 127) / 128, num_seqs, a.h), 160, L_::TOTAL, st>>>(tq, tk, tv, a, seq_base, error_word());
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

// ---- one new token: mma.sync over register-resident pages --------------------------------------------------------------
// One CTA of 4 warps = (sequence, key / value head, split of the visible pages); the splits of a head form a cluster
// and merge through distributed shared memory. A warp takes one 16-key page at a time: its K and V rows go straight
// from the cache into MMA fragments with 16-byte loads (dimensions and value columns are permuted the same way on both
// sides of each product, so no transposition is needed). The rows of the fragments are the query heads that share the
// key head. The kernel is a stream over the cache; the tensor instructions only keep the arithmetic out of its way.
__device__ __forceinline__ void mma_16816(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

template <int KD, int ND>  // d = 32 KD, dv = 64 ND
__global__ void __launch_bounds__(128)
window_decode_kernel(WindowAttnArgs a, int seq_base, int groups) {
  extern __shared__ float sm[];
  const int splits = gridDim.x, split = blockIdx.x;
  const int kh = blockIdx.y / groups, part = blockIdx.y % groups;
  const int b = blockIdx.z + seq_base;
  const int gq = a.h / a.hk;
  const int head0 = kh * gq + part * 16;
  const int g = min(16, gq - part * 16);        // query heads of this CTA
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int r = lane >> 2, j = lane & 3;
  constexpr int DV = ND * 64;
  float* sO = sm;                               // [4][g][DV]
  float* sM = sO + 4 * g * DV;                  // [4][16]
  float* sL = sM + 64;                          // [4][16]
  float* cM = sL + 64;                          // [16] of this CTA
  float* cL = cM + 16;

  const int t = a.cu_q[b];
  const int pos = a.kv_lens[b] - 1;
  const int lo = a.window_start(pos);
  const int p0 = lo >> 4;
  const int n_kept = min((a.keep >> 4) + ((a.keep & 15) != 0), p0);  // pages of kept tokens ahead of the window's
  const int pages = n_kept + (pos >> 4) - p0 + 1;
  const int per = (pages + splits - 1) / splits;
  const int first = split * per, last = min(first + per, pages);
  const int* bt = a.block_tables + static_cast<size_t>(b) * a.max_blocks;
  const __nv_bfloat16* cache = static_cast<const __nv_bfloat16*>(a.cache);
  const size_t block_elems = a.block_elems();
  const size_t k_off = static_cast<size_t>(kh) * 16 * a.d;
  const size_t v_off = a.v_off() + static_cast<size_t>(kh) * 16 * a.dv;

  uint32_t qf[2 * KD][4];
  {
    const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q) + static_cast<size_t>(t) * a.ldq + head0 * a.d;
#pragma unroll
    for (int kb = 0; kb < KD; ++kb) {
      uint4 x = make_uint4(0, 0, 0, 0), y = x;
      if (r < g) x = *reinterpret_cast<const uint4*>(q + r * a.d + kb * 32 + j * 8);
      if (r + 8 < g) y = *reinterpret_cast<const uint4*>(q + (r + 8) * a.d + kb * 32 + j * 8);
      qf[2 * kb][0] = x.x; qf[2 * kb][1] = y.x; qf[2 * kb][2] = x.y; qf[2 * kb][3] = y.y;
      qf[2 * kb + 1][0] = x.z; qf[2 * kb + 1][1] = y.z; qf[2 * kb + 1][2] = x.w; qf[2 * kb + 1][3] = y.w;
    }
  }
  const float scale2 = a.scale * 1.4426950408889634f;
  const float* bias0 = a.bias ? a.bias + static_cast<size_t>(head0 + min(r, g - 1)) * a.bias_len : nullptr;
  const float* bias1 = a.bias ? a.bias + static_cast<size_t>(head0 + min(r + 8, g - 1)) * a.bias_len : nullptr;
  float o[ND * 8][4];
#pragma unroll
  for (int i = 0; i < ND * 8; ++i)
#pragma unroll
    for (int u = 0; u < 4; ++u) o[i][u] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};

  for (int i = first + warp; i < last; i += 4) {
    const int pg = i < n_kept ? i : p0 + i - n_kept;
    const __nv_bfloat16* blk = cache + bt[pg] * block_elems;
    uint4 kf[2][KD], vf[4][ND];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int kb = 0; kb < KD; ++kb)
        kf[nt][kb] = *reinterpret_cast<const uint4*>(blk + k_off + (nt * 8 + r) * a.d + kb * 32 + j * 8);
#pragma unroll
    for (int u = 0; u < 4; ++u)
#pragma unroll
      for (int nb = 0; nb < ND; ++nb)
        vf[u][nb] = *reinterpret_cast<const uint4*>(blk + v_off + (j * 2 + (u & 1) + (u >> 1) * 8) * a.dv + nb * 64 + r * 8);
    float c[2][4];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
#pragma unroll
      for (int u = 0; u < 4; ++u) c[nt][u] = 0.f;
#pragma unroll
      for (int kb = 0; kb < KD; ++kb) {
        mma_16816(c[nt], qf[2 * kb], kf[nt][kb].x, kf[nt][kb].y);
        mma_16816(c[nt], qf[2 * kb + 1], kf[nt][kb].z, kf[nt][kb].w);
      }
    }
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int key = pg * 16 + nt * 8 + j * 2 + (u & 1);
        const float* bias = (u >> 1) ? bias1 : bias0;
        float s = -INFINITY;
        if ((key >= lo || key < a.keep) && key <= pos) {
          s = c[nt][u] * scale2;
          if (bias) s = fmaf(bias[min(pos - key, a.bias_len - 1)], 1.4426950408889634f, s);
        }
        c[nt][u] = s;
        mx[u >> 1] = fmaxf(mx[u >> 1], s);
      }
    float f[2];
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      mx[q] = fmaxf(mx[q], __shfl_xor_sync(0xffffffffu, mx[q], 1));
      mx[q] = fmaxf(mx[q], __shfl_xor_sync(0xffffffffu, mx[q], 2));
      mx[q] = fmaxf(mx[q], m[q]);  // finite: every page of the range holds a visible key
      f[q] = exp2f(m[q] - mx[q]);
      m[q] = mx[q];
      l[q] *= f[q];
    }
    uint32_t ph[4], pl[4];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        const float x = exp2f(c[nt][2 * q] - m[q]), y = exp2f(c[nt][2 * q + 1] - m[q]);
        l[q] += x + y;
        ph[nt * 2 + q] = split_bf16(x, y, &pl[nt * 2 + q]);
      }
#pragma unroll
    for (int nb = 0; nb < ND; ++nb) {
      const uint32_t* w0 = reinterpret_cast<const uint32_t*>(&vf[0][nb]);
      const uint32_t* w1 = reinterpret_cast<const uint32_t*>(&vf[1][nb]);
      const uint32_t* w2 = reinterpret_cast<const uint32_t*>(&vf[2][nb]);
      const uint32_t* w3 = reinterpret_cast<const uint32_t*>(&vf[3][nb]);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const uint32_t sel = (e & 1) ? 0x7632 : 0x5410;
        const uint32_t b0 = __byte_perm(w0[e >> 1], w1[e >> 1], sel), b1 = __byte_perm(w2[e >> 1], w3[e >> 1], sel);
        float* acc = o[nb * 8 + e];
        acc[0] *= f[0]; acc[1] *= f[0]; acc[2] *= f[1]; acc[3] *= f[1];
        mma_16816(acc, ph, b0, b1);
        mma_16816(acc, pl, b0, b1);
      }
    }
  }
#pragma unroll
  for (int q = 0; q < 2; ++q) {
    l[q] += __shfl_xor_sync(0xffffffffu, l[q], 1);
    l[q] += __shfl_xor_sync(0xffffffffu, l[q], 2);
    const int row = r + q * 8;
    if (row < g) {
      if (j == 0) {
        sM[warp * 16 + row] = m[q];
        sL[warp * 16 + row] = l[q];
      }
      float* dst = sO + (static_cast<size_t>(warp) * g + row) * DV;
#pragma unroll
      for (int nb = 0; nb < ND; ++nb)
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          float* p = dst + nb * 64 + (j * 2 + u) * 8;
          *reinterpret_cast<float4*>(p) = make_float4(o[nb * 8][q * 2 + u], o[nb * 8 + 1][q * 2 + u],
                                                      o[nb * 8 + 2][q * 2 + u], o[nb * 8 + 3][q * 2 + u]);
          *reinterpret_cast<float4*>(p + 4) = make_float4(o[nb * 8 + 4][q * 2 + u], o[nb * 8 + 5][q * 2 + u],
                                                          o[nb * 8 + 6][q * 2 + u], o[nb * 8 + 7][q * 2 + u]);
        }
    }
  }
  __syncthreads();
  // the four warps' parts -> one per CTA, in place of warp 0's
  if (tid < g) {
    float M = -INFINITY, S = 0.f;
    for (int w = 0; w < 4; ++w) M = fmaxf(M, sM[w * 16 + tid]);
    for (int w = 0; w < 4; ++w) {
      const float f = M == -INFINITY ? 0.f : exp2f(sM[w * 16 + tid] - M);
      S += sL[w * 16 + tid] * f;
      sL[w * 16 + tid] = f;  // from here on the warp's weight
    }
    cM[tid] = M;
    cL[tid] = S;
  }
  __syncthreads();
  for (int e = tid * 4; e < g * DV; e += 512) {
    const int row = e / DV;
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int w = 0; w < 4; ++w) {
      const float f = sL[w * 16 + row];
      const float4 v = *reinterpret_cast<const float4*>(sO + static_cast<size_t>(w) * g * DV + e);
      s.x += f * v.x; s.y += f * v.y; s.z += f * v.z; s.w += f * v.w;
    }
    *reinterpret_cast<float4*>(sO + e) = s;  // only this thread reads or writes these elements of warp 0's part
  }
  __syncwarp();
  if (splits > 1)
    cluster_sync_all();
  else
    __syncthreads();
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + static_cast<size_t>(t) * a.ldo + head0 * a.dv;
  for (int e = (split * 128 + tid) * 4; e < g * DV; e += splits * 512) {
    const int row = e / DV;
    float M = -INFINITY, S = 0.f, acc[4] = {0.f, 0.f, 0.f, 0.f};
    if (splits == 1) {
      S = cL[row];
      const float4 v = *reinterpret_cast<const float4*>(sO + e);
      acc[0] = v.x; acc[1] = v.y; acc[2] = v.z; acc[3] = v.w;
    } else {
      for (int s = 0; s < splits; ++s) M = fmaxf(M, ld_cluster_f1(mapa_u32(smem_u32(cM + row), s)));
      for (int s = 0; s < splits; ++s) {
        const float f = exp2f(ld_cluster_f1(mapa_u32(smem_u32(cM + row), s)) - M);
        S += f * ld_cluster_f1(mapa_u32(smem_u32(cL + row), s));
        const float4 v = ld_cluster_f4(mapa_u32(smem_u32(sO + e), s));
        acc[0] += f * v.x; acc[1] += f * v.y; acc[2] += f * v.z; acc[3] += f * v.w;
      }
    }
    const float inv = a.out_scale / S;
#pragma unroll
    for (int u = 0; u < 4; ++u) acc[u] *= inv;
    store_n<4>(out + row * a.dv + e % DV, acc);
  }
  __syncwarp();
  if (splits > 1) cluster_sync_all();  // nobody leaves while its memory is still read
}

template <int KD, int ND>
static int launch_decode(const WindowAttnArgs& a, int seq_base, int num_seqs, int max_kv, cudaStream_t st) {
  const int gq = a.h / a.hk, groups = (gq + 15) / 16, g = gq < 16 ? gq : 16;
  const int smem = static_cast<int>(sizeof(float)) * (4 * g * ND * 64 + 64 + 64 + 32);
  auto kern = window_decode_kernel<KD, ND>;
  if (KSANA_SMEM_ONCE(kern, 4 * 16 * ND * 64 * 4 + 1024) != 0) return -4;
  const int keys = a.window > 0 && a.window < max_kv - a.keep ? a.window + a.keep : max_kv;
  const int pages = keys / 16 + 1;
  const long long base = static_cast<long long>(num_seqs) * a.hk * groups;
  int splits = 1;
  while (splits < 8 && base * splits < 3 * sm_count() && pages / (splits * 2) >= 8) splits *= 2;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(splits, a.hk * groups, num_seqs);
  cfg.blockDim = dim3(128);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute at[1];
  at[0].id = cudaLaunchAttributeClusterDimension;
  at[0].val.clusterDim.x = splits;
  at[0].val.clusterDim.y = at[0].val.clusterDim.z = 1;
  cfg.attrs = at;
  cfg.numAttrs = 1;
  return cudaLaunchKernelEx(&cfg, kern, a, seq_base, groups) == cudaSuccess ? 0 : -5;
}

static bool rows16(const void* p, int ld) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0 && (ld & 7) == 0; }

}  // namespace ksana

using namespace ksana;

// bf16. Sequences [seq_base, seq_base + num_seqs), each with at most max_q new tokens. Returns -1 for sizes it does not
// take (heads of at most 128 dimensions in multiples of 8, pages of 16 tokens, 16-byte aligned rows).
KSANA_API int ksana_window_prefill(const void* q, int ldq, int total_tokens, const void* cache, int num_blocks,
                                   const int* block_tables, int max_blocks, const int* cu_q, const int* kv_lens, int h,
                                   int hk, int d, int dv, int bs, int window, int keep, int shared, float scale,
                                   const float* bias, int bias_len, float out_scale, void* out, int ldo, int seq_base,
                                   int num_seqs, int max_q, cudaStream_t st) {
  if (num_seqs <= 0 || max_q <= 0) return 0;
  if (keep < 0 || (shared && d != dv)) return -2;
  if (h % hk || bs != WP_PAGE || d > 128 || dv > 128 || (d & 7) || (dv & 7) || !rows16(q, ldq) || !rows16(cache, 0) ||
      !rows16(out, ldo))
    return -1;
  WindowAttnArgs a{q, ldq, cache, block_tables, max_blocks, cu_q, kv_lens, nullptr, h, hk, d, dv, bs, window, keep,
                   shared, scale, bias, bias_len, out_scale, out, ldo};
  if (shared)
    return d <= 64 ? launch_prefill<64, 64, true>(a, total_tokens, num_blocks, seq_base, num_seqs, max_q, st)
                   : launch_prefill<128, 128, true>(a, total_tokens, num_blocks, seq_base, num_seqs, max_q, st);
  if (d <= 64)
    return dv <= 64 ? launch_prefill<64, 64>(a, total_tokens, num_blocks, seq_base, num_seqs, max_q, st)
                    : launch_prefill<64, 128>(a, total_tokens, num_blocks, seq_base, num_seqs, max_q, st);
  return dv <= 64 ? launch_prefill<128, 64>(a, total_tokens, num_blocks, seq_base, num_seqs, max_q, st)
                  : launch_prefill<128, 128>(a, total_tokens, num_blocks, seq_base, num_seqs, max_q, st);
}

// bf16. Sequences [seq_base, seq_base + num_seqs) with exactly one new token each. Returns -1 for sizes it does not
// take (d = 32, 64, 96 or 128, dv = 64 or 128, pages of 16 tokens, 16-byte aligned rows).
KSANA_API int ksana_window_decode(const void* q, int ldq, const void* cache, const int* block_tables, int max_blocks,
                                  const int* cu_q, const int* kv_lens, int h, int hk, int d, int dv, int bs, int window,
                                  int keep, int shared, float scale, const float* bias, int bias_len, float out_scale,
                                  void* out, int ldo, int seq_base, int num_seqs, int max_kv, cudaStream_t st) {
  if (num_seqs <= 0) return 0;
  if (keep < 0 || (shared && d != dv)) return -2;
  if (h % hk || bs != 16 || (d & 31) || d > 128 || (dv & 63) || dv > 128 || !rows16(q, ldq) || !rows16(cache, 0) ||
      !rows16(out, ldo))
    return -1;
  WindowAttnArgs a{q, ldq, cache, block_tables, max_blocks, cu_q, kv_lens, nullptr, h, hk, d, dv, bs, window, keep,
                   shared, scale, bias, bias_len, out_scale, out, ldo};
#define KSANA_WD(KD) \
  case KD: return dv == 64 ? launch_decode<KD, 1>(a, seq_base, num_seqs, max_kv, st) \
                           : launch_decode<KD, 2>(a, seq_base, num_seqs, max_kv, st)
  switch (d / 32) {
    KSANA_WD(1);
    KSANA_WD(2);
    KSANA_WD(3);
    KSANA_WD(4);
  }
#undef KSANA_WD
  return -1;
}

// Tokens [tok_base, tok_base + tokens) of the step, whatever sequences they belong to. kind: 0 fp32, 1 bf16.
KSANA_API int ksana_window_attention_any(const void* q, int ldq, const void* cache, const int* block_tables,
                                         int max_blocks, const int* cu_q, const int* kv_lens, const int* seq_of_token,
                                         int h, int hk, int d, int dv, int bs, int window, int keep, int shared,
                                         float scale, const float* bias, int bias_len, float out_scale, void* out,
                                         int ldo, int tok_base, int tokens, int kind, cudaStream_t st) {
  if (tokens <= 0) return 0;
  if (h % hk || keep < 0 || (shared && d != dv)) return -2;
  WindowAttnArgs a{q, ldq, cache, block_tables, max_blocks, cu_q, kv_lens, seq_of_token, h, hk, d, dv, bs, window, keep,
                   shared, scale, bias, bias_len, out_scale, out, ldo};
  return kind ? launch_any<__nv_bfloat16>(a, tok_base, tokens, st) : launch_any<float>(a, tok_base, tokens, st);
}
