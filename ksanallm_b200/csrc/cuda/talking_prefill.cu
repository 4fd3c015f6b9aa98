// Weight-mixing attention (see talking_attention.cu) over prompts on the tensor cores, bf16. A head's output needs all heads'
// normalised weights, so the work goes in three launches per round of 128-row query blocks:
//   statistics   the logarithm of every (query, head)'s softmax denominator, sink included
//   weights      scores again, weights of all heads, their mix -> W[block][hi | lo][head] as two bf16 matrices
//   values       O = (W_hi + W_lo) V per (block, head), times the output gate
// The weights' kernel comes in two forms. For 16, 32 or 64 heads in groups of 2, 4 or 8 both of its products run on tcgen05,
// and a matrix of W is [16][key][8 rows], which is the layout of an MMA operand without swizzle; for other sizes they run on
// mma.sync, and it is [row][key].
// Rounds keep W within a budget; keys beyond a query's position have zero weights in it.
#include "talking.cuh"

namespace ksana {

struct TalkRound {
  int num_seqs;       // of the prompts
  int unit0;          // first 128-row block of the round, counted over the sequences' blocks
  int pitch;          // keys per row of W (a multiple of 128)
  const float* lse;   // [tokens][h], in units where exp2 is the exponential
  __nv_bfloat16* w;
};

// The sequence and the block in it of the round's unit `u`; false: past the last one.
__device__ __forceinline__ bool find_unit(const TalkArgs& a, int num_seqs, int u, int* seq, int* block) {
  for (int b = 0; b < num_seqs; ++b) {
    const int n = (a.cu_q[b + 1] - a.cu_q[b] + 127) / 128;
    if (u < n) {
      *seq = b;
      *block = u;
      return true;
    }
    u -= n;
  }
  return false;
}

// ---- statistics ------------------------------------------------------------------------------------------------------
// One CTA = (block of 128 query rows, head), 160 threads: thread r of warps 0-3 owns row r (TMEM lane r), one lane of warp 4
// issues TMA loads and MMAs. Two score buffers of 128 columns, so Q K^T of the next tile runs under this one's exponentials.
template <int DP>
struct TalkStatsSmem {
  static constexpr int TILE = 128 * DP * 2;
  static constexpr int OFF_BAR = 3 * TILE;
  static constexpr int TOTAL = OFF_BAR + 128 + 1024;
};

template <int DP>
__global__ void __launch_bounds__(160)
talking_stats_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, TalkArgs a, TalkRound rd,
                     float* __restrict__ lse, unsigned int* err) {
  using L_ = TalkStatsSmem<DP>;
  int b, qt;
  // (blocks further along a prompt are longer: they go first)
  if (!find_unit(a, rd.num_seqs, rd.unit0 + gridDim.y - 1 - blockIdx.y, &b, &qt)) return;
  const int head = blockIdx.x, kh = head / (a.h / a.hk);
  const int q0 = a.cu_q[b], q_len = a.cu_q[b + 1] - q0, L = a.kv_lens[b];
  const int row_pos = L - q_len + qt * 128;
  const int tid = threadIdx.x, warp = tid >> 5;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;
  uint8_t* sK = smem + L_::TILE;
  uint64_t* q_bar = reinterpret_cast<uint64_t*>(smem + L_::OFF_BAR);
  uint64_t* k_full = q_bar + 1;   // [2]
  uint64_t* s_done = k_full + 2;  // [2]
  uint64_t* s_free = s_done + 2;  // [2]
  uint32_t* holder = reinterpret_cast<uint32_t*>(s_free + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(holder + 1);
  if (tid == 0) {
    mbar_init(q_bar, 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(&k_full[s], 1);
      mbar_init(&s_done[s], 1);
      mbar_init(&s_free[s], 128);
    }
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 0) {
    tmem_alloc(holder, 256);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *holder;
  const int n = (min(L, row_pos + 128) + 127) / 128;
  const int n_pages = (L + TALK_PAGE - 1) / TALK_PAGE;
  const int* bt = a.block_tables + static_cast<size_t>(b) * a.max_blocks;
  if (warp == 4) {
    if ((tid & 31) == 0) {
      int loads = 0, blk[128 / TALK_PAGE];
      auto pages = [&](int i) {  // of a tile, ahead of its turn
#pragma unroll
        for (int p = 0; p < 128 / TALK_PAGE; ++p) blk[p] = bt[min(i * (128 / TALK_PAGE) + p, n_pages - 1)];  // (past the end: masked)
      };
      auto load_k = [&](int i) {
        uint64_t* bar = &k_full[i & 1];
        mbar_expect_tx(bar, L_::TILE);
#pragma unroll
        for (int p = 0; p < 128 / TALK_PAGE; ++p)
          for (int hf = 0; hf < DP / 64; ++hf)
            tma_load_3d(sK + (i & 1) * L_::TILE + hf * (128 * 128) + p * (TALK_PAGE * 128), &tmK, bar, hf * 64,
                        kh * TALK_PAGE, blk[p]);
        loads = i + 1;
        pages(i + 1);
      };
      pages(0);
      mbar_expect_tx(q_bar, L_::TILE);
      for (int hf = 0; hf < DP / 64; ++hf) tma_load_3d(sQ + hf * (128 * 128), &tmQ, q_bar, hf * 64, head, q0 + qt * 128);
      for (int i = 0; i < 2 && i < n; ++i) load_k(i);
      bool ok = mbar_wait_bounded(q_bar, 0, abort_flag, err);
      for (int i = 0; ok && i < n; ++i) {
        ok = mbar_wait_bounded(&k_full[i & 1], (i >> 1) & 1, abort_flag, err);
        if (ok && i >= 2) ok = mbar_wait_bounded(&s_free[i & 1], ((i >> 1) - 1) & 1, abort_flag, err);
        if (!ok) break;
        tc_fence_after();
        constexpr uint32_t idesc = umma_idesc(128, 128, 1, 1);
        const uint32_t kb = smem_u32(sK + (i & 1) * L_::TILE), qb = smem_u32(sQ);
#pragma unroll
        for (int k = 0; k < DP / 16; ++k) {
          const uint32_t off = (k >> 2) * (128 * 128) + (k & 3) * 32;
          umma_f16(tmem + (i & 1) * 128, umma_desc_k128(qb + off), umma_desc_k128(kb + off), idesc, k > 0 ? 1u : 0u);
        }
        umma_commit(&s_done[i & 1]);
        if (i > 0 && i + 1 < n) {  // the tile before this one has been multiplied: its room takes the next one
          ok = mbar_wait_bounded(&s_done[(i - 1) & 1], ((i - 1) >> 1) & 1, abort_flag, err);
          if (ok) load_k(i + 1);
        }
      }
      if (!ok)  // copies in flight still write to this CTA's memory: give them their (bounded) time before leaving
        for (int i = max(loads - 2, 0); i < loads; ++i)
          for (int it = 0; it < (1 << 20) && !mbar_try_wait(&k_full[i & 1], (i >> 1) & 1); ++it) {}
    }
    __syncwarp();
  } else {
    const uint32_t lane_off = static_cast<uint32_t>(warp * 32) << 16;
    const float scale2 = a.scale * LOG2E;
    float m = a.sink[head] * LOG2E, l = 1.f;
    bool ok = true;
    for (int i = 0; i < n; ++i) {
      ok = mbar_wait_bounded(&s_done[i & 1], (i >> 1) & 1, abort_flag, err);
      if (!__all_sync(0xffffffffu, ok)) {
        ok = false;
        break;
      }
      tc_fence_after();
      float s[128];
#pragma unroll
      for (int c = 0; c < 4; ++c) tmem_ld32(tmem + (i & 1) * 128 + lane_off + c * 32, reinterpret_cast<uint32_t*>(s) + c * 32);
      tmem_wait_ld();
      tc_fence_before();
      mbar_arrive(&s_free[i & 1]);
      const int past = row_pos + tid - i * 128;  // columns beyond this one are later keys
      float top[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
      if (__any_sync(0xffffffffu, past < 127)) {
#pragma unroll
        for (int j = 0; j < 128; ++j)
          if (j > past) s[j] = -INFINITY;
      }
#pragma unroll
      for (int j = 0; j < 128; ++j) top[j & 3] = fmaxf(top[j & 3], s[j]);
      const float m_new = fmaxf(m, fmaxf(fmaxf(top[0], top[1]), fmaxf(top[2], top[3])) * scale2);
      float sum[4] = {l * ex2_ftz(m - m_new), 0.f, 0.f, 0.f};
      m = m_new;
#pragma unroll
      for (int j = 0; j < 128; ++j) sum[j & 3] += ex2_ftz(fmaf(s[j], scale2, -m));
      l = (sum[0] + sum[1]) + (sum[2] + sum[3]);
    }
    if (ok && qt * 128 + tid < q_len) lse[static_cast<size_t>(q0 + qt * 128 + tid) * a.h + head] = m + log2f(l);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(tmem, 256);
  }
}

// ---- weights, tcgen05 ----------------------------------------------------------------------------------------------------
// One CTA = (QN query rows of a block, all HP heads, a range of keys), 128 keys at a time; QN x HP = 256. Keys are the MMA
// rows, so that a thread owns one key, all heads of half of the queries of which are in its registers:
//   S = K_c Q_c^T          per key / value head c: 128 keys x (QN queries x R heads of the group)
//   P = exp(S - lse)       written back to TMEM as two bf16 matrices hi + lo, [query][head]
//   D_i = P_i talk^T       per query i, A = P_i from TMEM
//   W                      D as hi + lo, eight queries of a head side by side
// Two regions of 256 columns change places from tile to tile: S and then D of a tile are in one, its P in the other. Q K^T of
// the next tile runs while this one's D is written out. Warps 0-3 and 4-7 cover the 128 lanes once each; warp 8 loads, warp 9
// issues the MMAs.
template <int DP, int HP>
struct TalkWeightsTcSmem {
  static constexpr int QN = 256 / HP, STAGES = 4;
  static constexpr int TILE = 128 * DP * 2;           // 128 keys of one head
  static constexpr int OFF_Q = STAGES * TILE;
  static constexpr int Q_BYTES = 256 * DP * 2;
  static constexpr int OFF_T = OFF_Q + Q_BYTES;       // the mix, K-major
  static constexpr int OFF_LSE = OFF_T + HP * 128;
  static constexpr int OFF_BAR = OFF_LSE + 256 * 4;
  static constexpr int USED = OFF_BAR + 128 + 1024;
  // at least half of the SM's shared memory: two CTAs would compete for the 512 TMEM columns each of them takes
  static constexpr int TOTAL = USED > 120 * 1024 ? USED : 120 * 1024;
};

template <int DP, int HP, int R>
__global__ void __launch_bounds__(320, 1)
talking_weights_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, TalkArgs a,
                          TalkRound rd, int keys_per, unsigned int* err) {
  using L_ = TalkWeightsTcSmem<DP, HP>;
  constexpr int QN = L_::QN, STAGES = L_::STAGES, G = HP / R, N = QN * R;
  constexpr int QP = 64 / HP;                        // queries whose scores a thread has at a time
  constexpr int WP = QP * R < 8 ? QP * R : 8;        // columns per load of them
  constexpr int DW = QN == 16 ? 4 : 8;               // heads of D at a time
  static_assert(N % 16 == 0 && (WP == 4 || WP == 8), "");
  const int unit = gridDim.x - 1 - blockIdx.x;  // blocks further along a prompt are longer: they go first
  int b, qb;
  if (!find_unit(a, rd.num_seqs, rd.unit0 + unit, &b, &qb)) return;
  const int q_len = a.cu_q[b + 1] - a.cu_q[b], L = a.kv_lens[b];
  const int row0 = qb * 128 + blockIdx.y * QN;  // first query row, within the sequence's new tokens
  if (row0 >= q_len) return;
  const int pos0 = L - q_len + row0, t0 = a.cu_q[b] + row0;
  const int filled = (min(L, L - q_len + qb * 128 + 128) + 127) / 128 * 128;  // what the values' kernel reads
  const int key0 = blockIdx.z * keys_per, key1 = min(key0 + keys_per, filled);
  if (key0 >= key1) return;
  const int tiles = (key1 - key0) / 128;
  const int live = max(0, min(tiles, (min(pos0 + QN, L) - key0 + 127) / 128));  // tiles with a visible key
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t *sQ = smem + L_::OFF_Q, *sT = smem + L_::OFF_T;
  float* sLse = reinterpret_cast<float*>(smem + L_::OFF_LSE);  // [QN][HP]
  uint64_t* q_bar = reinterpret_cast<uint64_t*>(smem + L_::OFF_BAR);
  uint64_t* k_full = q_bar + 1;           // [STAGES]
  uint64_t* k_free = k_full + STAGES;     // [STAGES]
  uint64_t* s_done = k_free + STAGES;
  uint64_t* p_ready = s_done + 1;
  uint64_t* d_done = p_ready + 1;
  uint32_t* holder = reinterpret_cast<uint32_t*>(d_done + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(holder + 1);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (tid == 0) {
    mbar_init(q_bar, 1);
    for (int s = 0; s < STAGES; ++s) {
      mbar_init(&k_full[s], 1);
      mbar_init(&k_free[s], 1);
    }
    mbar_init(s_done, 1);
    mbar_init(p_ready, 256);
    mbar_init(d_done, 1);
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 0) {
    tmem_alloc(holder, 512);
    tmem_relinquish();
  }
  for (int i = tid; i < HP * 8; i += 320) {  // talk[to][from .. from + 7], rows of 128 bytes in the 128-byte swizzle
    const int to = i >> 3, ch = i & 7;
    uint32_t v[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const int from = ch * 8 + u * 2;
      v[u] = from < HP ? pack_bf16(a.talk[to * HP + from], a.talk[to * HP + from + 1]) : 0u;
    }
    *reinterpret_cast<uint4*>(sT + (to >> 3) * 1024 + (to & 7) * 128 + ((ch ^ (to & 7)) << 4)) = make_uint4(v[0], v[1], v[2], v[3]);
  }
  for (int i = tid; i < 256; i += 320)
    sLse[i] = row0 + i / HP < q_len ? rd.lse[static_cast<size_t>(t0 + i / HP) * HP + i % HP] : 0.f;
  fence_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *holder;
  if (warp == 8) {
    if (lane == 0 && live > 0) {
      const int* bt = a.block_tables + static_cast<size_t>(b) * a.max_blocks;
      const int n_pages = (L + TALK_PAGE - 1) / TALK_PAGE;
      mbar_expect_tx(q_bar, L_::Q_BYTES);
      for (int c = 0; c < G; ++c)
        for (int hf = 0; hf < DP / 64; ++hf)
          tma_load_3d(sQ + (c * (DP / 64) + hf) * (N * 128), &tmQ, q_bar, hf * 64, c * R, t0);
      bool ok = true;
      int n = 0, blk[128 / TALK_PAGE];
      for (int t = 0; ok && t < live; ++t) {
#pragma unroll
        for (int p = 0; p < 128 / TALK_PAGE; ++p)
          blk[p] = bt[min((key0 + t * 128) / TALK_PAGE + p, n_pages - 1)];  // (past the end: masked keys)
        for (int c = 0; c < G; ++c, ++n) {
          const int st = n % STAGES;
          if (n >= STAGES) ok = mbar_wait_bounded(&k_free[st], (n / STAGES - 1) & 1, abort_flag, err);
          if (!ok) break;
          mbar_expect_tx(&k_full[st], L_::TILE);
#pragma unroll
          for (int p = 0; p < 128 / TALK_PAGE; ++p)
            for (int hf = 0; hf < DP / 64; ++hf)
              tma_load_3d(smem + st * L_::TILE + hf * (128 * 128) + p * (TALK_PAGE * 128), &tmK, &k_full[st], hf * 64,
                          c * TALK_PAGE, blk[p]);
        }
      }
      if (!ok) {  // copies in flight still write to this CTA's memory: give them their (bounded) time before leaving
        for (int it = 0; it < (1 << 20) && !mbar_try_wait(q_bar, 0); ++it) {}
        for (int i = max(n - STAGES, 0); i < n; ++i)
          for (int it = 0; it < (1 << 20) && !mbar_try_wait(&k_full[i % STAGES], (i / STAGES) & 1); ++it) {}
      }
    }
    __syncwarp();
  } else if (warp == 9) {
    if (lane == 0 && live > 0) {
      bool ok = mbar_wait_bounded(q_bar, 0, abort_flag, err);
      int n = 0;
      for (int t = 0; ok && t < live; ++t) {
        const uint32_t own = tmem + (t & 1) * 256, other = tmem + 256 - (t & 1) * 256;
        for (int c = 0; c < G; ++c, ++n) {
          const int st = n % STAGES;
          ok = mbar_wait_bounded(&k_full[st], (n / STAGES) & 1, abort_flag, err);
          if (!ok) break;
          tc_fence_after();
          constexpr uint32_t idesc = umma_idesc(128, N, 1, 1);
          const uint32_t kb = smem_u32(smem + st * L_::TILE), qa = smem_u32(sQ + c * (DP / 64) * (N * 128));
#pragma unroll
          for (int k = 0; k < DP / 16; ++k)
            umma_f16(own + c * N, umma_desc_k128(kb + (k >> 2) * (128 * 128) + (k & 3) * 32),
                     umma_desc_k128(qa + (k >> 2) * (N * 128) + (k & 3) * 32), idesc, k > 0 ? 1u : 0u);
          umma_commit(&k_free[st]);
        }
        if (!ok) break;
        umma_commit(s_done);
        ok = mbar_wait_bounded(p_ready, t & 1, abort_flag, err);
        if (!ok) break;
        tc_fence_after();
        constexpr uint32_t idesc = umma_idesc(128, HP, 1, 1);
        const uint32_t tb = smem_u32(sT);
#pragma unroll 2
        for (int i = 0; i < QN; ++i)
#pragma unroll
          for (int k = 0; k < HP / 8; ++k)  // hi, then lo
            umma_f16_ts(own + i * HP, other + i * HP + k * 8, umma_desc_k128(tb + (k % (HP / 16)) * 32), idesc, k > 0 ? 1u : 0u);
        umma_commit(d_done);
        ok = mbar_wait_bounded(d_done, t & 1, abort_flag, err);  // (the next scores go over this tile's weights)
      }
    }
    __syncwarp();
  } else {
    const int wg = warp >> 2, j = (warp & 3) * 32 + lane;
    const uint32_t lane_off = static_cast<uint32_t>((warp & 3) * 32) << 16;
    const float scale2 = a.scale * LOG2E;
    const size_t step = static_cast<size_t>(16) * rd.pitch * 8, plane = step * HP;
    __nv_bfloat16* wout = rd.w + unit * 2 * plane + static_cast<size_t>(blockIdx.y * QN / 8) * rd.pitch * 8 + blockIdx.y * QN % 8 +
                          (wg * (HP / 2)) * step + static_cast<size_t>(key0 + j) * 8;
    bool ok = true;
    for (int t = 0; t < live; ++t) {
      const uint32_t own = tmem + (t & 1) * 256 + lane_off, other = tmem + 256 - (t & 1) * 256 + lane_off;
      if (ok) ok = mbar_wait_bounded(s_done, t & 1, abort_flag, err);
      ok = __all_sync(0xffffffffu, ok);
      tc_fence_before();
      asm volatile("bar.sync 1, 256;" ::: "memory");  // everybody has read the last tile's D, which P goes over
      if (ok) {
        tc_fence_after();
        const int past = pos0 + wg * (QN / 2) - (key0 + t * 128 + j);  // queries up to -past - 1 do not see this key
        const bool edge = __any_sync(0xffffffffu, past < 0);
#pragma unroll 1
        for (int i0 = 0; i0 < QN / 2; i0 += QP) {
          float s[64];  // [key / value head][query of this pass][head of the group]
          const uint32_t src = own + (wg * (QN / 2) + i0) * R;
#pragma unroll
          for (int f = 0; f < 64; f += WP) {
            if constexpr (WP == 4)
              tmem_ld4(src + (f / (QP * R)) * N + f % (QP * R), reinterpret_cast<uint32_t*>(s) + f);
            else
              tmem_ld8(src + (f / (QP * R)) * N + f % (QP * R), reinterpret_cast<uint32_t*>(s) + f);
          }
          tmem_wait_ld();
#pragma unroll
          for (int i = 0; i < QP; ++i) {
            const float* lse = sLse + (wg * (QN / 2) + i0 + i) * HP;
            uint32_t p[HP];  // hi, then lo
#pragma unroll
            for (int g = 0; g < HP; g += 2) {
              const int f = (g / R) * (QP * R) + i * R + g % R;
              const float2 l = *reinterpret_cast<const float2*>(lse + g);
              float x = ex2_ftz(fmaf(s[f], scale2, -l.x)), y = ex2_ftz(fmaf(s[f + 1], scale2, -l.y));
              if (edge && i0 + i + past < 0) x = y = 0.f;
              p[g / 2] = split_bf16(x, y, &p[HP / 2 + g / 2]);
            }
            const uint32_t dst = other + (wg * (QN / 2) + i0 + i) * HP;
            if constexpr (HP == 16) {
              tmem_st16(dst, p);
            } else {
#pragma unroll
              for (int c = 0; c < HP; c += 32) tmem_st32(dst + c, p + c);
            }
          }
        }
        tmem_wait_st();
        tc_fence_before();
        mbar_arrive(p_ready);
        ok = mbar_wait_bounded(d_done, t & 1, abort_flag, err);
      }
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) continue;  // keep meeting the other warps at the barrier
      tc_fence_after();
#pragma unroll 1
      for (int g = 0; g < HP / 2; g += DW) {
        float d[QN][DW];
#pragma unroll
        for (int i = 0; i < QN; ++i) {
          if constexpr (DW == 4)
            tmem_ld4(own + i * HP + wg * (HP / 2) + g, reinterpret_cast<uint32_t*>(d[i]));
          else
            tmem_ld8(own + i * HP + wg * (HP / 2) + g, reinterpret_cast<uint32_t*>(d[i]));
        }
        tmem_wait_ld();
        __nv_bfloat16* dst = wout + g * step + static_cast<size_t>(t) * (128 * 8);
#pragma unroll
        for (int x = 0; x < DW; ++x) {
          uint32_t hi[QN / 2], lo[QN / 2];
#pragma unroll
          for (int i = 0; i < QN; i += 2) hi[i / 2] = split_bf16(d[i][x], d[i + 1][x], &lo[i / 2]);
          if constexpr (QN == 4) {
            *reinterpret_cast<uint2*>(dst + x * step) = make_uint2(hi[0], hi[1]);
            *reinterpret_cast<uint2*>(dst + x * step + plane) = make_uint2(lo[0], lo[1]);
          } else {
#pragma unroll
            for (int q = 0; q < QN / 8; ++q) {
              const size_t at = x * step + static_cast<size_t>(q) * rd.pitch * 8;
              *reinterpret_cast<uint4*>(dst + at) = make_uint4(hi[q * 4], hi[q * 4 + 1], hi[q * 4 + 2], hi[q * 4 + 3]);
              *reinterpret_cast<uint4*>(dst + at + plane) = make_uint4(lo[q * 4], lo[q * 4 + 1], lo[q * 4 + 2], lo[q * 4 + 3]);
            }
          }
        }
      }
    }
    for (int t = live; t < tiles; ++t)
      for (int g = 0; g < HP / 2; ++g)
        for (int part = 0; part < 2; ++part) {
          __nv_bfloat16* dst = wout + g * step + part * plane + static_cast<size_t>(t) * (128 * 8);
          if constexpr (QN == 4) {
            *reinterpret_cast<uint2*>(dst) = make_uint2(0, 0);
          } else {
#pragma unroll
            for (int q = 0; q < QN / 8; ++q)
              *reinterpret_cast<uint4*>(dst + static_cast<size_t>(q) * rd.pitch * 8) = make_uint4(0, 0, 0, 0);
          }
        }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

// ---- weights, other sizes --------------------------------------------------------------------------------------------------
// One CTA of 8 warps = (QN query rows of a block, all heads, a range of keys), 32 keys at a time, QN x (heads filled up to
// HP = 16 HK) = 512 rows. Scores: the rows of one key / value head are cut into units of 16 (queries x heads of the group);
// a warp keeps the queries of up to four units in registers and streams those heads' keys through a ring of its own with
// TMA. The normalised weights go to shared memory [query][hi | lo][head][key]; then a warp takes a query and multiplies by
// the mix, W = talk P (talk is bf16 by storage; P as hi + lo), in place, and copies the result out.
template <int DP, int HK>
struct TalkWeightsSmem {
  static constexpr int HP = 16 * HK, QN = 512 / HP;
  static constexpr int SLOT = 32 * DP * 2;           // 32 keys of one head
  static constexpr int RING = 8 * 2 * SLOT;
  static constexpr int ROW = 80;                     // 32 weights, rows four banks apart from one another
  static constexpr int QUERY = 2 * HP * ROW + 64;    // both parts of a query's weights
  static constexpr int OFF_P = RING;
  static constexpr int TROW = HP * 2 + 16;
  static constexpr int OFF_T = OFF_P + QN * QUERY;
  static constexpr int OFF_BAR = OFF_T + HP * TROW;
  static constexpr int TOTAL = OFF_BAR + 8 * 2 * 8 + 16 + 1024;
};

template <int DP, int HK>
__global__ void __launch_bounds__(256, 1)
talking_weights_kernel(const __grid_constant__ CUtensorMap tmK, TalkArgs a, TalkRound rd, int keys_per, unsigned int* err) {
  using L_ = TalkWeightsSmem<DP, HK>;
  constexpr int HP = L_::HP, QN = L_::QN, ROW = L_::ROW, UW = 4;
  int b, qb;
  if (!find_unit(a, rd.num_seqs, rd.unit0 + blockIdx.x, &b, &qb)) return;
  const int q_len = a.cu_q[b + 1] - a.cu_q[b], L = a.kv_lens[b];
  const int row0 = qb * 128 + blockIdx.y * QN;  // first query row, within the sequence's new tokens
  if (row0 >= q_len) return;
  const int pos0 = L - q_len + row0;
  const int t0 = a.cu_q[b] + row0, rows = min(QN, q_len - row0);
  const int filled = (min(L, L - q_len + qb * 128 + 128) + 127) / 128 * 128;  // what the values' kernel reads
  const int key0 = blockIdx.z * keys_per, key1 = min(key0 + keys_per, filled);
  if (key0 >= key1) return;
  const int tiles = (key1 - key0) / 32;
  const int live = max(0, min(tiles, (min(pos0 + QN, L) - key0 + 31) / 32));  // tiles with a visible key
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sP = smem + L_::OFF_P;
  __nv_bfloat16* sT = reinterpret_cast<__nv_bfloat16*>(smem + L_::OFF_T);
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + L_::OFF_BAR);  // [8][2]
  volatile int* abort_flag = reinterpret_cast<volatile int*>(full + 16);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int r = lane >> 2, j2 = (lane & 3) * 2;
  if (tid == 0) {
    for (int i = 0; i < 16; ++i) mbar_init(&full[i], 1);
    *abort_flag = 0;
    fence_mbar_init();
  }
  for (int i = tid; i < QN * L_::QUERY / 16; i += 256) reinterpret_cast<uint4*>(sP)[i] = make_uint4(0, 0, 0, 0);
  for (int i = tid; i < HP * HP; i += 256) {
    const int to = i / HP, from = i % HP;
    sT[to * (L_::TROW / 2) + from] = __float2bfloat16_rn(to < a.h && from < a.h ? a.talk[to * a.h + from] : 0.f);
  }
  __syncthreads();

  // this warp's units
  const int R = a.h / a.hk, upc = (QN * R + 15) / 16, total = a.hk * upc;
  const int per = (total + 7) / 8, u0 = min(warp * per, total), u1 = min(u0 + per, total);  // per <= UW
  const int c_first = u0 / upc, nc = u1 > u0 ? (u1 - 1) / upc - c_first + 1 : 0;
  uint32_t qf[UW][DP / 16][4];
  float ls[UW][2];
  int at[UW][2], pos[UW][2];  // of this thread's two rows: offset of the weights' row (-1: none), position of the query
#pragma unroll
  for (int k = 0; k < UW; ++k)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int u = u0 + k, c = u / upc, row = (u % upc) * 16 + r + e * 8, i = row / R, g = c * R + row % R;
      const bool is = u < u1 && row < QN * R && i < rows;
      at[k][e] = is ? i * L_::QUERY + g * ROW : -1;
      pos[k][e] = pos0 + i;
      ls[k][e] = is ? rd.lse[static_cast<size_t>(t0 + i) * a.h + g] : 0.f;
      const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q) + static_cast<size_t>(t0 + i) * a.ldq + g * a.d;
#pragma unroll
      for (int kb = 0; kb < DP / 16; ++kb)
#pragma unroll
        for (int w = 0; w < 2; ++w) {
          const int col = kb * 16 + w * 8 + j2;
          qf[k][kb][w * 2 + e] = is && col < a.d ? *reinterpret_cast<const uint32_t*>(q + col) : 0u;
        }
    }
  const int* bt = a.block_tables + static_cast<size_t>(b) * a.max_blocks;
  const int n_pages = (L + TALK_PAGE - 1) / TALK_PAGE;
  uint8_t* ring = smem + warp * 2 * L_::SLOT;
  const int loads = live * nc;
  int issued = 0;
  auto issue = [&](int n) {
    if (lane == 0) {
      uint8_t* dst = ring + (n & 1) * L_::SLOT;
      uint64_t* bar = &full[warp * 2 + (n & 1)];
      mbar_expect_tx(bar, L_::SLOT);
      const int page0 = (key0 + n / nc * 32) / TALK_PAGE, kh = c_first + n % nc;
#pragma unroll
      for (int p = 0; p < 2; ++p) {
        const int blk = bt[min(page0 + p, n_pages - 1)];
#pragma unroll
        for (int hf = 0; hf < DP / 64; ++hf)
          tma_load_3d(dst + p * (16 * DP * 2) + hf * 2048, &tmK, bar, hf * 64, kh * TALK_PAGE, blk);
      }
    }
    issued = n + 1;
  };
  for (int n = 0; n < 2 && n < loads; ++n) issue(n);
  const float scale2 = a.scale * LOG2E;
  const int k_row = (lane & 7) + ((lane >> 4) << 3), k_col = (lane >> 3) & 1;
  const size_t plane = static_cast<size_t>(a.h) * 128 * rd.pitch;
  __nv_bfloat16* wout = rd.w + blockIdx.x * 2 * plane + static_cast<size_t>(blockIdx.y * QN) * rd.pitch;
  bool ok = true;
  for (int t = 0; t < live; ++t) {
    const int key = key0 + t * 32;
    const bool edge = key + 31 > pos0;  // some of these keys are later than some query
    for (int ci = 0; ci < nc; ++ci) {
      const int n = t * nc + ci;
      if (ok) ok = mbar_wait_bounded(&full[warp * 2 + (n & 1)], (n >> 1) & 1, abort_flag, err);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      const uint32_t kb0 = smem_u32(ring + (n & 1) * L_::SLOT);
      float acc[UW][4][4];
#pragma unroll
      for (int k = 0; k < UW; ++k)
#pragma unroll
        for (int nt = 0; nt < 4; ++nt)
#pragma unroll
          for (int e = 0; e < 4; ++e) acc[k][nt][e] = 0.f;
      const int ua = max(u0, (c_first + ci) * upc) - u0, ub = min(u1, (c_first + ci + 1) * upc) - u0;  // the head's units
#pragma unroll
      for (int kb = 0; kb < DP / 16; ++kb) {
        const int ch = kb * 2 + k_col;
        const uint32_t off = (ch >> 3) * 2048 + k_row * 128 + (((ch & 7) ^ (k_row & 7)) << 4);
        uint32_t f[2][4];
        ldmatrix_x4<false>(f[0], kb0 + off);
        ldmatrix_x4<false>(f[1], kb0 + 16 * DP * 2 + off);
#pragma unroll
        for (int k = 0; k < UW; ++k)
          if (k >= ua && k < ub) {
#pragma unroll
            for (int nt = 0; nt < 4; ++nt)
              mma_16816(acc[k][nt], qf[k][kb], f[nt >> 1][(nt & 1) * 2], f[nt >> 1][(nt & 1) * 2 + 1]);
          }
      }
      __syncwarp();  // every lane has read these keys
      if (n + 2 < loads) issue(n + 2);
#pragma unroll
      for (int k = 0; k < UW; ++k)
        if (k >= ua && k < ub) {
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            if (at[k][e] < 0) continue;
            uint8_t* dst = sP + at[k][e] + j2 * 2;
            if (edge) {
#pragma unroll
              for (int nt = 0; nt < 4; ++nt) {
                const int j = key + nt * 8 + j2;
                if (j > pos[k][e]) acc[k][nt][e * 2] = -INFINITY;
                if (j + 1 > pos[k][e]) acc[k][nt][e * 2 + 1] = -INFINITY;
              }
            }
#pragma unroll
            for (int nt = 0; nt < 4; ++nt) {
              const float x = ex2_ftz(fmaf(acc[k][nt][e * 2], scale2, -ls[k][e]));
              const float y = ex2_ftz(fmaf(acc[k][nt][e * 2 + 1], scale2, -ls[k][e]));
              uint32_t low;
              *reinterpret_cast<uint32_t*>(dst + nt * 16) = split_bf16(x, y, &low);
              *reinterpret_cast<uint32_t*>(dst + HP * ROW + nt * 16) = low;
            }
          }
        }
    }
    __syncthreads();
    for (int i = warp; i < rows; i += 8) {
      uint8_t* P = sP + i * L_::QUERY;
      const uint32_t pa = smem_u32(P) + ((lane & 7) + (lane & 8)) * ROW + (lane >> 4) * 16;
#pragma unroll
      for (int jb = 0; jb < 2; ++jb) {
        uint32_t fh[HK][4], fl[HK][4];
#pragma unroll
        for (int kt = 0; kt < HK; ++kt) {
          ldmatrix_x4<true>(fh[kt], pa + kt * 16 * ROW + jb * 32);
          ldmatrix_x4<true>(fl[kt], pa + (HP + kt * 16) * ROW + jb * 32);
        }
        __syncwarp();  // (written over below)
#pragma unroll
        for (int mt = 0; mt < HK; ++mt) {
          float c[2][4];
#pragma unroll
          for (int e = 0; e < 4; ++e) c[0][e] = c[1][e] = 0.f;
#pragma unroll
          for (int kt = 0; kt < HK; ++kt) {
            uint32_t ta[4];
            ldmatrix_x4<false>(ta, smem_u32(sT) + (mt * 16 + (lane & 7) + (lane & 8)) * L_::TROW + kt * 32 + (lane >> 4) * 16);
#pragma unroll
            for (int x = 0; x < 2; ++x) {
              mma_16816(c[x], ta, fh[kt][x * 2], fh[kt][x * 2 + 1]);
              mma_16816(c[x], ta, fl[kt][x * 2], fl[kt][x * 2 + 1]);
            }
          }
#pragma unroll
          for (int x = 0; x < 2; ++x)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              uint8_t* dst = P + (mt * 16 + r + e * 8) * ROW + jb * 32 + x * 16 + j2 * 2;
              uint32_t low;
              *reinterpret_cast<uint32_t*>(dst) = split_bf16(c[x][e * 2], c[x][e * 2 + 1], &low);
              *reinterpret_cast<uint32_t*>(dst + HP * ROW) = low;
            }
        }
      }
      __syncwarp();
      {
        const int ch = lane & 3;
        const uint8_t* src = P + (lane >> 2) * ROW + ch * 16;
        __nv_bfloat16* dst = wout + (static_cast<size_t>(lane >> 2) * 128 + i) * rd.pitch + key + ch * 8;
        const size_t step = static_cast<size_t>(8 * 128) * rd.pitch;
#pragma unroll
        for (int g0 = 0; g0 < HP; g0 += 8, src += 8 * ROW, dst += step)
          if (g0 + (lane >> 2) < a.h) {
            *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(src);
            *reinterpret_cast<uint4*>(dst + plane) = *reinterpret_cast<const uint4*>(src + HP * ROW);
          }
      }
    }
    __syncthreads();
  }
  // copies in flight still write to this CTA's memory: give them their (bounded) time before leaving
  if (!ok && lane == 0)
    for (int n = max(issued - 2, 0); n < issued; ++n)
      for (int it = 0; it < (1 << 20) && !mbar_try_wait(&full[warp * 2 + (n & 1)], (n >> 1) & 1); ++it) {}
  const int dead = (tiles - live) * 4;  // words of 8 zeros per row
  for (int x = tid; x < 2 * a.h * rows * dead; x += 256) {
    const int ch = x % dead, row = x / dead, i = row % rows, g = row / rows % a.h, part = row / (rows * a.h);
    *reinterpret_cast<uint4*>(wout + part * plane + (static_cast<size_t>(g) * 128 + i) * rd.pitch + key0 + live * 32 + ch * 8) =
        make_uint4(0, 0, 0, 0);
  }
}

// ---- values ------------------------------------------------------------------------------------------------------------
// One CTA = (block of 128 query rows, head): warp 4 loads tiles of 128 keys (both parts of W, the values' pages), warp 5
// issues the MMAs, warps 0-3 write the result out. BLOCKED: the layout of W that the tcgen05 form of the weights' kernel
// leaves.
template <int DVP>
struct TalkValuesSmem {
  static constexpr int W_BYTES = 128 * 128 * 2;  // one part
  static constexpr int STAGE = 2 * W_BYTES + 128 * DVP * 2;
  static constexpr int OFF_BAR = 2 * STAGE;
  static constexpr int TOTAL = OFF_BAR + 128 + 1024;
};

// MN-major operand without swizzle: 8 elements along MN are 16 bytes, 8 K-rows of them 128 bytes; the next 8 K-rows lie lbo
// bytes on, the next 8 elements along MN sbo bytes.
__device__ __forceinline__ uint64_t umma_desc_mn_plain(uint32_t smem_addr, uint32_t lbo_bytes, uint32_t sbo_bytes) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((smem_addr >> 4) & 0x3FFF);
  d |= static_cast<uint64_t>((lbo_bytes >> 4) & 0x3FFF) << 16;
  d |= static_cast<uint64_t>((sbo_bytes >> 4) & 0x3FFF) << 32;
  d |= static_cast<uint64_t>(1) << 46;
  return d;
}

template <int DVP, bool BLOCKED>
__global__ void __launch_bounds__(192)
talking_values_kernel(const __grid_constant__ CUtensorMap tmW, const __grid_constant__ CUtensorMap tmV, TalkArgs a,
                      TalkRound rd, unsigned int* err) {
  using L_ = TalkValuesSmem<DVP>;
  const int unit = gridDim.y - 1 - blockIdx.y;  // longest first
  int b, qt;
  if (!find_unit(a, rd.num_seqs, rd.unit0 + unit, &b, &qt)) return;
  const int head = blockIdx.x, kh = head / (a.h / a.hk);
  const int q_len = a.cu_q[b + 1] - a.cu_q[b], L = a.kv_lens[b];
  const int n = (min(L, L - q_len + qt * 128 + 128) + 127) / 128;
  const int tid = threadIdx.x, warp = tid >> 5;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + L_::OFF_BAR);  // [2]
  uint64_t* freed = full + 2;                                        // [2]
  uint64_t* done = freed + 2;
  uint32_t* holder = reinterpret_cast<uint32_t*>(done + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(holder + 1);
  if (tid == 0) {
    for (int s = 0; s < 2; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&freed[s], 1);
    }
    mbar_init(done, 1);
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 0) {
    tmem_alloc(holder, DVP);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *holder;
  if (warp == 4) {
    if ((tid & 31) == 0) {
      const int* bt = a.block_tables + static_cast<size_t>(b) * a.max_blocks;
      const int n_pages = (L + TALK_PAGE - 1) / TALK_PAGE;
      const int row_hi = (unit * 2 * a.h + head) * 128, row_lo = row_hi + a.h * 128;
      bool ok = true;
      int loads = 0;
      for (int i = 0; i < n; ++i) {
        int blk[128 / TALK_PAGE];
#pragma unroll
        for (int p = 0; p < 128 / TALK_PAGE; ++p) blk[p] = bt[min(i * (128 / TALK_PAGE) + p, n_pages - 1)];  // (past the end: zero weights)
        if (i >= 2) ok = mbar_wait_bounded(&freed[i & 1], ((i >> 1) - 1) & 1, abort_flag, err);
        if (!ok) break;
        uint8_t* dst = smem + (i & 1) * L_::STAGE;
        uint64_t* bar = &full[i & 1];
        mbar_expect_tx(bar, L_::STAGE);
        if constexpr (BLOCKED) {
          tma_load_2d(dst, &tmW, bar, i * 256, row_hi / 8);  // (128 keys x 8 rows as 256 words of 8 bytes, 16 times)
          tma_load_2d(dst + L_::W_BYTES, &tmW, bar, i * 256, row_lo / 8);
        }
        for (int hf = 0; hf < (BLOCKED ? 0 : 2); ++hf) {
          tma_load_2d(dst + hf * (128 * 128), &tmW, bar, i * 128 + hf * 64, row_hi);
          tma_load_2d(dst + L_::W_BYTES + hf * (128 * 128), &tmW, bar, i * 128 + hf * 64, row_lo);
        }
#pragma unroll
        for (int p = 0; p < 128 / TALK_PAGE; ++p)
          for (int hf = 0; hf < DVP / 64; ++hf)
            tma_load_3d(dst + 2 * L_::W_BYTES + hf * (128 * 128) + p * (TALK_PAGE * 128), &tmV, bar, hf * 64,
                        kh * TALK_PAGE, blk[p]);
        loads = i + 1;
      }
      if (!ok)  // copies in flight still write to this CTA's memory: give them their (bounded) time before leaving
        for (int i = max(loads - 2, 0); i < loads; ++i)
          for (int it = 0; it < (1 << 20) && !mbar_try_wait(&full[i & 1], (i >> 1) & 1); ++it) {}
    }
    __syncwarp();
  } else if (warp == 5) {
    if ((tid & 31) == 0) {
      bool ok = true;
      for (int i = 0; ok && i < n; ++i) {
        ok = mbar_wait_bounded(&full[i & 1], (i >> 1) & 1, abort_flag, err);
        if (!ok) break;
        tc_fence_after();
        constexpr uint32_t idesc = umma_idesc_major(128, DVP, BLOCKED, true);
        const uint32_t wb = smem_u32(smem + (i & 1) * L_::STAGE), vb = wb + 2 * L_::W_BYTES;
#pragma unroll
        for (int k = 0; k < 16; ++k) {  // hi, then lo
          const uint32_t part = wb + (k >> 3) * L_::W_BYTES;
          const uint64_t aw = BLOCKED ? umma_desc_mn_plain(part + (k & 7) * 256, 128, 2048)
                                      : umma_desc_k128(part + ((k >> 2) & 1) * (128 * 128) + (k & 3) * 32);
          umma_f16(tmem, aw, umma_desc_mn128(vb + (k & 7) * (16 * 128), 128 * 128), idesc,
                   i > 0 || k > 0 ? 1u : 0u);
        }
        umma_commit(&freed[i & 1]);
      }
      if (ok) umma_commit(done);
    }
    __syncwarp();
  } else {
    const bool ok = mbar_wait_bounded(done, 0, abort_flag, err);
    if (__all_sync(0xffffffffu, ok)) {
      tc_fence_after();
      const bool valid = qt * 128 + tid < q_len;
      const size_t tok = a.cu_q[b] + qt * 128 + tid;
#pragma unroll 1
      for (int c = 0; c < DVP / 32; ++c) {
        uint32_t v[32];
        tmem_ld32(tmem + (static_cast<uint32_t>(warp * 32) << 16) + c * 32, v);
        tmem_wait_ld();
#pragma unroll
        for (int j = 0; j < 32; j += 8)
          if (valid && c * 32 + j < a.dv) talk_store8(a, tok, head * a.dv + c * 32 + j, reinterpret_cast<float*>(v) + j);
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(tmem, DVP);
  }
}

// ---- launches ----------------------------------------------------------------------------------------------------------
constexpr long long TALK_W_BYTES = 1ll << 30;  // weights written out at a time, unless one block of rows needs more

static int talk_units(const int* cu, int b) { return (cu[b + 1] - cu[b] + 127) / 128; }
// keys of a block's rows, up to the multiple of 128 that its tiles cover
static int talk_keys(const int* cu, const int* kv, int b, int block) {
  const int pos = kv[b] - (cu[b + 1] - cu[b]) + block * 128 + 128;
  return ((pos < kv[b] ? pos : kv[b]) + 127) / 128 * 128;
}

struct TalkPlan {
  int units = 0, pitch = 0;  // of one round
};
// The round that starts with block `block` of sequence `b`; both move on to the next round's.
static TalkPlan talk_plan(int h, int num_seqs, const int* cu, const int* kv, int* b, int* block) {
  TalkPlan p;
  while (*b < num_seqs) {
    if (*block >= talk_units(cu, *b)) {
      ++*b;
      *block = 0;
      continue;
    }
    const int keys = talk_keys(cu, kv, *b, *block), pitch = keys > p.pitch ? keys : p.pitch;
    if (p.units > 0 && (p.units + 1ll) * 128 * pitch * h * 4 > TALK_W_BYTES) break;
    if (p.units >= 2048) break;
    ++p.units;
    p.pitch = pitch;
    ++*block;
  }
  return p;
}

template <int DP>
static int launch_stats(const TalkArgs& a, const CUtensorMap& tq, const CUtensorMap& tk, const TalkRound& rd, int units,
                        float* lse, cudaStream_t st) {
  auto kern = talking_stats_kernel<DP>;
  if (KSANA_SMEM_ONCE(kern, TalkStatsSmem<DP>::TOTAL) != 0) return -4;
  kern<<<dim3(a.h, units), 160, TalkStatsSmem<DP>::TOTAL, st>>>(tq, tk, a, rd, lse, error_word());
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}
template <int DP, int HK>
static int launch_weights(const TalkArgs& a, const CUtensorMap& tk, const TalkRound& rd, int units, cudaStream_t st) {
  using L_ = TalkWeightsSmem<DP, HK>;
  static_assert(L_::TOTAL <= 232448, "does not fit");
  auto kern = talking_weights_kernel<DP, HK>;
  if (KSANA_SMEM_ONCE(kern, L_::TOTAL) != 0) return -4;
  const int subs = 128 / L_::QN;
  // key ranges: several waves of CTAs, none of them shorter than 256 keys
  int parts = 1;
  while (static_cast<long long>(units) * subs * parts < 4ll * sm_count() && rd.pitch / (parts + 1) >= 256) ++parts;
  const int keys_per = ((rd.pitch + parts - 1) / parts + 31) / 32 * 32;
  kern<<<dim3(units, subs, (rd.pitch + keys_per - 1) / keys_per), 256, L_::TOTAL, st>>>(tk, a, rd, keys_per, error_word());
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}
template <int DP, int HP, int R>
static int launch_weights_tc(const TalkArgs& a, int total_tokens, const CUtensorMap& tk, const TalkRound& rd, int units,
                             cudaStream_t st) {
  using L_ = TalkWeightsTcSmem<DP, HP>;
  static_assert(L_::TOTAL <= 232448, "does not fit");
  CUtensorMap tq;
  const uint64_t dims[3] = {static_cast<uint64_t>(a.d), static_cast<uint64_t>(a.h), static_cast<uint64_t>(total_tokens)};
  const uint64_t str[2] = {static_cast<uint64_t>(a.d) * 2, static_cast<uint64_t>(a.ldq) * 2};
  const uint32_t box[3] = {64, R, L_::QN};
  if (make_tmap_nd(&tq, a.q, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, dims, str, box, CU_TENSOR_MAP_SWIZZLE_128B)) return -2;
  auto kern = talking_weights_tc_kernel<DP, HP, R>;
  if (KSANA_SMEM_ONCE(kern, L_::TOTAL) != 0) return -4;
  const int subs = 128 / L_::QN;
  // key ranges: several waves of CTAs, none of them shorter than 512 keys
  int parts = 1;
  while (static_cast<long long>(units) * subs * parts < 6ll * sm_count() && rd.pitch / (parts + 1) >= 512) ++parts;
  const int keys_per = ((rd.pitch + parts - 1) / parts + 127) / 128 * 128;
  kern<<<dim3(units, subs, (rd.pitch + keys_per - 1) / keys_per), 320, L_::TOTAL, st>>>(tq, tk, a, rd, keys_per, error_word());
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}
// -1: not a size of the tcgen05 form
static int weights_tc(const TalkArgs& a, int total_tokens, const CUtensorMap& tk, const TalkRound& rd, int units,
                      cudaStream_t st) {
  const int r = a.h / a.hk;
#define KSANA_TWT(HP, R)                                                                                 \
  if (a.h == HP && r == R)                                                                               \
    return a.d <= 64 ? launch_weights_tc<64, HP, R>(a, total_tokens, tk, rd, units, st)                  \
                     : launch_weights_tc<128, HP, R>(a, total_tokens, tk, rd, units, st)
  KSANA_TWT(16, 2);
  KSANA_TWT(16, 4);
  KSANA_TWT(16, 8);
  KSANA_TWT(32, 2);
  KSANA_TWT(32, 4);
  KSANA_TWT(32, 8);
  KSANA_TWT(64, 4);
  KSANA_TWT(64, 8);
#undef KSANA_TWT
  return -1;
}
template <int DVP, bool BLOCKED>
static int launch_values(const TalkArgs& a, const CUtensorMap& tv, const TalkRound& rd, int units, cudaStream_t st) {
  CUtensorMap tw;
  const uint64_t rows = static_cast<uint64_t>(units) * 2 * a.h * 128;
  if (BLOCKED) {
    const uint64_t dims[2] = {static_cast<uint64_t>(rd.pitch) * 2, rows / 8}, str[1] = {static_cast<uint64_t>(rd.pitch) * 16};
    const uint32_t box[2] = {256, 16};
    if (make_tmap_nd(&tw, rd.w, CU_TENSOR_MAP_DATA_TYPE_FLOAT64, 2, dims, str, box, CU_TENSOR_MAP_SWIZZLE_NONE)) return -2;
  } else if (make_tmap_2d(&tw, rd.w, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, rows, rd.pitch, rd.pitch, 128, 64, CU_TENSOR_MAP_SWIZZLE_128B))
    return -2;
  auto kern = talking_values_kernel<DVP, BLOCKED>;
  if (KSANA_SMEM_ONCE(kern, TalkValuesSmem<DVP>::TOTAL) != 0) return -4;
  kern<<<dim3(a.h, units), 192, TalkValuesSmem<DVP>::TOTAL, st>>>(tw, tv, a, rd, error_word());
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

// units of 16 rows that one CTA of the weights' kernel has
static bool weights_fit(const TalkArgs& a) {
  const int hp = a.h <= 16 ? 16 : a.h <= 32 ? 32 : 64, qn = 512 / hp;
  return a.hk * ((qn * (a.h / a.hk) + 15) / 16) <= 32;
}

}  // namespace ksana

using namespace ksana;

// Scratch bytes of ksana_talking_prefill for sequences [0, num_seqs), whose tokens are the step's first ones.
KSANA_API long long ksana_talking_prefill_bytes(int h, int num_seqs, const int* cu_q_host, const int* kv_lens_host) {
  long long most = 0;
  for (int b = 0, block = 0; b < num_seqs;) {
    const TalkPlan p = talk_plan(h, num_seqs, cu_q_host, kv_lens_host, &b, &block);
    const long long n = static_cast<long long>(p.units) * 128 * p.pitch * h * 4;
    if (n > most) most = n;
  }
  return (static_cast<long long>(num_seqs > 0 ? cu_q_host[num_seqs] : 0) * h * 4 + 255) / 256 * 256 + most + 256;
}

// bf16. Sequences [0, num_seqs). Returns -1 for sizes it does not take (pages of 16 tokens, at most 64 heads, heads of at
// most 128 dimensions in multiples of 8, 16-byte aligned rows).
KSANA_API int ksana_talking_prefill(const void* q, int ldq, int total_tokens, const void* cache, int num_blocks,
                                    const int* block_tables, int max_blocks, const int* cu_q, const int* kv_lens, int h,
                                    int hk, int d, int dv, int bs, float scale, const float* sink, const float* talk,
                                    float out_scale, const void* gate, int ldg, void* out, int ldo, int num_seqs,
                                    const int* cu_q_host, const int* kv_lens_host, void* scratch, long long scratch_bytes,
                                    int* launches, cudaStream_t st) {
  if (num_seqs <= 0) return 0;
  TalkArgs a{q, ldq, cache, block_tables, max_blocks, cu_q, kv_lens, nullptr, h, hk, d, dv, bs, scale, sink, talk,
             out_scale, gate, ldg, out, ldo};
  if (!talk_tc_sizes(a) || !weights_fit(a)) return -1;
  if (scratch_bytes < ksana_talking_prefill_bytes(h, num_seqs, cu_q_host, kv_lens_host)) return -6;
  char* base = reinterpret_cast<char*>((reinterpret_cast<uintptr_t>(scratch) + 255) & ~uintptr_t(255));
  float* lse = reinterpret_cast<float*>(base);
  CUtensorMap tq, tk, tv;
  {
    const uint64_t dims[3] = {static_cast<uint64_t>(d), static_cast<uint64_t>(h), static_cast<uint64_t>(total_tokens)};
    const uint64_t str[2] = {static_cast<uint64_t>(d) * 2, static_cast<uint64_t>(ldq) * 2};
    const uint32_t box[3] = {64, 1, 128};
    if (make_tmap_nd(&tq, q, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, dims, str, box, CU_TENSOR_MAP_SWIZZLE_128B)) return -2;
  }
  if (int rc = talk_cache_map(a, num_blocks, 0, &tk)) return rc;
  if (int rc = talk_cache_map(a, num_blocks, 1, &tv)) return rc;
  TalkRound rd{num_seqs, 0, 0, lse, reinterpret_cast<__nv_bfloat16*>(
                                        base + (static_cast<long long>(cu_q_host[num_seqs]) * h * 4 + 255) / 256 * 256)};
  int all = 0;
  for (int b = 0; b < num_seqs; ++b) all += talk_units(cu_q_host, b);
  if (all == 0) return 0;
  if (int rc = d <= 64 ? launch_stats<64>(a, tq, tk, rd, all, lse, st) : launch_stats<128>(a, tq, tk, rd, all, lse, st)) return rc;
  *launches = 1;
  for (int b = 0, block = 0; rd.unit0 < all;) {
    const TalkPlan p = talk_plan(h, num_seqs, cu_q_host, kv_lens_host, &b, &block);
    rd.pitch = p.pitch;
    int rc = weights_tc(a, total_tokens, tk, rd, p.units, st);
    const bool blocked = rc != -1;
#define KSANA_TW(DP) \
  rc = h <= 16 ? launch_weights<DP, 1>(a, tk, rd, p.units, st) \
       : h <= 32 ? launch_weights<DP, 2>(a, tk, rd, p.units, st) : launch_weights<DP, 4>(a, tk, rd, p.units, st)
    if (!blocked) {
      if (d <= 64) KSANA_TW(64); else KSANA_TW(128);
    }
#undef KSANA_TW
    if (rc) return rc;
    if (blocked)
      rc = dv <= 64 ? launch_values<64, true>(a, tv, rd, p.units, st) : launch_values<128, true>(a, tv, rd, p.units, st);
    else
      rc = dv <= 64 ? launch_values<64, false>(a, tv, rd, p.units, st) : launch_values<128, false>(a, tv, rd, p.units, st);
    if (rc) return rc;
    *launches += 2;
    rd.unit0 += p.units;
  }
  return 0;
}
