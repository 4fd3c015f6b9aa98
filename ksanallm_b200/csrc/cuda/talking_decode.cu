// Weight-mixing attention (see talking_attention.cu) of sequences with one new token, bf16: two streams over the cache.
//   scores   over the keys: every score to a small fp32 buffer [sequence][key][heads], and each range's maximum and sum
//   values   over the values: the softmax's denominators, then per page the normalised weights of all heads, their mix for
//            the heads of this key / value head, and the weighted sum
// Both multiply with mma.sync over 16-key pages that every warp brings in through a TMA ring of its own; keys are the rows
// of the products and heads their columns, so few heads cost no padding rows.
#include "talking.cuh"

namespace ksana {

struct TalkDecode {
  float* s;        // [num_seqs][pitch][hp], in units where exp2 is the exponential
  float2* stats;   // [num_seqs][score_splits][h]: maximum, sum
  int pitch;       // keys per sequence
  int hp;          // heads filled up to a multiple of 16
  int score_splits;
};

// a warp's share of a CTA's range of pages and its ring of them in flight
template <int BYTES>
struct PageRing {
  static constexpr int STAGES = BYTES <= 2048 ? 4 : 3;
  static constexpr int RING = 4 * STAGES * BYTES;
};

// ---- scores --------------------------------------------------------------------------------------------------------------
template <int DP, int NT>
__global__ void __launch_bounds__(128)
talking_scores_kernel(const __grid_constant__ CUtensorMap tmK, TalkArgs a, TalkDecode td, int seq_base, int groups,
                      unsigned int* err) {
  constexpr int PAGE = 16 * DP * 2, STAGES = PageRing<PAGE>::STAGES;
  extern __shared__ uint8_t smem_raw[];
  __shared__ uint64_t full[4][STAGES];
  __shared__ float sM[4][16], sL[4][16];
  __shared__ int abort_word;
  volatile int* abort_flag = &abort_word;
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int splits = gridDim.x, split = blockIdx.x, kh = blockIdx.y / groups, hpart = blockIdx.y % groups;
  const int b = blockIdx.z + seq_base, gq = a.h / a.hk;
  const int head0 = kh * gq + hpart * 8 * NT, g = min(8 * NT, gq - hpart * 8 * NT);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r = lane >> 2, j2 = (lane & 3) * 2;
  const int t = a.cu_q[b], pos = a.kv_lens[b] - 1, pages = (pos >> 4) + 1;
  const int per = (pages + splits - 1) / splits;
  const int first = split * per + warp, last = min(split * per + per, pages);
  const int count = first < last ? (last - first + 3) / 4 : 0;  // of this warp
  const int* bt = a.block_tables + static_cast<size_t>(b) * a.max_blocks;
  if (tid == 0) {
    for (int w = 0; w < 4; ++w)
      for (int s = 0; s < STAGES; ++s) mbar_init(&full[w][s], 1);
    abort_word = 0;
    fence_mbar_init();
  }
  __syncthreads();
  uint8_t* ring = smem + warp * STAGES * PAGE;
  int my_block = 0, issued = 0;  // lane l holds the block of this warp's page 32 c + l
  auto issue = [&](int n) {
    if ((n & 31) == 0) my_block = n + lane < count ? bt[first + 4 * (n + lane)] : 0;
    const int blk = __shfl_sync(0xffffffffu, my_block, n & 31);
    if (lane == 0) {
      mbar_expect_tx(&full[warp][n % STAGES], PAGE);
#pragma unroll
      for (int hf = 0; hf < DP / 64; ++hf)
        tma_load_3d(ring + (n % STAGES) * PAGE + hf * 2048, &tmK, &full[warp][n % STAGES], hf * 64, kh * 16, blk);
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
  const float scale2 = a.scale * LOG2E;
  float m[NT][2], l[NT][2];  // of heads nt * 8 + j2 + {0, 1}; l: this thread's keys only
#pragma unroll
  for (int nt = 0; nt < NT; ++nt) m[nt][0] = m[nt][1] = -INFINITY, l[nt][0] = l[nt][1] = 0.f;
  const int k_row = (lane & 7) + (lane & 8), k_col = lane >> 4;
  float* out = td.s + static_cast<size_t>(blockIdx.z) * td.pitch * td.hp + head0;
  const bool pairs = (head0 & 1) == 0;
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
    const uint32_t kb0 = smem_u32(ring + (n % STAGES) * PAGE);
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
    __syncwarp();  // every lane has read this page
    if (n + STAGES < count) issue(n + STAGES);
    const int key0 = (first + 4 * n) * 16 + r;
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int key = key0 + u * 8;
      float* row = out + static_cast<size_t>(key) * td.hp;
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        const int hd = nt * 8 + j2;
        const float x = key <= pos ? c[nt][u * 2] * scale2 : -INFINITY, y = key <= pos ? c[nt][u * 2 + 1] * scale2 : -INFINITY;
        c[nt][u * 2] = x;
        c[nt][u * 2 + 1] = y;
        if (pairs && hd + 1 < g) {
          *reinterpret_cast<float2*>(row + hd) = make_float2(x, y);
        } else {
          if (hd < g) row[hd] = x;
          if (hd + 1 < g) row[hd + 1] = y;
        }
      }
    }
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {  // per thread: its own two keys of the page
        const float top = fmaxf(m[nt][e], fmaxf(c[nt][e], c[nt][2 + e]));
        if (top > -INFINITY) {
          l[nt][e] = l[nt][e] * ex2_ftz(m[nt][e] - top) + ex2_ftz(c[nt][e] - top) + ex2_ftz(c[nt][2 + e] - top);
          m[nt][e] = top;
        }
      }
  }
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      float top = m[nt][e];
#pragma unroll
      for (int o = 4; o <= 16; o <<= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));
      float s = top == -INFINITY ? 0.f : l[nt][e] * ex2_ftz(m[nt][e] - top);
#pragma unroll
      for (int o = 4; o <= 16; o <<= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
      if (r == 0) {
        sM[warp][nt * 8 + j2 + e] = top;
        sL[warp][nt * 8 + j2 + e] = s;
      }
    }
  __syncthreads();
  if (tid < g) {
    float top = -INFINITY, s = 0.f;
    for (int w = 0; w < 4; ++w) top = fmaxf(top, sM[w][tid]);
    for (int w = 0; w < 4; ++w) s += sM[w][tid] == -INFINITY ? 0.f : sL[w][tid] * ex2_ftz(sM[w][tid] - top);
    td.stats[(static_cast<size_t>(blockIdx.z) * splits + split) * a.h + head0 + tid] = make_float2(top, s);
  }
}

// ---- values --------------------------------------------------------------------------------------------------------------
template <int DVP>
struct TalkStreamSmem {
  static constexpr int PAGE = 16 * DVP * 2;
  static constexpr int LDO = DVP + 4;
  static constexpr int MERGE = 4 * 16 * LDO * 4;  // over the ring, once every page has been multiplied
  static constexpr int TOTAL = (PageRing<PAGE>::RING > MERGE ? PageRing<PAGE>::RING : MERGE) + 1024;
};

template <int DVP, int NT, int HK>
__global__ void __launch_bounds__(128)
talking_stream_kernel(const __grid_constant__ CUtensorMap tmV, TalkArgs a, TalkDecode td, int seq_base, int groups,
                      unsigned int* err) {
  using L_ = TalkStreamSmem<DVP>;
  constexpr int PAGE = L_::PAGE, STAGES = PageRing<PAGE>::STAGES, LDO = L_::LDO;
  extern __shared__ uint8_t smem_raw[];
  __shared__ uint64_t full[4][STAGES];
  __shared__ float sLse[16 * HK];
  __shared__ int abort_word;
  volatile int* abort_flag = &abort_word;
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int splits = gridDim.x, split = blockIdx.x, kh = blockIdx.y / groups, hpart = blockIdx.y % groups;
  const int b = blockIdx.z + seq_base, gq = a.h / a.hk;
  const int head0 = kh * gq + hpart * 8 * NT, g = min(8 * NT, gq - hpart * 8 * NT);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r = lane >> 2, j2 = (lane & 3) * 2;
  const int t = a.cu_q[b], pos = a.kv_lens[b] - 1, pages = (pos >> 4) + 1;
  const int per = (pages + splits - 1) / splits;
  const int first = split * per + warp, last = min(split * per + per, pages);
  const int count = first < last ? (last - first + 3) / 4 : 0;
  const int* bt = a.block_tables + static_cast<size_t>(b) * a.max_blocks;
  if (tid == 0) {
    for (int w = 0; w < 4; ++w)
      for (int s = 0; s < STAGES; ++s) mbar_init(&full[w][s], 1);
    abort_word = 0;
    fence_mbar_init();
  }
  __syncthreads();
  uint8_t* ring = smem + warp * STAGES * PAGE;
  int my_block = 0, issued = 0;
  auto issue = [&](int n) {
    if ((n & 31) == 0) my_block = n + lane < count ? bt[first + 4 * (n + lane)] : 0;
    const int blk = __shfl_sync(0xffffffffu, my_block, n & 31);
    if (lane == 0) {
      mbar_expect_tx(&full[warp][n % STAGES], PAGE);
#pragma unroll
      for (int hf = 0; hf < DVP / 64; ++hf)
        tma_load_3d(ring + (n % STAGES) * PAGE + hf * 2048, &tmV, &full[warp][n % STAGES], hf * 64, kh * 16, blk);
    }
    issued = n + 1;
  };
  for (int n = 0; n < STAGES && n < count; ++n) issue(n);
  // scores of this warp's next page: rows r and r + 8, heads 16 kt + j2 + {0, 1, 8, 9}
  const float* sbase = td.s + static_cast<size_t>(blockIdx.z) * td.pitch * td.hp + j2;
  float2 sc[HK][4];
  auto fetch = [&](int n) {
    const float* row = sbase + static_cast<size_t>((first + 4 * n) * 16 + r) * td.hp;
#pragma unroll
    for (int kt = 0; kt < HK; ++kt)
#pragma unroll
      for (int e = 0; e < 4; ++e)
        sc[kt][e] = *reinterpret_cast<const float2*>(row + (e & 1) * 8 * td.hp + kt * 16 + (e >> 1) * 8);
  };
  if (count > 0) fetch(0);
  for (int i = tid; i < 16 * HK; i += 128) {
    float top = 0.f, s = 1.f;
    if (i < a.h) {
      const float2* st = td.stats + static_cast<size_t>(blockIdx.z) * td.score_splits * a.h + i;
      const float sink = a.sink[i] * LOG2E;
      top = sink;
      for (int p = 0; p < td.score_splits; ++p) top = fmaxf(top, st[p * a.h].x);
      s = ex2_ftz(sink - top);
      for (int p = 0; p < td.score_splits; ++p) s += st[p * a.h].y * ex2_ftz(st[p * a.h].x - top);
    }
    sLse[i] = top + log2f(s);
  }
  uint32_t tf[HK][NT][2];  // the mix, from heads on the rows: talk[head0 + 8 nt + r][16 kt + j2 + ...]
#pragma unroll
  for (int kt = 0; kt < HK; ++kt)
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int to = nt * 8 + r, from = kt * 16 + u * 8 + j2;
        const float* row = a.talk + static_cast<size_t>(head0 + to) * a.h + from;
        tf[kt][nt][u] = pack_bf16(to < g && from < a.h ? row[0] : 0.f, to < g && from + 1 < a.h ? row[1] : 0.f);
      }
  __syncthreads();
  float ls[HK][4];
#pragma unroll
  for (int kt = 0; kt < HK; ++kt)
#pragma unroll
    for (int e = 0; e < 4; ++e) ls[kt][e] = sLse[kt * 16 + (e >> 1) * 8 + j2 + (e & 1)];
  float acc[DVP / 16][NT][4];
#pragma unroll
  for (int i = 0; i < DVP / 16; ++i)
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int u = 0; u < 4; ++u) acc[i][nt][u] = 0.f;
  const int v_row = (lane & 7) + ((lane >> 4) << 3), v_col = (lane >> 3) & 1;
  bool ok = true;
  for (int n = 0; n < count; ++n) {
    uint32_t ph[HK][4], pl[HK][4];
#pragma unroll
    for (int kt = 0; kt < HK; ++kt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int from = kt * 16 + (e >> 1) * 8 + j2;
        const float x = from < a.h ? ex2_ftz(sc[kt][e].x - ls[kt][(e >> 1) * 2]) : 0.f;
        const float y = from + 1 < a.h ? ex2_ftz(sc[kt][e].y - ls[kt][(e >> 1) * 2 + 1]) : 0.f;
        ph[kt][e] = split_bf16(x, y, &pl[kt][e]);
      }
    if (n + 1 < count) fetch(n + 1);
    uint32_t wh[NT][2], wl[NT][2];
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
      float c[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int kt = 0; kt < HK; ++kt) {
        mma_16816(c, ph[kt], tf[kt][nt][0], tf[kt][nt][1]);
        mma_16816(c, pl[kt], tf[kt][nt][0], tf[kt][nt][1]);
      }
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        uint32_t low;
        wh[nt][u] = transpose_8x8(split_bf16(c[u * 2], c[u * 2 + 1], &low));
        wl[nt][u] = transpose_8x8(low);
      }
    }
    ok = mbar_wait_bounded(&full[warp][n % STAGES], (n / STAGES) & 1, abort_flag, err);
    if (!__all_sync(0xffffffffu, ok)) {
      ok = false;
      // copies in flight still write to this CTA's memory: give them their (bounded) time before leaving
      for (int i = n; i < issued; ++i)
        for (int it = 0; it < (1 << 20) && !mbar_try_wait(&full[warp][i % STAGES], (i / STAGES) & 1); ++it) {}
      break;
    }
    const uint32_t vb0 = smem_u32(ring + (n % STAGES) * PAGE);
#pragma unroll
    for (int i = 0; i < DVP / 16; ++i) {
      uint32_t f[4];
      const int ch = i * 2 + v_col;
      ldmatrix_x4<true>(f, vb0 + (ch >> 3) * 2048 + v_row * 128 + (((ch & 7) ^ (v_row & 7)) << 4));
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        mma_16816(acc[i][nt], f, wh[nt][0], wh[nt][1]);
        mma_16816(acc[i][nt], f, wl[nt][0], wl[nt][1]);
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
      const int hd = nt * 8 + j2 + e;
      if (hd < g) {
        float* dst = sO + (warp * g + hd) * LDO + r;
#pragma unroll
        for (int i = 0; i < DVP / 16; ++i) {
          dst[i * 16] = acc[i][nt][e];
          dst[i * 16 + 8] = acc[i][nt][2 + e];
        }
      }
    }
  __syncthreads();
  const int octs = a.dv / 8;
  for (int e = tid; e < g * octs * 2; e += 128) {
    const int hd = e / (octs * 2), col = e % (octs * 2) * 4;
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int w = 0; w < 4; ++w) {
      const float4 v = *reinterpret_cast<const float4*>(sO + (w * g + hd) * LDO + col);
      s.x += v.x; s.y += v.y; s.z += v.z; s.w += v.w;
    }
    *reinterpret_cast<float4*>(sO + hd * LDO + col) = s;  // only this thread reads or writes these elements of warp 0's part
  }
  __syncwarp();
  if (splits > 1)
    cluster_sync_all();
  else
    __syncthreads();
  for (int e = split * 128 + tid; e < g * octs; e += splits * 128) {
    const int hd = e / octs, col = e % octs * 8;
    float o[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    for (int s = 0; s < splits; ++s)
#pragma unroll
      for (int u = 0; u < 8; u += 4) {
        const float4 v = splits == 1 ? *reinterpret_cast<const float4*>(sO + hd * LDO + col + u)
                                     : ld_cluster_f4(mapa_u32(smem_u32(sO + hd * LDO + col + u), s));
        o[u] += v.x; o[u + 1] += v.y; o[u + 2] += v.z; o[u + 3] += v.w;
      }
    talk_store8(a, t, (head0 + hd) * a.dv + col, o);
  }
  __syncwarp();
  if (splits > 1) cluster_sync_all();  // nobody leaves while its memory is still read
}

// ---- launches ------------------------------------------------------------------------------------------------------------
static int talk_splits(long long base, int pages, int most) {
  int splits = 1;
  while (splits < most && base * splits < 8ll * sm_count() && pages / (splits * 2) >= 8) splits *= 2;
  return splits;
}
constexpr int TALK_MAX_SPLITS = 8;

template <int DP, int NT>
static int launch_scores(const TalkArgs& a, const CUtensorMap& tk, const TalkDecode& td, int seq_base, int num_seqs,
                         cudaStream_t st) {
  const int gq = a.h / a.hk, groups = (gq + 8 * NT - 1) / (8 * NT);
  constexpr int smem = PageRing<16 * DP * 2>::RING + 1024;
  auto kern = talking_scores_kernel<DP, NT>;
  if (KSANA_SMEM_ONCE(kern, smem) != 0) return -4;
  kern<<<dim3(td.score_splits, a.hk * groups, num_seqs), 128, smem, st>>>(tk, a, td, seq_base, groups, error_word());
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}
template <int DVP, int NT, int HK>
static int launch_stream(const TalkArgs& a, const CUtensorMap& tv, const TalkDecode& td, int seq_base, int num_seqs, int pages,
                         cudaStream_t st) {
  const int gq = a.h / a.hk, groups = (gq + 8 * NT - 1) / (8 * NT);
  auto kern = talking_stream_kernel<DVP, NT, HK>;
  if (KSANA_SMEM_ONCE(kern, TalkStreamSmem<DVP>::TOTAL) != 0) return -4;
  const int splits = talk_splits(static_cast<long long>(num_seqs) * a.hk * groups, pages, TALK_MAX_SPLITS);
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(splits, a.hk * groups, num_seqs);
  cfg.blockDim = dim3(128);
  cfg.dynamicSmemBytes = TalkStreamSmem<DVP>::TOTAL;
  cfg.stream = st;
  cudaLaunchAttribute at[1];
  at[0].id = cudaLaunchAttributeClusterDimension;
  at[0].val.clusterDim.x = splits;
  at[0].val.clusterDim.y = at[0].val.clusterDim.z = 1;
  cfg.attrs = at;
  cfg.numAttrs = 1;
  return cudaLaunchKernelEx(&cfg, kern, tv, a, td, seq_base, groups, error_word()) == cudaSuccess ? 0 : -5;
}
template <int DVP, int HK>
static int launch_stream_nt(const TalkArgs& a, const CUtensorMap& tv, const TalkDecode& td, int seq_base, int num_seqs,
                            int pages, cudaStream_t st) {
  return a.h / a.hk <= 8 ? launch_stream<DVP, 1, HK>(a, tv, td, seq_base, num_seqs, pages, st)
                         : launch_stream<DVP, 2, HK>(a, tv, td, seq_base, num_seqs, pages, st);
}

static int talk_hp(int h) { return h <= 16 ? 16 : h <= 32 ? 32 : 64; }

}  // namespace ksana

using namespace ksana;

// Scratch bytes of ksana_talking_decode for `num_seqs` sequences of at most max_kv keys.
KSANA_API long long ksana_talking_decode_bytes(int h, int num_seqs, int max_kv) {
  const long long pitch = (max_kv + 15) / 16 * 16;
  return num_seqs * (pitch * talk_hp(h) * 4 + static_cast<long long>(TALK_MAX_SPLITS) * h * 8) + 512;
}

// bf16. Sequences [seq_base, seq_base + num_seqs) with exactly one new token each. Returns -1 for sizes it does not take
// (pages of 16 tokens, at most 64 heads, heads of at most 128 dimensions in multiples of 8, 16-byte aligned rows).
KSANA_API int ksana_talking_decode(const void* q, int ldq, const void* cache, int num_blocks, const int* block_tables,
                                   int max_blocks, const int* cu_q, const int* kv_lens, int h, int hk, int d, int dv, int bs,
                                   float scale, const float* sink, const float* talk, float out_scale, const void* gate,
                                   int ldg, void* out, int ldo, int seq_base, int num_seqs, int max_kv, void* scratch,
                                   long long scratch_bytes, cudaStream_t st) {
  if (num_seqs <= 0) return 0;
  TalkArgs a{q, ldq, cache, block_tables, max_blocks, cu_q, kv_lens, nullptr, h, hk, d, dv, bs, scale, sink, talk,
             out_scale, gate, ldg, out, ldo};
  if (!talk_tc_sizes(a)) return -1;
  if (scratch_bytes < ksana_talking_decode_bytes(h, num_seqs, max_kv)) return -6;
  const int pages = (max_kv + 15) / 16, gq = h / hk, groups = gq <= 8 ? 1 : (gq + 15) / 16;
  char* base = reinterpret_cast<char*>((reinterpret_cast<uintptr_t>(scratch) + 255) & ~uintptr_t(255));
  TalkDecode td;
  td.pitch = pages * 16;
  td.hp = talk_hp(h);
  td.score_splits = talk_splits(static_cast<long long>(num_seqs) * hk * groups, pages, TALK_MAX_SPLITS);
  td.stats = reinterpret_cast<float2*>(base);
  td.s = reinterpret_cast<float*>(base + (static_cast<long long>(num_seqs) * TALK_MAX_SPLITS * h * 8 + 255) / 256 * 256);
  CUtensorMap tk, tv;
  if (int rc = talk_cache_map(a, num_blocks, 0, &tk)) return rc;
  if (int rc = talk_cache_map(a, num_blocks, 1, &tv)) return rc;
  int rc;
  if (d <= 64)
    rc = gq <= 8 ? launch_scores<64, 1>(a, tk, td, seq_base, num_seqs, st) : launch_scores<64, 2>(a, tk, td, seq_base, num_seqs, st);
  else
    rc = gq <= 8 ? launch_scores<128, 1>(a, tk, td, seq_base, num_seqs, st) : launch_scores<128, 2>(a, tk, td, seq_base, num_seqs, st);
  if (rc) return rc;
#define KSANA_TS(DVP)                                                                               \
  return h <= 16   ? launch_stream_nt<DVP, 1>(a, tv, td, seq_base, num_seqs, pages, st)             \
         : h <= 32 ? launch_stream_nt<DVP, 2>(a, tv, td, seq_base, num_seqs, pages, st)             \
                   : launch_stream_nt<DVP, 4>(a, tv, td, seq_base, num_seqs, pages, st)
  if (dv <= 64) KSANA_TS(64);
  KSANA_TS(128);
#undef KSANA_TS
}
