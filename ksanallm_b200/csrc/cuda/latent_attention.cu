// Latent attention over pages of 16 tokens: the cache holds one RMS-normed latent and one rotated key part per token,
// [block][16 x (rank + rot)].
#include "host_common.h"
#include "mixer_common.cuh"

namespace ksana {

// ---- what happens between the projections and the scores -------------------------------------------------------------
// One warp per (token, head): the last rot dimensions of a query head are rotated in place (pairs (2i, 2i + 1)), and
// also written behind the head's absorbed query in q_cat for tokens from cat_from on. One further warp per token: the
// latent's RMS norm and the rotated key part go to the cache.
template <typename T>
__global__ void __launch_bounds__(256)
latent_append_kernel(T* __restrict__ q, int ldq, int dim, T* __restrict__ q_cat, int cat_from, const T* __restrict__ x,
                     int ldx, const float* __restrict__ norm_w, float eps, const int* __restrict__ positions,
                     const float* __restrict__ rotary, const int* __restrict__ slots, T* __restrict__ cache, int tokens,
                     int h, int rank, int rd) {
  const int units = h + 1;
  const long long unit = static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (unit >= static_cast<long long>(tokens) * units) return;
  const int t = static_cast<int>(unit / units), hd = static_cast<int>(unit % units);
  const float* cs = rotary + static_cast<size_t>(positions[t]) * rd;
  const int half = rd / 2;
  if (hd < h) {
    T* src = q + static_cast<size_t>(t) * ldq + static_cast<size_t>(hd) * (dim + rd) + dim;
    T* cat = q_cat && t >= cat_from ? q_cat + (static_cast<size_t>(t - cat_from) * h + hd) * (rank + rd) + rank : nullptr;
    for (int i = lane; i < half; i += 32) {
      const float a = to_f(src[2 * i]), b = to_f(src[2 * i + 1]), c = cs[i], s = cs[half + i];
      const T u = from_f<T>(a * c - b * s), v = from_f<T>(b * c + a * s);
      src[2 * i] = u;
      src[2 * i + 1] = v;
      if (cat) {
        cat[2 * i] = u;
        cat[2 * i + 1] = v;
      }
    }
    return;
  }
  if (slots[t] < 0) return;
  const T* a = x + static_cast<size_t>(t) * ldx;
  T* dst = cache + static_cast<size_t>(slots[t]) * (rank + rd);
  float ss = 0.f;
  for (int i = lane; i < rank; i += 32) {
    const float f = to_f(a[i]);
    ss += f * f;
  }
  const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(rank) + eps);
  for (int i = lane; i < rank; i += 32) dst[i] = from_f<T>(to_f(a[i]) * inv * norm_w[i]);
  for (int i = lane; i < half; i += 32) {
    const float u = to_f(a[rank + 2 * i]), v = to_f(a[rank + 2 * i + 1]), c = cs[i], s = cs[half + i];
    dst[rank + 2 * i] = from_f<T>(u * c - v * s);
    dst[rank + 2 * i + 1] = from_f<T>(v * c + u * s);
  }
}

// The contexts of sequences [seq_base, seq_base + gridDim.y), row by row behind one another: [rows][rank + rot]. One warp
// per row, 16 bytes per lane.
__global__ void __launch_bounds__(256)
latent_gather_kernel(const uint4* __restrict__ cache, const int* __restrict__ block_tables, int max_blocks,
                     const int* __restrict__ kv_lens, int seq_base, int bs, int words, uint4* __restrict__ out) {
  const int b = seq_base + blockIdx.y, L = kv_lens[b];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int j0 = blockIdx.x * 32;
  if (j0 >= L) return;
  int row0 = 0;
  for (int i = seq_base + lane; i < b; i += 32) row0 += kv_lens[i];
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) row0 += __shfl_xor_sync(0xffffffffu, row0, o);
  for (int j = j0 + warp; j < min(j0 + 32, L); j += 8) {
    const uint4* src = cache + (static_cast<size_t>(block_tables[static_cast<size_t>(b) * max_blocks + j / bs]) * bs + j % bs) * words;
    uint4* dst = out + static_cast<size_t>(row0 + j) * words;
    for (int i = lane; i < words; i += 32) dst[i] = src[i];
  }
}

// ---- single tokens: tcgen05, keys on the MMA rows --------------------------------------------------------------------
// All heads share the cached vectors, and a vector's first `rank` numbers are its value. One CTA = one new token x NH
// heads x one split of the context, 192 threads; the splits of a token form a cluster that merges through distributed
// shared memory. Per tile of 128 tokens (8 pages):
//   S^T = C Q^T        128 tokens x NH heads, the tile's 64-column chunks K-major          -> TMEM, NH columns
//   softmax            thread = token; weights as two bf16 matrices hi | lo, 2 NH columns  -> shared memory
//   O^T += C^T [P_hi | P_lo]   blocks of 128 value dimensions, the same chunks MN-major    -> TMEM, 2 NH columns a block
// so small head counts cost no padding rows and both products read one copy of the tile. The tile is single buffered, but
// its chunks are refilled one by one: those without values when the scores are out, the others behind their block's
// product; meanwhile the next tile's pages come into L2.
//   warps 0-3  softmax: thread t = token t of the tile, and value dimension t of each block
//   warp 4     one lane issues the MMAs        warp 5     one lane issues the loads
// Running maxima move only when a score exceeds one by more than 8 (x 256), as a vote over the warps.
constexpr int LD_PAGE = 16, LD_TILE = 128, LD_CHUNK = LD_TILE * 128, LD_MAX_CHUNKS = 9, LD_MAX_BLOCKS = 4;

struct LatentDecodeArgs {
  const __nv_bfloat16* cache;
  const int* block_tables;
  int max_blocks;
  const int* cu_q;
  const int* kv_lens;
  int h, width, rank, chunks, blocks, slots, groups, max_q, seq_base;  // slots: chunks a tile has room for
  float scale2;
  const __nv_bfloat16* gate;  // by token of the step
  int ldg;
  __nv_bfloat16* out;         // [token][h * rank] (pitch ldo)
  int ldo;
};

template <int NH>
__host__ __device__ constexpr int latent_decode_smem(int slots, int chunks) {
  return slots * LD_CHUNK + chunks * NH * 128 + NH * 512 + 3 * 4 * NH * 4 + 256 + 1024;
}

// true in every one of the 128 softmax threads when it is true in any
__device__ __forceinline__ bool vote128(bool v) {
  uint32_t r;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.u32 p, %1, 0;\n\t"
      "barrier.cta.red.or.pred q, 1, 128, p;\n\t"
      "selp.u32 %0, 1, 0, q;\n\t}"
      : "=r"(r) : "r"(v ? 1u : 0u) : "memory");
  return r != 0;
}
__device__ __forceinline__ int float_key(float f) {  // ordered as the floats are
  const int b = __float_as_int(f);
  return b ^ ((b >> 31) & 0x7fffffff);
}

template <int NH>
__device__ __forceinline__ void tmem_ld_n(uint32_t addr, uint32_t* r) {
  if constexpr (NH == 32) tmem_ld32(addr, r); else tmem_ld16(addr, r);
}
template <int NH>
__device__ __forceinline__ void tmem_st_n(uint32_t addr, const uint32_t* r) {
  if constexpr (NH == 32) tmem_st32(addr, r); else tmem_st16(addr, r);
}

template <int NH>
__global__ void __launch_bounds__(192)
latent_decode_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmC, LatentDecodeArgs a,
                     int tmem_cols, unsigned int* err) {
  const int splits = gridDim.x, split = blockIdx.x;
  const int head0 = blockIdx.y * NH, g = min(NH, a.h - head0);
  const int b = a.seq_base + blockIdx.z / a.max_q, j = blockIdx.z % a.max_q;
  const int q0 = a.cu_q[b], q_len = a.cu_q[b + 1] - q0;
  if (j >= q_len) return;  // the whole cluster
  const int t = q0 + j;
  const int pos = a.kv_lens[b] - q_len + j;
  const int tiles = pos / LD_TILE + 1, per = (tiles + splits - 1) / splits;
  const int first = split * per, n_it = max(min(tiles - first, per), 0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;

  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sC = smem;
  uint8_t* sQ = sC + a.slots * LD_CHUNK;
  uint8_t* sP = sQ + a.chunks * NH * 128;
  float* red = reinterpret_cast<float*>(sP + NH * 512);  // [4][NH] maxima, then sums
  float* cM = red + 4 * NH;
  float* cL = cM + NH;
  uint64_t* bars = reinterpret_cast<uint64_t*>(red + 12 * NH);
  uint64_t* q_bar = bars;
  uint64_t* full = bars + 1;                   // [LD_MAX_CHUNKS]
  uint64_t* s_done = full + LD_MAX_CHUNKS;
  uint64_t* p_ready = s_done + 1;
  uint64_t* v_done = p_ready + 1;              // [LD_MAX_BLOCKS]
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(v_done + LD_MAX_BLOCKS);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_holder + 1);
  if (tid == 0) {
    mbar_init(q_bar, 1);
    for (int c = 0; c < LD_MAX_CHUNKS; ++c) mbar_init(&full[c], 1);
    mbar_init(s_done, 1);
    mbar_init(p_ready, 128);
    for (int i = 0; i < LD_MAX_BLOCKS; ++i) mbar_init(&v_done[i], 1);
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 4) {
    tmem_alloc(tmem_holder, tmem_cols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_S = *tmem_holder, tmem_O = tmem_S + NH;
  const int v_chunks = min(2 * a.blocks, a.chunks);
  // the order in which a tile's chunks are loaded and multiplied: those without values first
  auto chunk_at = [&](int i) { return i < a.chunks - v_chunks ? v_chunks + i : i - (a.chunks - v_chunks); };
  bool bad = false;
  float m_ref[NH], l[NH];

  if (warp == 5) {
    if (lane == 0 && n_it > 0) {
      const int* bt = a.block_tables + static_cast<size_t>(b) * a.max_blocks;
      const int pages = pos / LD_PAGE + 1;
      mbar_expect_tx(q_bar, a.chunks * NH * 128);
      for (int c = 0; c < a.chunks; ++c) tma_load_3d(sQ + c * NH * 128, &tmQ, q_bar, c * 64, head0, t);
      int loads = 0;  // of chunks, in order
      bool ok = true;
      for (int it = 0; it < n_it && ok; ++it) {
        int blk[LD_TILE / LD_PAGE];
#pragma unroll
        for (int p = 0; p < LD_TILE / LD_PAGE; ++p)  // pages past the context repeat its last one (masked)
          blk[p] = bt[min((first + it) * (LD_TILE / LD_PAGE) + p, pages - 1)];
        for (int i = 0; i < a.chunks; ++i) {
          const int c = chunk_at(i);
          if (it > 0) {
            ok = mbar_wait_bounded(c < v_chunks ? &v_done[c >> 1] : s_done, (it - 1) & 1, abort_flag, err);
            if (!ok) break;
          }
          mbar_expect_tx(&full[c], LD_CHUNK);
#pragma unroll
          for (int p = 0; p < LD_TILE / LD_PAGE; ++p)
            tma_load_2d(sC + c * LD_CHUNK + p * (LD_PAGE * 128), &tmC, &full[c], c * 64, blk[p] * LD_PAGE);
          ++loads;
        }
        if (it + 1 < n_it)
#pragma unroll
          for (int p = 0; p < LD_TILE / LD_PAGE; ++p) {
            const int pg = (first + it + 1) * (LD_TILE / LD_PAGE) + p;
            if (pg < pages)
              l2_prefetch(a.cache + static_cast<size_t>(bt[pg]) * LD_PAGE * a.width, LD_PAGE * a.width * 2);
          }
      }
      if (!ok) {
        // copies in flight still write to this CTA's memory: give them their (bounded) time before leaving
        for (int n = max(loads - a.chunks, 0); n < loads; ++n)
          for (int s = 0; s < (1 << 20) && !mbar_try_wait(&full[chunk_at(n % a.chunks)], (n / a.chunks) & 1); ++s) {}
        for (int s = 0; s < (1 << 20) && !mbar_try_wait(q_bar, 0); ++s) {}
      }
    }
    __syncwarp();
  } else if (warp == 4) {
    if (lane == 0 && n_it > 0) {
      bool ok = mbar_wait_bounded(q_bar, 0, abort_flag, err);
      constexpr uint32_t idesc_s = umma_idesc(128, NH, 1, 1), idesc_o = umma_idesc_major(128, 2 * NH, true, false);
      const uint32_t cb = smem_u32(sC), qb = smem_u32(sQ), pb = smem_u32(sP);
      for (int it = 0; ok && it < n_it; ++it) {
        for (int i = 0; i < a.chunks; ++i) {
          const int c = chunk_at(i);
          ok = mbar_wait_bounded(&full[c], it & 1, abort_flag, err);
          if (!ok) break;
          tc_fence_after();
#pragma unroll
          for (int k = 0; k < 4; ++k)
            umma_f16(tmem_S, umma_desc_k128(cb + c * LD_CHUNK + k * 32), umma_desc_k128(qb + c * NH * 128 + k * 32), idesc_s,
                     i > 0 || k > 0 ? 1u : 0u);
        }
        if (!ok) break;
        umma_commit(s_done);
        ok = mbar_wait_bounded(p_ready, it & 1, abort_flag, err);
        if (!ok) break;
        tc_fence_after();
        for (int i = 0; i < a.blocks; ++i) {
#pragma unroll
          for (int k = 0; k < LD_TILE / 16; ++k)
            umma_f16(tmem_O + i * 2 * NH, umma_desc_mn128(cb + 2 * i * LD_CHUNK + k * (16 * 128), LD_CHUNK),
                     umma_desc_k128(pb + (k >> 2) * (2 * NH * 128) + (k & 3) * 32), idesc_o, it > 0 || k > 0 ? 1u : 0u);
          umma_commit(&v_done[i]);
        }
      }
    }
    __syncwarp();
  } else {
    const uint32_t lane_off = static_cast<uint32_t>(warp * 32) << 16;
#pragma unroll
    for (int n = 0; n < NH; ++n) m_ref[n] = -INFINITY, l[n] = 0.f;
    for (int it = 0; it < n_it; ++it) {
      bad = !mbar_wait_bounded(s_done, it & 1, abort_flag, err);
      tc_fence_after();
      float s[NH];
      __syncwarp();
      tmem_ld_n<NH>(tmem_S + lane_off, reinterpret_cast<uint32_t*>(s));
      tmem_wait_ld();
      const bool seen = (first + it) * LD_TILE + tid <= pos;
      bool grown = false;
#pragma unroll
      for (int n = 0; n < NH; ++n) {
        s[n] = seen ? s[n] * a.scale2 : -INFINITY;
        grown = grown || s[n] > m_ref[n] + 8.f;
      }
      if (vote128(bad)) {
        bad = true;
        break;
      }
      if (vote128(grown)) {
#pragma unroll
        for (int n = 0; n < NH; ++n) {
          const int k = __reduce_max_sync(0xffffffffu, float_key(s[n]));
          if (lane == 0) red[warp * NH + n] = __int_as_float(k ^ ((k >> 31) & 0x7fffffff));
        }
        vote128(false);
        float f[NH];
#pragma unroll
        for (int n = 0; n < NH; ++n) {
          const float m = fmaxf(m_ref[n], fmaxf(fmaxf(red[n], red[NH + n]), fmaxf(red[2 * NH + n], red[3 * NH + n])));
          f[n] = m_ref[n] == -INFINITY ? 1.f : ex2_ftz(m_ref[n] - m);
          m_ref[n] = m;
          l[n] *= f[n];
        }
        vote128(false);  // the maxima have been read
        if (it > 0) {  // scores are out, so the products before them are in
          for (int i = 0; i < 2 * a.blocks; ++i) {
            uint32_t o[NH];
            tmem_ld_n<NH>(tmem_O + lane_off + i * NH, o);
            tmem_wait_ld();
#pragma unroll
            for (int n = 0; n < NH; ++n) o[n] = __float_as_uint(__uint_as_float(o[n]) * f[n]);
            tmem_st_n<NH>(tmem_O + lane_off + i * NH, o);
          }
          tmem_wait_st();
        }
      }
      uint8_t* base = sP + (tid >> 6) * (2 * NH * 128) + (tid & 7) * 2;
      const int chunk = (tid & 63) >> 3;
#pragma unroll
      for (int n = 0; n < NH; ++n) {
        const float p = ex2_ftz(s[n] - m_ref[n]);  // (m_ref is finite: every tile holds a visible token)
        l[n] += p;
        const __nv_bfloat16 hi = __float2bfloat16_rn(p);
        *reinterpret_cast<__nv_bfloat16*>(base + n * 128 + ((chunk ^ (n & 7)) << 4)) = hi;
        *reinterpret_cast<__nv_bfloat16*>(base + (NH + n) * 128 + ((chunk ^ (n & 7)) << 4)) =
            __float2bfloat16_rn(p - __bfloat162float(hi));
      }
      fence_async_smem();
      tc_fence_before();
      mbar_arrive(p_ready);
    }
    if (!bad && n_it > 0) bad = !mbar_wait_bounded(&v_done[a.blocks - 1], (n_it - 1) & 1, abort_flag, err);
    tc_fence_after();
    __syncwarp();
  }
  __syncthreads();  // every load and product is through with the tile: the results go over it
  const int ldo = a.rank + 4;
  float* sO = reinterpret_cast<float*>(sC);  // [g][ldo]
  if (warp < 4) {
    const uint32_t lane_off = static_cast<uint32_t>(warp * 32) << 16;
    tc_fence_after();
#pragma unroll
    for (int n = 0; n < NH; ++n) {
      const float v = warp_sum(l[n]);
      if (lane == 0) red[warp * NH + n] = v;
      if (tid == 0) cM[n] = m_ref[n];
    }
    for (int i = 0; i < a.blocks && n_it > 0; ++i) {
      uint32_t hi[NH], lo[NH];
      tmem_ld_n<NH>(tmem_O + lane_off + i * 2 * NH, hi);
      tmem_ld_n<NH>(tmem_O + lane_off + i * 2 * NH + NH, lo);
      tmem_wait_ld();
      if (i * 128 + tid < a.rank)
#pragma unroll
        for (int n = 0; n < NH; ++n)
          if (n < g) sO[n * ldo + i * 128 + tid] = __uint_as_float(hi[n]) + __uint_as_float(lo[n]);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 4) {
    tc_fence_after();
    tmem_dealloc(tmem_S, tmem_cols);
  }
  if (tid < NH) cL[tid] = red[tid] + red[NH + tid] + red[2 * NH + tid] + red[3 * NH + tid];
  __syncwarp();
  if (splits > 1)
    cluster_sync_all();
  else
    __syncthreads();
  __nv_bfloat16* out = a.out + static_cast<size_t>(t) * a.ldo + static_cast<size_t>(head0) * a.rank;
  const int quads = a.rank / 4;
  for (int e = split * 192 + tid; e < g * quads; e += splits * 192) {
    const int hd = e / quads, col = e % quads * 4;
    float M = -INFINITY, S = 0.f, o[4] = {0.f, 0.f, 0.f, 0.f};
    if (splits == 1) {
      S = cL[hd];
      const float4 v = *reinterpret_cast<const float4*>(sO + hd * ldo + col);
      o[0] = v.x; o[1] = v.y; o[2] = v.z; o[3] = v.w;
    } else {
      for (int s = 0; s < splits; ++s) M = fmaxf(M, ld_cluster_f1(mapa_u32(smem_u32(cM + hd), s)));
      for (int s = 0; s < splits; ++s) {
        const float m = ld_cluster_f1(mapa_u32(smem_u32(cM + hd), s));
        if (m == -INFINITY) continue;  // a split without tokens
        const float f = exp2f(m - M);
        S += f * ld_cluster_f1(mapa_u32(smem_u32(cL + hd), s));
        const float4 v = ld_cluster_f4(mapa_u32(smem_u32(sO + hd * ldo + col), s));
        o[0] += f * v.x; o[1] += f * v.y; o[2] += f * v.z; o[3] += f * v.w;
      }
    }
    float inv = 1.f / S;
    if (a.gate) inv *= sigmoid_f(__bfloat162float(a.gate[static_cast<size_t>(t) * a.ldg + head0 + hd]));
#pragma unroll
    for (int u = 0; u < 4; ++u) o[u] *= inv;
    store_n<4>(out + static_cast<size_t>(hd) * a.rank + col, o);
  }
  __syncwarp();
  if (splits > 1) cluster_sync_all();  // nobody leaves while its memory is still read
}

template <int NH>
static int launch_latent_decode(const LatentDecodeArgs& a, const void* q, int ldq, int total_tokens, int num_blocks,
                                int num_seqs, int max_kv, cudaStream_t st) {
  CUtensorMap tq, tc;
  {
    const uint64_t dims[3] = {static_cast<uint64_t>(a.width), static_cast<uint64_t>(a.h), static_cast<uint64_t>(total_tokens)};
    const uint64_t str[2] = {static_cast<uint64_t>(a.width) * 2, static_cast<uint64_t>(ldq) * 2};
    const uint32_t box[3] = {64, NH, 1};
    if (make_tmap_nd(&tq, q, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, dims, str, box, CU_TENSOR_MAP_SWIZZLE_128B)) return -2;
  }
  if (make_tmap_2d(&tc, a.cache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, static_cast<uint64_t>(num_blocks) * LD_PAGE, a.width,
                   a.width, LD_PAGE, 64, CU_TENSOR_MAP_SWIZZLE_128B))
    return -3;
  auto kern = latent_decode_kernel<NH>;
  if (KSANA_SMEM_ONCE(kern, latent_decode_smem<NH>(LD_MAX_CHUNKS, LD_MAX_CHUNKS)) != 0) return -4;
  const int need = NH + a.blocks * 2 * NH;
  int cols = 32;
  while (cols < need) cols *= 2;
  const int smem = latent_decode_smem<NH>(a.slots, a.chunks);
  const int resident = sm_count() * (smem > 113 * 1024 || cols > 256 ? 1 : 2);
  // splits by waves of CTAs x (tiles of a split + what a CTA costs besides)
  const int tiles = (max_kv + LD_TILE - 1) / LD_TILE;
  const long long base = static_cast<long long>(num_seqs) * a.max_q * a.groups;
  int splits = 1;
  float best = 1e30f;
  for (int sp = 1; sp <= 8 && sp <= tiles; sp *= 2) {
    const float cost = static_cast<float>((base * sp + resident - 1) / resident) * ((tiles + sp - 1) / sp + 2.5f + (sp > 1 ? 0.5f : 0.f));
    if (cost < best - 1e-3f) {
      best = cost;
      splits = sp;
    }
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(splits, a.groups, num_seqs * a.max_q);
  cfg.blockDim = dim3(192);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute at[1];
  at[0].id = cudaLaunchAttributeClusterDimension;
  at[0].val.clusterDim.x = splits;
  at[0].val.clusterDim.y = at[0].val.clusterDim.z = 1;
  cfg.attrs = at;
  cfg.numAttrs = 1;
  return cudaLaunchKernelEx(&cfg, kern, tq, tc, a, cols, error_word()) == cudaSuccess ? 0 : -5;
}

}  // namespace ksana

using namespace ksana;

// bf16. -1: rows are not multiples of 16 bytes.
KSANA_API int ksana_latent_gather(const void* cache, const int* block_tables, int max_blocks, const int* kv_lens,
                                  int seq_base, int num_seqs, int max_kv, int bs, int width, void* out, cudaStream_t st) {
  if (num_seqs <= 0 || max_kv <= 0) return 0;
  if (width & 7) return -1;
  latent_gather_kernel<<<dim3((max_kv + 31) / 32, num_seqs), 256, 0, st>>>(
      static_cast<const uint4*>(cache), block_tables, max_blocks, kv_lens, seq_base, bs, width / 8,
      static_cast<uint4*>(out));
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

// q: [tokens, h * (dim + rot)] (pitch ldq); q_cat: [tokens - cat_from, h, rank + rot] or null; x: [tokens, rank + rot]
// (pitch ldx). A slot is a row of the cache. kind: 0 fp32, 1 bf16.
KSANA_API int ksana_latent_append(void* q, int ldq, int dim, void* q_cat, int cat_from, const void* x, int ldx,
                                  const float* norm_w, float eps, const int* positions, const float* rotary,
                                  const int* slots, void* cache, int tokens, int h, int rank, int rot, int kind,
                                  cudaStream_t st) {
  if (tokens <= 0) return 0;
  if (rot < 0 || (rot & 1) || rank < 1) return -2;
  const unsigned grid = static_cast<unsigned>((static_cast<long long>(tokens) * (h + 1) + 7) / 8);
#define KSANA_LA(T)                                                                                                 \
  latent_append_kernel<T><<<grid, 256, 0, st>>>(static_cast<T*>(q), ldq, dim, static_cast<T*>(q_cat), cat_from,     \
                                                static_cast<const T*>(x), ldx, norm_w, eps, positions, rotary,      \
                                                slots, static_cast<T*>(cache), tokens, h, rank, rot)
  if (kind) KSANA_LA(__nv_bfloat16); else KSANA_LA(float);
#undef KSANA_LA
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

// bf16. Absorbed queries q [total_tokens, h, rank + rot] (pitch ldq) over the latents: sequences [seq_base, seq_base +
// num_seqs), each with at most max_q new tokens; out [total_tokens, h * rank] = the weighted latents, times the heads' gates.
// -1: sizes it does not take (rank at most 512 and rank + rot at most 576, both multiples of 8, pages of 16 tokens).
KSANA_API int ksana_latent_decode(const void* q, int ldq, int total_tokens, const void* cache, int num_blocks,
                                  const int* block_tables, int max_blocks, const int* cu_q, const int* kv_lens, int h,
                                  int rank, int rot, int bs, float scale, const void* gate, int ldg, void* out, int ldo,
                                  int seq_base, int num_seqs, int max_q, int max_kv, cudaStream_t st) {
  if (num_seqs <= 0 || max_q <= 0) return 0;
  const int width = rank + rot;
  auto rows16 = [](const void* p, int ld) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0 && (ld & 7) == 0; };
  if (bs != LD_PAGE || (rank & 7) || (rot & 7) || rank < 8 || rank > 512 || width > 576 || h < 1 || !rows16(q, ldq) ||
      !rows16(cache, 0) || !rows16(out, ldo) || static_cast<long long>(num_seqs) * max_q > 65535)
    return -1;
  const int chunks = (width + 63) / 64, blocks = (rank + 127) / 128;
  const int slots = chunks > 2 * blocks ? chunks : 2 * blocks, nh = h <= 16 ? 16 : 32;
  LatentDecodeArgs a{static_cast<const __nv_bfloat16*>(cache), block_tables, max_blocks, cu_q, kv_lens, h, width, rank,
                     chunks, blocks, slots, (h + nh - 1) / nh, max_q, seq_base, scale * LOG2E,
                     static_cast<const __nv_bfloat16*>(gate), ldg, static_cast<__nv_bfloat16*>(out), ldo};
  return nh == 16 ? launch_latent_decode<16>(a, q, ldq, total_tokens, num_blocks, num_seqs, max_kv, st)
                  : launch_latent_decode<32>(a, q, ldq, total_tokens, num_blocks, num_seqs, max_kv, st);
}
