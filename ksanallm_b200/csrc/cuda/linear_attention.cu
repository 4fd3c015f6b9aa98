// Linear attention with a fixed decay per head over a pool of fp32 state slots: S <- decay S + k v^T, o = S^T q.
//
// q, k, v are the projections as they left the GEMM; the activation, the rotation and the key's scale are applied here
// in 32-bit floats. A sequence whose first token is part of the step starts from a zero state whatever its slot holds.
#include "host_common.h"
#include "mixer_common.cuh"

namespace ksana {

struct LinearAttnArgs {
  const void* q;
  const void* k;
  const void* v;
  int ldq, ldk, ldv;          // token pitches (elements)
  float* state;               // [slots][h][d][dv]
  const int* slots;           // [B]
  const int* cu_q;            // [B + 1]
  const int* kv_lens;         // [B]
  const int* positions;       // [T]
  const float* decay;         // [h]
  const float* rotary;        // [positions][rd] = [cos | sin], or null
  int rd, act, h, d, dv;      // act: 0 none, 1 silu
  float key_scale;
  void* out;                  // [T][h][dv]
};

template <typename T>
__device__ __forceinline__ float la_act(float x, int act) {
  return act ? silu_f(x) : x;
}

// Element c of a head of q or k after activation and rotation.
template <typename T>
__device__ __forceinline__ float la_feature(const T* head, int c, const float* cs, int rd, int act) {
  float x = la_act<T>(to_f(head[c]), act);
  if (c < rd) {
    const int half = rd >> 1;
    const bool low = c < half;
    const int i = low ? c : c - half;
    const float y = la_act<T>(to_f(head[low ? c + half : i]), act);
    x = low ? x * cs[i] - y * cs[half + i] : x * cs[i] + y * cs[half + i];
  }
  return x;
}

// ---- token by token ---------------------------------------------------------------------------------------------
// One CTA = one (sequence, head, 32 columns of the state). Thread (tx, ty) owns VEC columns and every 128 / TX-th row.
// A single new token reads and writes the state in global memory once; several keep it in shared memory between them.
template <typename T, int VEC, bool ONE>
__global__ void __launch_bounds__(128)
linear_recurrent_kernel(LinearAttnArgs a, int seq_base) {
  constexpr int TX = 32 / VEC, TY = 128 / TX;
  extern __shared__ float sm[];
  float* sq = sm;                 // [d]
  float* sk = sq + a.d;           // [d]
  float* sv = sk + a.d;           // [32]
  float* red = sv + 32;           // [TY][32]
  float* sS = red + TY * 32;      // [d][32], several tokens only
  const int b = blockIdx.z + seq_base, head = blockIdx.y, col0 = blockIdx.x * 32;
  const int slot = a.slots[b];
  const int t0 = a.cu_q[b], t1 = a.cu_q[b + 1];
  if (t1 <= t0 || slot < 0) return;
  const bool fresh = a.kv_lens[b] == t1 - t0;
  const int tid = threadIdx.x, tx = tid % TX, ty = tid / TX;
  const int col = col0 + tx * VEC;
  const bool live = col < a.dv;
  float* S = a.state + (static_cast<size_t>(slot) * a.h + head) * a.d * a.dv + col;
  const float dec = a.decay[head];
  if (!ONE && live) {
    for (int r = ty; r < a.d; r += TY) {
      float s[VEC];
#pragma unroll
      for (int j = 0; j < VEC; ++j) s[j] = 0.f;
      if (!fresh) load_n<VEC>(S + static_cast<size_t>(r) * a.dv, s);
      store_n<VEC>(sS + r * 32 + tx * VEC, s);
    }
  }
  for (int t = t0; t < t1; ++t) {
    const T* q = static_cast<const T*>(a.q) + static_cast<size_t>(t) * a.ldq + head * a.d;
    const T* k = static_cast<const T*>(a.k) + static_cast<size_t>(t) * a.ldk + head * a.d;
    const T* v = static_cast<const T*>(a.v) + static_cast<size_t>(t) * a.ldv + head * a.dv;
    const float* cs = a.rotary ? a.rotary + static_cast<size_t>(a.positions[t]) * a.rd : nullptr;
    for (int c = tid; c < a.d; c += 128) {
      sq[c] = la_feature(q, c, cs, a.rd, a.act);
      sk[c] = la_feature(k, c, cs, a.rd, a.act) * a.key_scale;
    }
    if (tid < 32 && col0 + tid < a.dv) sv[tid] = to_f(from_f<T>(la_act<T>(to_f(v[col0 + tid]), a.act)));
    __syncthreads();
    float acc[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) acc[j] = 0.f;
    if (live) {
      float vv[VEC];
#pragma unroll
      for (int j = 0; j < VEC; ++j) vv[j] = sv[tx * VEC + j];
#pragma unroll 8
      for (int r = ty; r < a.d; r += TY) {
        float s[VEC];
        if (ONE) {
#pragma unroll
          for (int j = 0; j < VEC; ++j) s[j] = 0.f;
          if (!fresh) load_n<VEC>(S + static_cast<size_t>(r) * a.dv, s);
        } else {
          load_n<VEC>(sS + r * 32 + tx * VEC, s);
        }
        const float kr = sk[r], qr = sq[r];
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          s[j] = dec * s[j] + kr * vv[j];
          acc[j] += qr * s[j];
        }
        if (ONE)
          store_n<VEC>(S + static_cast<size_t>(r) * a.dv, s);
        else
          store_n<VEC>(sS + r * 32 + tx * VEC, s);
      }
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) red[ty * 32 + tx * VEC + j] = acc[j];
    __syncthreads();
    if (tid < 32 && col0 + tid < a.dv) {
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < TY; ++i) o += red[i * 32 + tid];
      static_cast<T*>(a.out)[(static_cast<size_t>(t) * a.h + head) * a.dv + col0 + tid] = from_f<T>(o);
    }
  }
  if (!ONE && live) {
    for (int r = ty; r < a.d; r += TY) {
      float s[VEC];
      load_n<VEC>(sS + r * 32 + tx * VEC, s);
      store_n<VEC>(S + static_cast<size_t>(r) * a.dv, s);
    }
  }
}

// ---- prompts: chunks of 128 tokens on the tensor cores -----------------------------------------------------------------
// With chunk-local index i and the state S entering the chunk,
//   o_i   = sum_{j <= i} decay^(i - j) (q_i . k_j) v_j  +  decay^(i + 1) S^T q_i
//   S_out = decay^n S + sum_j decay^(n - 1 - j) k_j v_j^T          (n = tokens of the chunk)
// in three launches: every chunk's own sum of k v^T (parallel), the scan over a sequence's chunks (elementwise), and the
// outputs (parallel). What is 32-bit by definition (scores, state, rotated q and k) enters the bf16 tensor-core products
// as a pair hi + lo: x y ~ x_hi y_hi + x_lo y_hi + x_hi y_lo.
// Chunk c of sequence b has its scratch entry at (cu_q[b] - cu_q[seq_base]) / 128 + (b - seq_base) + c.
constexpr int LC = 128;

__device__ __forceinline__ size_t chunk_entry(const LinearAttnArgs& a, int seq_base, int b, int c) {
  return static_cast<size_t>((a.cu_q[b] - a.cu_q[seq_base]) / LC + (b - seq_base) + c);
}

// decay^e for e in [0, 128] (0 for a decay of 0 and e > 0)
__device__ __forceinline__ float decay_pow(float decay, int e) {
  if (e == 0) return 1.f;
  return decay > 0.f ? exp2f(static_cast<float>(e) * log2f(decay)) : 0.f;
}

// Eight consecutive features of a head of q or k after activation and rotation (c0 % 8 == 0; rd % 16 == 0).
__device__ __forceinline__ void la_feature8(const __nv_bfloat16* head, int c0, const float* cs, int rd, int act, float* f) {
  load_n<8>(head + c0, f);
  if (act) {
#pragma unroll
    for (int i = 0; i < 8; ++i) f[i] = silu_f(f[i]);
  }
  if (c0 < rd) {
    const int half = rd >> 1;
    const bool low = c0 < half;
    const int i0 = low ? c0 : c0 - half;
    float y[8], co[8], si[8];
    load_n<8>(head + (low ? c0 + half : i0), y);
    load_n<8>(cs + i0, co);
    load_n<8>(cs + half + i0, si);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const float z = act ? silu_f(y[i]) : y[i];
      f[i] = low ? f[i] * co[i] - z * si[i] : f[i] * co[i] + z * si[i];
    }
  }
}

// Row r, 8 features from c0 of a 128-row operand in the 128-byte swizzle (64-column panels of 16 KB).
__device__ __forceinline__ uint4* operand_at(uint8_t* base, int r, int c0) {
  return reinterpret_cast<uint4*>(base + (c0 >> 6) * (128 * 128) + r * 128 + ((((c0 >> 3) & 7) ^ (r & 7)) << 4));
}
__device__ __forceinline__ void store_split8(uint8_t* hi, uint8_t* lo, int r, int c0, const float* f) {
  uint32_t h[4], l[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) h[i] = split_bf16(f[2 * i], f[2 * i + 1], &l[i]);
  *operand_at(hi, r, c0) = make_uint4(h[0], h[1], h[2], h[3]);
  *operand_at(lo, r, c0) = make_uint4(l[0], l[1], l[2], l[3]);
}

// n valid rows of q or k (scaled per row by rs[r], if given), zero elsewhere, as hi + lo operands of DK columns.
template <int DK>
__device__ __forceinline__ void stage_features(const LinearAttnArgs& a, const void* src, int ld, int head, int t0, int n,
                                               float scale, const float* rs, uint8_t* hi, uint8_t* lo) {
  for (int u = threadIdx.x; u < 128 * (DK / 8); u += 256) {
    const int r = u / (DK / 8), c0 = (u % (DK / 8)) * 8;
    float f[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) f[i] = 0.f;
    if (r < n && c0 < a.d) {
      const int t = t0 + r;
      const __nv_bfloat16* p = static_cast<const __nv_bfloat16*>(src) + static_cast<size_t>(t) * ld + head * a.d;
      const float* cs = a.rotary ? a.rotary + static_cast<size_t>(a.positions[t]) * a.rd : nullptr;
      la_feature8(p, c0, cs, a.rd, a.act, f);
      const float m = rs ? scale * rs[r] : scale;
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] *= m;
    }
    store_split8(hi, lo, r, c0, f);
  }
}

// n valid rows of v, columns [col0, col0 + DVT), zero elsewhere: one bf16 operand.
template <int DVT>
__device__ __forceinline__ void stage_values(const LinearAttnArgs& a, int head, int col0, int t0, int n, uint8_t* dst) {
  for (int u = threadIdx.x; u < 128 * (DVT / 8); u += 256) {
    const int r = u / (DVT / 8), c0 = (u % (DVT / 8)) * 8;
    uint4 w = make_uint4(0, 0, 0, 0);
    if (r < n && col0 + c0 < a.dv) {
      const __nv_bfloat16* p =
          static_cast<const __nv_bfloat16*>(a.v) + static_cast<size_t>(t0 + r) * a.ldv + head * a.dv + col0 + c0;
      if (a.act) {
        float f[8];
        load_n<8>(p, f);
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] = silu_f(f[i]);
        w = make_uint4(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]), pack_bf16(f[4], f[5]), pack_bf16(f[6], f[7]));
      } else {
        w = *reinterpret_cast<const uint4*>(p);
      }
    }
    *operand_at(dst, r, c0) = w;
  }
}

// Launch 1: L = sum_j decay^(n - 1 - j) k_j v_j^T of one (chunk, head, DVT value columns) -> scratch [entry][h][d][dv].
// A = K^T (features on the MMA rows) and B = V are both read as MN-major operands from token-major tiles.
template <int DVT>
__global__ void __launch_bounds__(256)
linear_chunk_kv_kernel(LinearAttnArgs a, int seq_base, int tiles, float* __restrict__ scratch, unsigned int* err) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int b = blockIdx.z + seq_base, c = blockIdx.x;
  const int head = blockIdx.y / tiles, col0 = (blockIdx.y % tiles) * DVT;
  const int t0 = a.cu_q[b] + c * LC;
  const int n = min(LC, a.cu_q[b + 1] - t0);
  if (n <= 0) return;
  uint8_t* k_hi = smem;
  uint8_t* k_lo = smem + 128 * 128 * 2;
  uint8_t* sv = k_lo + 128 * 128 * 2;
  float* rs = reinterpret_cast<float*>(sv + 128 * DVT * 2);  // [128]
  uint64_t* bar = reinterpret_cast<uint64_t*>(rs + 128);
  uint32_t* holder = reinterpret_cast<uint32_t*>(bar + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(holder + 1);
  const int tid = threadIdx.x, warp = tid >> 5;
  if (tid == 0) {
    mbar_init(bar, 1);
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 0) {
    tmem_alloc(holder, DVT);
    tmem_relinquish();
  }
  if (tid < 128) rs[tid] = decay_pow(a.decay[head], max(n - 1 - tid, 0));
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *holder;
  stage_features<128>(a, a.k, a.ldk, head, t0, n, a.key_scale, rs, k_hi, k_lo);
  stage_values<DVT>(a, head, col0, t0, n, sv);
  fence_async_smem();
  __syncthreads();
  if (tid == 0) {
    constexpr uint32_t idesc = umma_idesc_major(128, DVT, true, true);
#pragma unroll
    for (int p = 0; p < 2; ++p)
#pragma unroll
      for (int k = 0; k < 8; ++k)
        umma_f16(tmem, umma_desc_mn128(smem_u32(p ? k_lo : k_hi) + k * (16 * 128), 128 * 128),
                 umma_desc_mn128(smem_u32(sv) + k * (16 * 128), 128 * 128), idesc, (p || k) ? 1u : 0u);
    umma_commit(bar);
  }
  if (mbar_wait_bounded(bar, 0, abort_flag, err)) {
    tc_fence_after();
    const int row = (warp & 3) * 32 + (tid & 31), half = warp >> 2;
    float* dst = scratch + ((chunk_entry(a, seq_base, b, c) * a.h + head) * a.d + row) * a.dv + col0;
#pragma unroll 1
    for (int cc = half * (DVT / 2); cc < (half + 1) * (DVT / 2); cc += 32) {
      uint32_t r[32];
      __syncwarp();
      tmem_ld32(tmem + (static_cast<uint32_t>((warp & 3) * 32) << 16) + cc, r);
      tmem_wait_ld();
#pragma unroll
      for (int j = 0; j < 32; j += 4)
        if (row < a.d && col0 + cc + j < a.dv)
          *reinterpret_cast<uint4*>(dst + cc + j) = make_uint4(r[j], r[j + 1], r[j + 2], r[j + 3]);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(tmem, DVT);
  }
}

// Launch 2: turns every chunk's own sum into the state entering that chunk and leaves the final state in the slot.
__global__ void __launch_bounds__(256)
linear_chunk_scan_kernel(LinearAttnArgs a, int seq_base, float* __restrict__ scratch) {
  const int b = blockIdx.z + seq_base, head = blockIdx.y;
  const int per = a.d * a.dv;  // a multiple of 4
  const int e = (blockIdx.x * 256 + threadIdx.x) * 4;
  const int slot = a.slots[b], q_len = a.cu_q[b + 1] - a.cu_q[b];
  if (e >= per || q_len <= 0 || slot < 0) return;
  float4* S = reinterpret_cast<float4*>(a.state + (static_cast<size_t>(slot) * a.h + head) * per + e);
  float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
  if (a.kv_lens[b] != q_len) s = *S;
  const int chunks = (q_len + LC - 1) / LC;
  const float whole = decay_pow(a.decay[head], LC);
  const size_t step = static_cast<size_t>(a.h) * per;
  float4* p = reinterpret_cast<float4*>(scratch + (chunk_entry(a, seq_base, b, 0) * a.h + head) * per + e);
  float4 next = *p;
  for (int c = 0; c < chunks; ++c) {
    const float4 v = next;
    float4* here = p;
    p = reinterpret_cast<float4*>(reinterpret_cast<float*>(p) + step);
    if (c + 1 < chunks) next = *p;
    *here = s;
    const float f = c + 1 < chunks ? whole : decay_pow(a.decay[head], q_len - c * LC);
    s.x = f * s.x + v.x; s.y = f * s.y + v.y; s.z = f * s.z + v.z; s.w = f * s.w + v.w;
  }
  *S = s;
}

// Launch 3: outputs of one (chunk, head, DVT value columns). TMEM: scores | own part | state's part.
template <int DK, int DVT>
struct ChunkOutSmem {
  static constexpr int F = 128 * DK * 2;
  static constexpr int OFF_K = 2 * F;
  static constexpr int OFF_V = 4 * F;
  static constexpr int OFF_S = OFF_V + 128 * DVT * 2;         // state rows [DK][DVT], hi and lo
  static constexpr int S_BYTES = DK * DVT * 2;
  static constexpr int OFF_TAB = OFF_S + 2 * S_BYTES;
  static constexpr int USED = OFF_TAB + 256 * 4 + 64;
  static constexpr int TOTAL = USED + 1024 > 232448 ? 232448 : USED + 1024;
  static_assert(USED + 960 <= 232448, "does not fit");
};

template <int DK, int DVT>
__global__ void __launch_bounds__(256)
linear_chunk_out_kernel(LinearAttnArgs a, int seq_base, int tiles, const float* __restrict__ scratch, unsigned int* err) {
  using M_ = ChunkOutSmem<DK, DVT>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int b = blockIdx.z + seq_base, c = blockIdx.x;
  const int head = blockIdx.y / tiles, col0 = (blockIdx.y % tiles) * DVT;
  const int t0 = a.cu_q[b] + c * LC;
  const int q_len = a.cu_q[b + 1] - a.cu_q[b];
  const int n = min(LC, q_len - c * LC);
  if (n <= 0) return;
  const bool has_state = c > 0 || a.kv_lens[b] != q_len;
  uint8_t* q_hi = smem;
  uint8_t* q_lo = smem + M_::F;
  uint8_t* k_hi = smem + M_::OFF_K;
  uint8_t* k_lo = k_hi + M_::F;
  uint8_t* sv = smem + M_::OFF_V;
  uint8_t* s_hi = smem + M_::OFF_S;
  uint8_t* s_lo = s_hi + M_::S_BYTES;
  float* tab = reinterpret_cast<float*>(smem + M_::OFF_TAB);  // tab[127 + e] = decay^e (e >= 0), 0 below
  uint64_t* bar = reinterpret_cast<uint64_t*>(tab + 256);     // [3]
  uint32_t* holder = reinterpret_cast<uint32_t*>(bar + 3);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(holder + 1);
  constexpr uint32_t COLS = 128 + 2 * DVT <= 256 ? 256 : 512;
  const int tid = threadIdx.x, warp = tid >> 5;
  if (tid == 0) {
    for (int i = 0; i < 3; ++i) mbar_init(&bar[i], 1);
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 0) {
    tmem_alloc(holder, COLS);
    tmem_relinquish();
  }
  tab[tid] = tid >= 127 ? decay_pow(a.decay[head], tid - 127) : 0.f;
  stage_features<DK>(a, a.q, a.ldq, head, t0, n, 1.f, nullptr, q_hi, q_lo);
  stage_features<DK>(a, a.k, a.ldk, head, t0, n, a.key_scale, nullptr, k_hi, k_lo);
  fence_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *holder;
  const uint32_t tm_own = tmem + 128, tm_state = tm_own + DVT;
  if (tid == 0) {
    constexpr uint32_t idesc = umma_idesc(128, 128, 1, 1);
#pragma unroll
    for (int p = 0; p < 3; ++p)
#pragma unroll
      for (int k = 0; k < DK / 16; ++k) {
        const uint32_t off = (k >> 2) * (128 * 128) + (k & 3) * 32;
        umma_f16(tmem, umma_desc_k128(smem_u32(p == 1 ? q_lo : q_hi) + off),
                 umma_desc_k128(smem_u32(p == 2 ? k_lo : k_hi) + off), idesc, (p || k) ? 1u : 0u);
      }
    umma_commit(&bar[0]);
  }
  stage_values<DVT>(a, head, col0, t0, n, sv);
  if (has_state) {
    // state rows: panels of 64 columns, DK rows each
    const float* src = scratch + (chunk_entry(a, seq_base, b, c) * a.h + head) * a.d * a.dv + col0;
    for (int u = tid; u < DK * (DVT / 8); u += 256) {
      const int r = u / (DVT / 8), c0 = (u % (DVT / 8)) * 8;
      float f[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] = 0.f;
      if (r < a.d && col0 + c0 < a.dv) load_n<8>(src + static_cast<size_t>(r) * a.dv + c0, f);
      uint32_t h[4], l[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) h[i] = split_bf16(f[2 * i], f[2 * i + 1], &l[i]);
      const int off = (c0 >> 6) * (DK * 128) + r * 128 + ((((c0 >> 3) & 7) ^ (r & 7)) << 4);
      *reinterpret_cast<uint4*>(s_hi + off) = make_uint4(h[0], h[1], h[2], h[3]);
      *reinterpret_cast<uint4*>(s_lo + off) = make_uint4(l[0], l[1], l[2], l[3]);
    }
  }
  fence_async_smem();
  __syncthreads();
  if (has_state && tid == 0) {
    constexpr uint32_t idesc = umma_idesc_major(128, DVT, false, true);
#pragma unroll
    for (int p = 0; p < 3; ++p)
#pragma unroll
      for (int k = 0; k < DK / 16; ++k)
        umma_f16(tm_state, umma_desc_k128(smem_u32(p == 1 ? q_lo : q_hi) + (k >> 2) * (128 * 128) + (k & 3) * 32),
                 umma_desc_mn128(smem_u32(p == 2 ? s_lo : s_hi) + k * (16 * 128), DK * 128), idesc, (p || k) ? 1u : 0u);
    umma_commit(&bar[1]);
  }
  // scores -> decayed, causal weights, written over them as two bf16 matrices. A warp and the one four further on share
  // 32 rows; each takes half of the columns.
  const uint32_t lane_off = static_cast<uint32_t>((warp & 3) * 32) << 16;
  const int row = (warp & 3) * 32 + (tid & 31), half = warp >> 2;
  int bad = !mbar_wait_bounded(&bar[0], 0, abort_flag, err);
  bad = __any_sync(0xffffffffu, bad);
  uint32_t s[64];
  if (!bad) {
    tc_fence_after();
    tmem_ld32(tmem + lane_off + half * 64, s);
    tmem_ld32(tmem + lane_off + half * 64 + 32, s + 32);
    tmem_wait_ld();
  }
  if (__syncthreads_or(bad)) bad = 1;  // both halves of a row have been read
  if (!bad) {
    uint32_t hi[32], lo[32];
#pragma unroll
    for (int j = 0; j < 32; ++j) {
      const int c0 = half * 64 + 2 * j;
      hi[j] = split_bf16(__uint_as_float(s[2 * j]) * tab[row - c0 + 127],
                         __uint_as_float(s[2 * j + 1]) * tab[row - c0 + 126], &lo[j]);
    }
    tmem_st32(tmem + lane_off + half * 32, hi);
    tmem_st32(tmem + lane_off + 64 + half * 32, lo);
    tmem_wait_st();
  }
  tc_fence_before();
  __syncthreads();
  if (!bad && tid == 0) {
    tc_fence_after();
    constexpr uint32_t idesc = umma_idesc_major(128, DVT, false, true);
#pragma unroll
    for (int k = 0; k < 16; ++k)  // hi, then lo
      umma_f16_ts(tm_own, tmem + k * 8, umma_desc_mn128(smem_u32(sv) + (k & 7) * (16 * 128), 128 * 128), idesc,
                  k > 0 ? 1u : 0u);
    umma_commit(&bar[2]);
  }
  if (!bad) {
    bad = !mbar_wait_bounded(&bar[2], 0, abort_flag, err);
    if (!bad && has_state) bad = !mbar_wait_bounded(&bar[1], 0, abort_flag, err);
    bad = __any_sync(0xffffffffu, bad);
  }
  if (!bad) {
    tc_fence_after();
    const float f = tab[128 + row];  // decay^(row + 1)
    __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + (static_cast<size_t>(t0 + row) * a.h + head) * a.dv + col0;
#pragma unroll 1
    for (int cc = half * (DVT / 2); cc < (half + 1) * (DVT / 2); cc += 32) {
      uint32_t x[32], y[32];
      tmem_ld32(tm_own + lane_off + cc, x);
      if (has_state) tmem_ld32(tm_state + lane_off + cc, y);
      tmem_wait_ld();
#pragma unroll
      for (int j = 0; j < 32; j += 8) {
        float v[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) {
          v[u] = __uint_as_float(x[j + u]);
          if (has_state) v[u] = fmaf(f, __uint_as_float(y[j + u]), v[u]);
        }
        if (row < n && col0 + cc + j < a.dv) store_n<8>(out + cc + j, v);
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(tmem, COLS);
  }
}

template <int DVT>
static int launch_chunk_kv(const LinearAttnArgs& a, int seq_base, int num_seqs, int max_q, float* scratch, cudaStream_t st) {
  const int tiles = (a.dv + DVT - 1) / DVT;
  const int smem = 2 * 128 * 128 * 2 + 128 * DVT * 2 + 512 + 64 + 1024;
  auto kern = linear_chunk_kv_kernel<DVT>;
  if (KSANA_SMEM_ONCE(kern, smem) != 0) return -4;
  kern<<<dim3((max_q + LC - 1) / LC, a.h * tiles, num_seqs), 256, smem, st>>>(a, seq_base, tiles, scratch, error_word());
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}
template <int DK, int DVT>
static int launch_chunk_out(const LinearAttnArgs& a, int seq_base, int num_seqs, int max_q, const float* scratch,
                            cudaStream_t st) {
  const int tiles = (a.dv + DVT - 1) / DVT;
  auto kern = linear_chunk_out_kernel<DK, DVT>;
  if (KSANA_SMEM_ONCE(kern, (ChunkOutSmem<DK, DVT>::TOTAL)) != 0) return -4;
  kern<<<dim3((max_q + LC - 1) / LC, a.h * tiles, num_seqs), 256, ChunkOutSmem<DK, DVT>::TOTAL, st>>>(
      a, seq_base, tiles, scratch, error_word());
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

template <typename T, int VEC, bool ONE>
static int launch_recurrent(const LinearAttnArgs& a, int seq_base, int num_seqs, cudaStream_t st) {
  constexpr int TY = 128 / (32 / VEC);
  const int smem = static_cast<int>(sizeof(float)) * (2 * a.d + 32 + TY * 32 + (ONE ? 0 : a.d * 32));
  auto kern = linear_recurrent_kernel<T, VEC, ONE>;
  if (smem > 227 * 1024) return -1;
  if (smem > 48 * 1024 && KSANA_SMEM_ONCE(kern, 227 * 1024) != 0) return -4;
  kern<<<dim3((a.dv + 31) / 32, a.h, num_seqs), 128, smem, st>>>(a, seq_base);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

}  // namespace ksana

using namespace ksana;

// Token-by-token form for sequences [seq_base, seq_base + num_seqs). kind: 0 fp32, 1 bf16 storage of q, k, v and out.
// one_token: every one of these sequences has exactly one new token.
KSANA_API int ksana_linear_recurrent(const void* q, int ldq, const void* k, int ldk, const void* v, int ldv, float* state,
                                     const int* slots, const int* cu_q, const int* kv_lens, const int* positions,
                                     const float* decay, const float* rotary, int rd, int act, float key_scale, int h,
                                     int d, int dv, void* out, int seq_base, int num_seqs, int one_token, int kind,
                                     cudaStream_t st) {
  if (num_seqs <= 0) return 0;
  LinearAttnArgs a{q, k, v, ldq, ldk, ldv, state, slots, cu_q, kv_lens, positions, decay, rotary, rd, act, h, d, dv,
                   key_scale, out};
  const bool vec = (dv & 3) == 0;
#define KSANA_LR(T)                                                                                 \
  (vec ? (one_token ? launch_recurrent<T, 4, true>(a, seq_base, num_seqs, st)                       \
                    : launch_recurrent<T, 4, false>(a, seq_base, num_seqs, st))                     \
       : (one_token ? launch_recurrent<T, 1, true>(a, seq_base, num_seqs, st)                       \
                    : launch_recurrent<T, 1, false>(a, seq_base, num_seqs, st)))
  return kind ? KSANA_LR(__nv_bfloat16) : KSANA_LR(float);
#undef KSANA_LR
}

// fp32 scratch elements that ksana_linear_chunked needs for a step of `tokens` tokens in `num_seqs` sequences.
KSANA_API long long ksana_linear_chunk_scratch(int tokens, int num_seqs, int h, int d, int dv) {
  return (static_cast<long long>(tokens) / LC + num_seqs) * h * d * dv;
}

// bf16, chunked form for sequences [seq_base, seq_base + num_seqs), each with at most max_q new tokens. Returns -1 for
// sizes it does not take (d <= 128, d and dv multiples of 8, a rotation over a multiple of 16 dimensions, 16-byte
// aligned rows).
KSANA_API int ksana_linear_chunked(const void* q, int ldq, const void* k, int ldk, const void* v, int ldv, float* state,
                                   const int* slots, const int* cu_q, const int* kv_lens, const int* positions,
                                   const float* decay, const float* rotary, int rd, int act, float key_scale, int h, int d,
                                   int dv, void* out, int seq_base, int num_seqs, int max_q, float* scratch,
                                   cudaStream_t st) {
  if (num_seqs <= 0 || max_q <= 0) return 0;
  auto rows16 = [](const void* p, int ld) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0 && (ld & 7) == 0; };
  if (d > 128 || (d & 7) || (dv & 7) || (rotary && (rd & 15)) || !rows16(q, ldq) || !rows16(k, ldk) || !rows16(v, ldv) ||
      !rows16(out, 0) || !rows16(state, 0) || !rows16(scratch, 0) || (rotary && !rows16(rotary, 0)))
    return -1;
  LinearAttnArgs a{q, k, v, ldq, ldk, ldv, state, slots, cu_q, kv_lens, positions, decay, rotary, rotary ? rd : 0, act, h,
                   d, dv, key_scale, out};
  const bool narrow = dv <= 64;
  int rc = narrow ? launch_chunk_kv<64>(a, seq_base, num_seqs, max_q, scratch, st)
                  : launch_chunk_kv<128>(a, seq_base, num_seqs, max_q, scratch, st);
  if (rc) return rc;
  linear_chunk_scan_kernel<<<dim3((d * dv + 1023) / 1024, h, num_seqs), 256, 0, st>>>(a, seq_base, scratch);
  if (cudaGetLastError() != cudaSuccess) return -5;
  if (d <= 64)
    return narrow ? launch_chunk_out<64, 64>(a, seq_base, num_seqs, max_q, scratch, st)
                  : launch_chunk_out<64, 128>(a, seq_base, num_seqs, max_q, scratch, st);
  return narrow ? launch_chunk_out<128, 64>(a, seq_base, num_seqs, max_q, scratch, st)
                : launch_chunk_out<128, 128>(a, seq_base, num_seqs, max_q, scratch, st);
}
