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
  if (!act) return x;
  return sizeof(T) == 2 ? silu_fast(x) : silu_f(x);
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
  // the single token's share of the state is requested before anything else (up to RMAX rows per thread)
  constexpr int RMAX = ONE ? 8 : 1;
  float pre[RMAX][VEC];
  if (ONE && live) {
#pragma unroll
    for (int i = 0; i < RMAX; ++i) {
#pragma unroll
      for (int j = 0; j < VEC; ++j) pre[i][j] = 0.f;
      const int r = ty + i * TY;
      if (r < a.d && !fresh) load_n<VEC>(S + static_cast<size_t>(r) * a.dv, pre[i]);
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
      if (ONE) {
#pragma unroll
        for (int i = 0; i < RMAX; ++i) {
          const int r = ty + i * TY;
          if (r < a.d) {
            const float kr = sk[r], qr = sq[r];
#pragma unroll
            for (int j = 0; j < VEC; ++j) {
              pre[i][j] = dec * pre[i][j] + kr * vv[j];
              acc[j] += qr * pre[i][j];
            }
            store_n<VEC>(S + static_cast<size_t>(r) * a.dv, pre[i]);
          }
        }
      }
#pragma unroll 4
      for (int r = ty + (ONE ? RMAX * TY : 0); r < a.d; r += TY) {
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

// Features of a head are handled in slots of 16: slot u < rd / 16 holds the 8 dimensions from 8 u and their rotation
// partners half a rotation further, the others 16 consecutive ones. First dimension of each half of the slot:
__device__ __forceinline__ void slot_dims(int u, int rd, int* lo, int* hi) {
  const bool rot = u * 16 < rd;
  *lo = rot ? u * 8 : u * 16;
  *hi = rot ? *lo + (rd >> 1) : *lo + 8;
}

// cos and sin of a slot's 8 pairs.
struct SlotAngles {
  float4 c[2], s[2];
};
__device__ __forceinline__ void load_angles(const LinearAttnArgs& a, int pos, int lo, SlotAngles* x) {
  const float4* p = reinterpret_cast<const float4*>(a.rotary + static_cast<size_t>(pos) * a.rd + lo);
  const float4* q = p + (a.rd >> 3);
  x->c[0] = p[0]; x->c[1] = p[1];
  x->s[0] = q[0]; x->s[1] = q[1];
}

// Activation, rotation and scale of one slot, then its hi and lo parts go to row r of the operands.
__device__ __forceinline__ void finish_slot(uint4 w_lo, uint4 w_hi, bool rot, const SlotAngles& an, int act, float scale,
                                            uint8_t* hi, uint8_t* lo, int r, int c_lo, int c_hi) {
  float x[8], y[8];
  unpack8(w_lo, x);
  unpack8(w_hi, y);
  if (act) {
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      x[i] = silu_fast(x[i]);
      y[i] = silu_fast(y[i]);
    }
  }
  if (rot) {
    const float* c = reinterpret_cast<const float*>(an.c);
    const float* s = reinterpret_cast<const float*>(an.s);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const float u = x[i] * c[i] - y[i] * s[i];
      y[i] = y[i] * c[i] + x[i] * s[i];
      x[i] = u;
    }
  }
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    x[i] *= scale;
    y[i] *= scale;
  }
  store_split8(hi, lo, r, c_lo, x);
  store_split8(hi, lo, r, c_hi, y);
}

__device__ __forceinline__ uint4 value_word(uint4 w, int act) {
  if (!act) return w;
  float f[8];
  unpack8(w, f);
#pragma unroll
  for (int i = 0; i < 8; ++i) f[i] = silu_fast(f[i]);
  return make_uint4(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]), pack_bf16(f[4], f[5]), pack_bf16(f[6], f[7]));
}

__device__ __forceinline__ const __nv_bfloat16* head_row(const void* base, int t, int ld, int off) {
  return static_cast<const __nv_bfloat16*>(base) + static_cast<size_t>(t) * ld + off;
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
  const int pos0 = a.kv_lens[b] - (a.cu_q[b + 1] - t0);
  const uint4 zero = make_uint4(0, 0, 0, 0);
  constexpr int UV = 128 * (DVT / 8) / 256;
  uint4 vw[UV];
#pragma unroll
  for (int i = 0; i < UV; ++i) {
    const int u = i * 256 + tid, r = u / (DVT / 8), c0 = (u % (DVT / 8)) * 8;
    vw[i] = r < n && col0 + c0 < a.dv
                ? *reinterpret_cast<const uint4*>(head_row(a.v, t0 + r, a.ldv, head * a.dv + col0 + c0)) : zero;
  }
#pragma unroll
  for (int g = 0; g < 2; ++g) {
    uint4 wl[2], wh[2];
    SlotAngles an[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int u = (g * 2 + i) * 256 + tid, r = u / 8, sl = u % 8;
      int cl, ch;
      slot_dims(sl, a.rd, &cl, &ch);
      const __nv_bfloat16* p = head_row(a.k, t0 + r, a.ldk, head * a.d);
      wl[i] = r < n && cl < a.d ? *reinterpret_cast<const uint4*>(p + cl) : zero;
      wh[i] = r < n && ch < a.d ? *reinterpret_cast<const uint4*>(p + ch) : zero;
      if (r < n && sl * 16 < a.rd) load_angles(a, pos0 + r, cl, &an[i]);
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int u = (g * 2 + i) * 256 + tid, r = u / 8, sl = u % 8;
      int cl, ch;
      slot_dims(sl, a.rd, &cl, &ch);
      finish_slot(wl[i], wh[i], r < n && sl * 16 < a.rd, an[i], a.act, a.key_scale * rs[r], k_hi, k_lo, r, cl, ch);
    }
  }
#pragma unroll
  for (int i = 0; i < UV; ++i) {
    const int u = i * 256 + tid, r = u / (DVT / 8), c0 = (u % (DVT / 8)) * 8;
    *operand_at(sv, r, c0) = value_word(vw[i], a.act);
  }
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
  const float whole = decay_pow(a.decay[head], LC), last = decay_pow(a.decay[head], q_len - (chunks - 1) * LC);
  const size_t step = static_cast<size_t>(a.h) * per;
  float* p = scratch + (chunk_entry(a, seq_base, b, 0) * a.h + head) * per + e;
  auto at = [&](int c) { return reinterpret_cast<float4*>(p + c * step); };
  // the chain over the chunks is short arithmetic: what it costs is the loads, so AHEAD of them are kept in flight
  constexpr int AHEAD = 8;
  float4 ring[AHEAD];
#pragma unroll
  for (int i = 0; i < AHEAD; ++i)
    if (i < chunks) ring[i] = *at(i);
  for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      const int c = c0 + i;
      if (c < chunks) {
        const float4 v = ring[i];
        if (c + AHEAD < chunks) ring[i] = *at(c + AHEAD);
        *at(c) = s;
        const float f = c + 1 < chunks ? whole : last;
        s.x = f * s.x + v.x; s.y = f * s.y + v.y; s.z = f * s.z + v.z; s.w = f * s.w + v.w;
      }
    }
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

template <int DK, int DVT, int NT>
__global__ void __launch_bounds__(NT)
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
  const uint4 zero = make_uint4(0, 0, 0, 0);

  // ---- q, k and v: everything is requested before anything is used ----
  constexpr int UQ = 128 * (DK / 16) / NT, UV = 128 * (DVT / 8) / NT, US = DK * (DVT / 8) / NT;
  const int pos0 = a.kv_lens[b] - q_len + c * LC;
  uint4 ql[UQ], qh[UQ], kl[UQ], kh[UQ], vw[UV];
  SlotAngles an[UQ];
#pragma unroll
  for (int i = 0; i < UQ; ++i) {
    const int u = i * NT + tid, r = u / (DK / 16), sl = u % (DK / 16);
    int cl, ch;
    slot_dims(sl, a.rd, &cl, &ch);
    const __nv_bfloat16* q = head_row(a.q, t0 + r, a.ldq, head * a.d);
    const __nv_bfloat16* k = head_row(a.k, t0 + r, a.ldk, head * a.d);
    const bool in_lo = r < n && cl < a.d, in_hi = r < n && ch < a.d;
    ql[i] = in_lo ? *reinterpret_cast<const uint4*>(q + cl) : zero;
    qh[i] = in_hi ? *reinterpret_cast<const uint4*>(q + ch) : zero;
    kl[i] = in_lo ? *reinterpret_cast<const uint4*>(k + cl) : zero;
    kh[i] = in_hi ? *reinterpret_cast<const uint4*>(k + ch) : zero;
    if (r < n && sl * 16 < a.rd) load_angles(a, pos0 + r, cl, &an[i]);
  }
#pragma unroll
  for (int i = 0; i < UV; ++i) {
    const int u = i * NT + tid, r = u / (DVT / 8), c0 = (u % (DVT / 8)) * 8;
    vw[i] = r < n && col0 + c0 < a.dv
                ? *reinterpret_cast<const uint4*>(head_row(a.v, t0 + r, a.ldv, head * a.dv + col0 + c0)) : zero;
  }
  if (tid == 0) {
    for (int i = 0; i < 3; ++i) mbar_init(&bar[i], 1);
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 0) {
    tmem_alloc(holder, COLS);
    tmem_relinquish();
  }
  if (tid < 256) tab[tid] = tid >= 127 ? decay_pow(a.decay[head], tid - 127) : 0.f;
#pragma unroll
  for (int i = 0; i < UQ; ++i) {
    const int u = i * NT + tid, r = u / (DK / 16), sl = u % (DK / 16);
    int cl, ch;
    slot_dims(sl, a.rd, &cl, &ch);
    const bool rot = r < n && sl * 16 < a.rd;
    finish_slot(ql[i], qh[i], rot, an[i], a.act, 1.f, q_hi, q_lo, r, cl, ch);
    finish_slot(kl[i], kh[i], rot, an[i], a.act, a.key_scale, k_hi, k_lo, r, cl, ch);
  }
  // the state entering the chunk (fp32) is on its way while the scores are multiplied
  float4 sw[US][2];
  if (has_state) {
    const float* src = scratch + (chunk_entry(a, seq_base, b, c) * a.h + head) * a.d * a.dv + col0;
#pragma unroll
    for (int i = 0; i < US; ++i) {
      const int u = i * NT + tid, r = u / (DVT / 8), c0 = (u % (DVT / 8)) * 8;
      sw[i][0] = sw[i][1] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (r < a.d && col0 + c0 < a.dv) {
        const float4* p = reinterpret_cast<const float4*>(src + static_cast<size_t>(r) * a.dv + c0);
        sw[i][0] = p[0];
        sw[i][1] = p[1];
      }
    }
  }
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
#pragma unroll
  for (int i = 0; i < UV; ++i) {
    const int u = i * NT + tid, r = u / (DVT / 8), c0 = (u % (DVT / 8)) * 8;
    *operand_at(sv, r, c0) = value_word(vw[i], a.act);
  }
  if (has_state) {
    // state rows: panels of 64 columns, DK rows each
#pragma unroll
    for (int i = 0; i < US; ++i) {
      const int u = i * NT + tid, r = u / (DVT / 8), c0 = (u % (DVT / 8)) * 8;
      const float* f = reinterpret_cast<const float*>(sw[i]);
      uint32_t h[4], l[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) h[j] = split_bf16(f[2 * j], f[2 * j + 1], &l[j]);
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
  // scores -> decayed, causal weights, written over them as two bf16 matrices. The warps whose numbers agree modulo 4
  // share 32 rows; each takes its part of the columns.
  constexpr int PARTS = NT / 128, PC = 128 / PARTS;
  const uint32_t lane_off = static_cast<uint32_t>((warp & 3) * 32) << 16;
  const int row = (warp & 3) * 32 + (tid & 31), part = warp >> 2;
  int bad = !mbar_wait_bounded(&bar[0], 0, abort_flag, err);
  bad = __any_sync(0xffffffffu, bad);
  uint32_t s[PC];
  if (!bad) {
    tc_fence_after();
#pragma unroll
    for (int q = 0; q < PC / 32; ++q) tmem_ld32(tmem + lane_off + part * PC + q * 32, s + q * 32);
    tmem_wait_ld();
  }
  if (__syncthreads_or(bad)) bad = 1;  // every part of a row has been read
  if (!bad) {
    uint32_t hi[PC / 2], lo[PC / 2];
#pragma unroll
    for (int j = 0; j < PC / 2; ++j) {
      const int c0 = part * PC + 2 * j;
      hi[j] = split_bf16(__uint_as_float(s[2 * j]) * tab[row - c0 + 127],
                         __uint_as_float(s[2 * j + 1]) * tab[row - c0 + 126], &lo[j]);
    }
    if constexpr (PC == 64) {
      tmem_st32(tmem + lane_off + part * 32, hi);
      tmem_st32(tmem + lane_off + 64 + part * 32, lo);
    } else {
      tmem_st16(tmem + lane_off + part * 16, hi);
      tmem_st16(tmem + lane_off + 64 + part * 16, lo);
    }
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
    constexpr int OC = DVT / PARTS;  // 16, 32 or 64 output columns per thread
    __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + (static_cast<size_t>(t0 + row) * a.h + head) * a.dv + col0;
#pragma unroll 1
    for (int cc = part * OC; cc < (part + 1) * OC; cc += 16) {
      uint32_t x[16], y[16];
      tmem_ld16(tm_own + lane_off + cc, x);
      if (has_state) tmem_ld16(tm_state + lane_off + cc, y);
      tmem_wait_ld();
#pragma unroll
      for (int j = 0; j < 16; j += 8) {
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
  constexpr int NT = DK == 64 && DVT == 64 ? 256 : 512;  // two CTAs per SM fit the smallest size only
  auto kern = linear_chunk_out_kernel<DK, DVT, NT>;
  if (KSANA_SMEM_ONCE(kern, (ChunkOutSmem<DK, DVT>::TOTAL)) != 0) return -4;
  kern<<<dim3((max_q + LC - 1) / LC, a.h * tiles, num_seqs), NT, ChunkOutSmem<DK, DVT>::TOTAL, st>>>(
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
