// What the kernels of weight-mixing attention share: see talking_attention.cu.
#pragma once
#include "host_common.h"
#include "mixer_common.cuh"

namespace ksana {

constexpr int TALK_PAGE = 16;  // tokens per page that the tensor-core kernels take

struct TalkArgs {
  const void* q;
  int ldq;
  const void* cache;
  const int* block_tables;
  int max_blocks;
  const int* cu_q;
  const int* kv_lens;
  const int* seq_of_token;
  int h, hk, d, dv, bs;
  float scale;
  const float* sink;   // [h]
  const float* talk;   // [h][h]: to, from
  float out_scale;
  const void* gate;    // [T][ldg >= h * dv] in the storage type of q, or null
  int ldg;
  void* out;
  int ldo;
  __host__ __device__ size_t v_off() const { return static_cast<size_t>(hk) * bs * d; }
  __host__ __device__ size_t block_elems() const { return static_cast<size_t>(hk) * bs * (d + dv); }
};

// Pages of 16 keys (which 0) or values (1) of one head, 64 columns at a time; columns past the head's end read as zeros.
inline int talk_cache_map(const TalkArgs& a, int num_blocks, int which, CUtensorMap* m) {
  const uint32_t box[3] = {64, TALK_PAGE, 1};
  const uint64_t cols = which ? a.dv : a.d;
  const uint64_t dims[3] = {cols, static_cast<uint64_t>(a.hk) * a.bs, static_cast<uint64_t>(num_blocks)};
  const uint64_t str[2] = {cols * 2, a.block_elems() * 2};
  const void* base = static_cast<const char*>(a.cache) + (which ? a.v_off() * 2 : 0);
  return make_tmap_nd(m, base, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, dims, str, box, CU_TENSOR_MAP_SWIZZLE_128B) ? -3 : 0;
}

inline bool talk_rows16(const void* p, int ld) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0 && (ld & 7) == 0; }

// bf16 sizes that the tensor-core kernels take.
inline bool talk_tc_sizes(const TalkArgs& a) {
  return a.h % a.hk == 0 && a.h <= 64 && a.bs == TALK_PAGE && a.d <= 128 && a.dv <= 128 && !(a.d & 7) && !(a.dv & 7) &&
         talk_rows16(a.q, a.ldq) && talk_rows16(a.cache, 0) && talk_rows16(a.out, a.ldo) && talk_rows16(a.gate, a.ldg);
}

// eight gated results of one head
__device__ __forceinline__ void talk_store8(const TalkArgs& a, size_t tok, int col, float* f) {
  if (a.gate) {
    float g[8];
    load_n<8>(static_cast<const __nv_bfloat16*>(a.gate) + tok * a.ldg + col, g);
#pragma unroll
    for (int u = 0; u < 8; ++u) f[u] *= __fdividef(a.out_scale, 1.f + __expf(-g[u]));
  } else {
#pragma unroll
    for (int u = 0; u < 8; ++u) f[u] *= a.out_scale;
  }
  store_n<8>(static_cast<__nv_bfloat16*>(a.out) + tok * a.ldo + col, f);
}

}  // namespace ksana
