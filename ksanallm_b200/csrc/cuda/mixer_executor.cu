// One host call launches every kernel of a range of layers with mixers of their own sizes; the counterpart of
// dense_executor.cu for those layers. A layer is 6 to 14 launches, each of which costs 10 to 20 microseconds when it is
// issued from Python.
#include "mixer_executor.h"

#include "host_common.h"

extern "C" {
int ksana_gemm_bf16(const void* A, const void* W, void* C, const void* bias, int M, int N, int K, int lda, int ldw,
                    int ldc, int out_fp32, int bn, int force_splits, float* ws, long long ws_floats,
                    unsigned int* counters, int num_counters, cudaStream_t stream);
int ksana_gemm_bf16_geglu(const void* A, const void* W_interleaved, void* C, int M, int N, int K, int lda, int ldw,
                          int ldc, cudaStream_t stream);
int ksana_stream_norm(const void* x, int ldx, const void* res_in, void* res_out, int ldr, const void* w, const void* b,
                      void* out, int ldo, int rows, int H, float eps, int kinds, int center, const float* add_rows,
                      const float* add_vec, const void* y, const int* pos, const float* weights, int k,
                      cudaStream_t st);
int ksana_append_act(const void* k, const void* u, int ldx, const int* slots, void* cache, int tokens, int hk, int d,
                     int bs, void* out, int ldo, int I, int gated, int kind, cudaStream_t st);
int ksana_moe_topk(const float* logits, int ld, const float* bias, int T, int E, int k, int groups, int keep, int* ids,
                   float* weights, cudaStream_t st);
int ksana_moe_permute(const void* x, int ldx, const int* ids, int T, int k, int H, int expert_offset, int E_local,
                      int* meta, int* pos, int* row_src, void* xs, cudaStream_t stream);
int ksana_moe_grouped_gemm(const void* A, const void* W, void* C, const int* offsets, int E, int max_rows, int N, int K,
                           cudaStream_t stream);
int ksana_silu_mul(const void* x, int ldx, void* out, int ldo, int rows, int I, cudaStream_t stream);
int ksana_silu_mul_any(const void* x, void* out, int rows, int I, int kind, cudaStream_t st);
int ksana_gelu_mul(const void* x, int ldx, void* out, int ldo, int rows, int I, int kind, cudaStream_t st);
int ksana_qk_norm_cache(void* q, int ldq, const void* k, int ldk, const void* v, int ldv, const int* slots, void* cache,
                        const float* qw, const float* kw, float eps, const int* positions, const float* rotary, int rd,
                        int tokens, int h, int hk, int d, int dv, int bs, int kind, cudaStream_t st);
int ksana_gated_norm(const void* o, const void* g, int ldg, const float* w, void* out, int ldo, int tokens, int h, int dv,
                     float eps, int gate, float out_scale, int kind, cudaStream_t st);
int ksana_window_prefill(const void* q, int ldq, int total_tokens, const void* cache, int num_blocks,
                         const int* block_tables, int max_blocks, const int* cu_q, const int* kv_lens, int h, int hk,
                         int d, int dv, int bs, int window, int keep, int shared, float scale, const float* bias,
                         int bias_len, float out_scale, float softcap, int sink, const void* gate, int ldg, void* out,
                         int ldo, int seq_base, int num_seqs, int max_q, cudaStream_t st);
int ksana_window_decode(const void* q, int ldq, const void* cache, int num_blocks, const int* block_tables, int max_blocks,
                        const int* cu_q, const int* kv_lens, int h, int hk, int d, int dv, int bs, int window,
                        int keep, int shared, float scale, const float* bias, int bias_len, float out_scale,
                        float softcap, int sink, const void* gate, int ldg, void* out, int ldo, int seq_base, int num_seqs,
                        int max_kv, cudaStream_t st);
int ksana_window_attention_any(const void* q, int ldq, const void* cache, const int* block_tables, int max_blocks,
                               const int* cu_q, const int* kv_lens, const int* seq_of_token, int h, int hk, int d, int dv,
                               int bs, int window, int keep, int shared, float scale, const float* bias, int bias_len,
                               float out_scale, float softcap, int sink, const void* gate, int ldg, void* out, int ldo,
                               int tok_base, int tokens, int kind, cudaStream_t st);
long long ksana_linear_chunk_scratch(int tokens, int num_seqs, int h, int d, int dv);
int ksana_linear_chunked(const void* q, int ldq, const void* k, int ldk, const void* v, int ldv, float* state,
                         const int* slots, const int* cu_q, const int* kv_lens, const int* positions, const float* decay,
                         const float* rotary, int rd, int act, float key_scale, int h, int d, int dv, void* out,
                         int seq_base, int num_seqs, int max_q, float* scratch, cudaStream_t st);
int ksana_linear_recurrent(const void* q, int ldq, const void* k, int ldk, const void* v, int ldv, float* state,
                           const int* slots, const int* cu_q, const int* kv_lens, const int* positions,
                           const float* decay, const float* rotary, int rd, int act, float key_scale, int h, int d, int dv,
                           void* out, int seq_base, int num_seqs, int one_token, int kind, cudaStream_t st);
}

namespace {

struct Exec {
  const KsanaMixerModel* m;
  const KsanaMixerStep* s;
  float* residual;
  int* launches;
  int* fail_code;
  cudaStream_t st;
  const void* h = nullptr;
  int pp = 0, failed = 0;

  bool step(int id, int rc) {
    ++*launches;
    if (rc == 0) return true;
    failed = id;
    *fail_code = rc;
    return false;
  }
  int gemm(const void* a, int K, const void* w, const void* bias, void* c, int N, int ldc, int fp32_out = 0) {
    return ksana_gemm_bf16(a, w, c, bias, s->total_tokens, N, K, K, K, ldc, fp32_out, 0, 0, m->gemm_ws, m->gemm_ws_floats,
                           m->gemm_counters, m->n_counters, st);
  }
  // the stream takes the sublayer's output (and that of routed experts, and what comes between two layers); the
  // normalised sum is the next input
  bool norm(int id, const void* y, const void* w, bool routed = false, const KsanaMixerLayer* last = nullptr) {
    const int H = m->hidden;
    void* out = m->h_buf[pp];
    const float* rows = last && last->next_start ? s->start : nullptr;
    const float* vec = last ? last->next_vec : nullptr;
    const void* e = routed ? m->rows_out_buf : nullptr;
    if (!step(id, ksana_stream_norm(y, H, residual, residual, H, w, nullptr, out, H, s->total_tokens, H, m->eps, 13,
                                    m->center, rows, vec, e, m->pair_pos, m->expert_weights, routed ? last->top : 0, st)))
      return false;
    h = out;
    pp ^= 1;
    return true;
  }

  bool attention(const KsanaMixerLayer& w, char* x, void* out) {
    const int T = s->total_tokens, ld = w.n_in, nq = w.h * w.d, nk = w.hk * w.d;
    char *k = x + static_cast<size_t>(nq) * 2, *v = k + static_cast<size_t>(nk) * 2;
    if (w.shared_kv) {  // the keys go to the cache in the launch that runs a parallel dense FFN's activation
      const int I = w.parallel ? w.inter : 0;
      if (!step(2, ksana_append_act(k, v, ld, s->slot_mapping, w.kv, T, w.hk, w.d, m->block_size,
                                    static_cast<char*>(out) + static_cast<size_t>(w.h * w.dv) * 2, w.k_out, I, w.gated, 1,
                                    st)))
        return false;
    } else if (!step(2, ksana_qk_norm_cache(x, ld, k, ld, v, ld, s->slot_mapping, w.kv, w.q_norm, w.k_norm, m->eps,
                                            nullptr, nullptr, 0, T, w.h, w.hk, w.d, w.dv, m->block_size, 1, st))) {
      return false;
    }
    auto general = [&](int first, int count) {
      return ksana_window_attention_any(x, ld, w.kv, s->block_tables, s->max_blocks, s->cu_q, s->kv_lens, s->seq_of_token,
                                        w.h, w.hk, w.d, w.dv, m->block_size, w.window, w.keep_first, w.shared_kv,
                                        w.scale, w.bias, w.bias_len, w.attn_out_scale, 0.f, 0, nullptr, 0, out, w.k_out, first,
                                        count, 1, st);
    };
    if (s->num_prefill > 0) {
      int rc = ksana_window_prefill(x, ld, T, w.kv, m->num_blocks, s->block_tables, s->max_blocks, s->cu_q, s->kv_lens,
                                    w.h, w.hk, w.d, w.dv, m->block_size, w.window, w.keep_first, w.shared_kv, w.scale,
                                    w.bias, w.bias_len, w.attn_out_scale, 0.f, 0, nullptr, 0, out, w.k_out, 0, s->num_prefill,
                                    s->max_q_prefill, st);
      if (rc == -1) rc = general(0, s->prefill_tokens);
      if (!step(3, rc)) return false;
    }
    if (s->num_decode > 0) {
      int rc = -1;
      if (s->one_token)
        rc = ksana_window_decode(x, ld, w.kv, m->num_blocks, s->block_tables, s->max_blocks, s->cu_q, s->kv_lens, w.h, w.hk, w.d, w.dv,
                                 m->block_size, w.window, w.keep_first, w.shared_kv, w.scale, w.bias, w.bias_len,
                                 w.attn_out_scale, 0.f, 0, nullptr, 0, out, w.k_out, s->num_prefill, s->num_decode,
                                 s->max_kv_decode, st);
      if (rc == -1) rc = general(s->prefill_tokens, T - s->prefill_tokens);
      if (!step(4, rc)) return false;
    }
    return true;
  }

  bool linear(const KsanaMixerLayer& w, char* x, void* out) {
    const int ld = w.n_in, nq = w.lh * w.ld, nv = w.lh * w.ldv;
    char *k = x + static_cast<size_t>(nq) * 2, *v = k + static_cast<size_t>(nq) * 2, *g = v + static_cast<size_t>(nv) * 2;
    int n_long = s->num_long;
    if (n_long > 0) {
      int rc = -1;
      if (ksana_linear_chunk_scratch(s->long_tokens, n_long, w.lh, w.ld, w.ldv) <= m->chunk_floats)
        rc = ksana_linear_chunked(x, ld, k, ld, v, ld, w.state, s->state_slots, s->cu_q, s->kv_lens, s->positions, w.decay,
                                  w.rotary, w.rd, w.act, w.key_scale, w.lh, w.ld, w.ldv, m->o_buf, 0, n_long,
                                  s->max_q_prefill, m->chunk_buf, st);
      if (rc == -1) {
        n_long = 0;  // not a size of the chunked form
      } else {
        *launches += 2;
        if (!step(5, rc)) return false;
      }
    }
    const int base[2] = {n_long, s->num_prefill}, count[2] = {s->num_prefill - n_long, s->num_decode};
    for (int i = 0; i < 2; ++i)
      if (count[i] > 0 &&
          !step(6, ksana_linear_recurrent(x, ld, k, ld, v, ld, w.state, s->state_slots, s->cu_q, s->kv_lens, s->positions,
                                          w.decay, w.rotary, w.rd, w.act, w.key_scale, w.lh, w.ld, w.ldv, m->o_buf,
                                          base[i], count[i], i == 1 && s->one_token, 1, st)))
        return false;
    return step(7, ksana_gated_norm(m->o_buf, g, ld, w.norm_w, out, w.k_out, s->total_tokens, w.lh, w.ldv, m->eps, w.gate,
                                    w.lin_out_scale, 1, st));
  }

  // experts of the tokens in `h`; their rows stay in sorted order for the norm that adds them up
  bool experts(const KsanaMixerLayer& w) {
    const int T = s->total_tokens, H = m->hidden, I = w.expert_inter, n = T * w.top;
    const int* offsets = m->sort_meta + w.experts;
    if (!step(15, gemm(h, H, w.w_router, nullptr, m->router_buf, w.router_rows, w.router_rows, 1))) return false;
    if (!step(16, ksana_moe_topk(m->router_buf, w.router_rows, w.b_router, T, w.experts, w.top, 1, 1, m->expert_ids,
                                 m->expert_weights, st)))
      return false;
    ++*launches;
    if (!step(17, ksana_moe_permute(h, H, m->expert_ids, T, w.top, H, 0, w.experts, m->sort_meta, m->pair_pos,
                                    m->pair_src, m->rows_buf, st)))
      return false;
    if (!step(18, ksana_moe_grouped_gemm(m->rows_buf, w.w_expert_gu, m->rows_gu_buf, offsets, w.experts, n, 2 * I, H, st)))
      return false;
    int rc = ksana_silu_mul(m->rows_gu_buf, 2 * I, m->rows_act_buf, I, n, I, st);
    if (rc == -1) rc = ksana_silu_mul_any(m->rows_gu_buf, m->rows_act_buf, n, I, 1, st);
    if (!step(19, rc)) return false;
    return step(20, ksana_moe_grouped_gemm(m->rows_act_buf, w.w_expert_down, m->rows_out_buf, offsets, w.experts, n, H, I,
                                           st));
  }

  bool layer(const KsanaMixerLayer& w) {
    const int T = s->total_tokens, H = m->hidden;
    char* x = static_cast<char*>(m->in_buf);
    char* mix = static_cast<char*>(m->mix_buf);
    if (!step(1, gemm(h, H, w.w_in, w.b_in, x, w.n_in, w.n_in))) return false;
    const int used = w.h * w.dv + w.lh * w.ldv + (w.parallel ? w.inter : 0);
    if (used < w.k_out &&
        cudaMemset2DAsync(mix + static_cast<size_t>(used) * 2, static_cast<size_t>(w.k_out) * 2, 0,
                          static_cast<size_t>(w.k_out - used) * 2, T, st) != cudaSuccess)
      return step(8, -5);
    if (w.h > 0 && !attention(w, x, mix)) return false;
    const size_t attn_in = w.h > 0 ? static_cast<size_t>(w.h * w.d + w.hk * (w.d + (w.shared_kv ? 0 : w.dv))) * 2 : 0;
    if (w.lh > 0 && !linear(w, x + attn_in, mix + static_cast<size_t>(w.h * w.dv) * 2)) return false;
    if (!step(9, gemm(mix, w.k_out, w.w_out, nullptr, m->proj_buf, H, H))) return false;
    if (w.experts > 0 && !experts(w)) return false;
    if (w.ln2 != nullptr) {
      if (!norm(10, m->proj_buf, w.ln2)) return false;
      const int I = w.inter;
      if (w.w_gu_il != nullptr && T >= 384) {
        if (!step(11, ksana_gemm_bf16_geglu(h, w.w_gu_il, m->act_buf, T, 2 * I, H, H, H, I, st))) return false;
      } else {
        if (!step(11, gemm(h, H, w.w_gu, nullptr, m->gu_buf, 2 * I, 2 * I))) return false;
        if (!step(12, ksana_gelu_mul(m->gu_buf, 2 * I, m->act_buf, I, T, I, 1, st))) return false;
      }
      if (!step(13, gemm(m->act_buf, w.inter, w.w_down, nullptr, m->proj_buf, H, H))) return false;
    }
    return norm(14, m->proj_buf, w.next_ln, w.experts > 0, &w);
  }
};

}  // namespace

KSANA_API int ksana_mixer_forward(const KsanaMixerModel* m, const KsanaMixerStep* s, const void* h, float* residual,
                                  int first, int last, void** out_h, int* fail_code, int* launches, cudaStream_t stream) {
  *fail_code = 0;
  *launches = 0;
  Exec ex{m, s, residual, launches, fail_code, stream};
  ex.h = h;
  for (int i = first; i < last && s->total_tokens > 0; ++i)
    if (!ex.layer(m->layers[i])) return (i + 1) * 100 + ex.failed;
  *out_h = const_cast<void*>(ex.h);
  return 0;
}
