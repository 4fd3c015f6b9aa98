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
int ksana_moe_topk(const float* logits, int ld, const float* bias, int T, int E, int k, int groups, int keep, int scoring,
                   float scale, int* ids, float* weights, cudaStream_t st);
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
                     float eps, int gate, float out_scale, int per_head, int kind, cudaStream_t st);
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
int ksana_hyper_norm(const void* x, int ldx, const float* scale, const void* rows, const int* pos, const float* weights,
                     int k, const float* streams, int one, const float* mix, const float* out_w, float* res,
                     const float* in_w, const void* w, void* out, int tokens, int H, int S, float eps, int kind,
                     cudaStream_t st);
int ksana_relu2(const void* x, int ldx, void* out, int rows, int cols, int kind, cudaStream_t st);
int ksana_clamped_gate_mul(const void* x, void* out, int rows, int I, float limit, float alpha, int kind,
                           cudaStream_t st);
int ksana_gemm_bf16_batched(const void* A, long long a_row_stride, long long a_batch_stride, const void* W, void* C,
                            long long c_row_stride, long long c_batch_stride, int T, int B, int N, int K,
                            cudaStream_t stream);
int ksana_head_gemm_any(const void* A, long long a_row, long long a_head, const void* W, void* C, long long c_row,
                        long long c_head, int rows, int heads, int N, int K, int kind, cudaStream_t st);
int ksana_latent_append(void* q, int ldq, int dim, void* q_cat, int cat_from, const void* x, int ldx, const float* norm_w,
                        float eps, const int* positions, const float* rotary, const int* slots, void* cache, int tokens,
                        int h, int rank, int rot, int kind, cudaStream_t st);
int ksana_latent_gather(const void* cache, const int* block_tables, int max_blocks, const int* kv_lens, int seq_base,
                        int num_seqs, int max_kv, int bs, int width, void* out, cudaStream_t st);
int ksana_latent_decode(const void* q, int ldq, int total_tokens, const void* cache, int num_blocks,
                        const int* block_tables, int max_blocks, const int* cu_q, const int* kv_lens, int h, int rank,
                        int rot, int bs, float scale, const void* gate, int ldg, void* out, int ldo, int seq_base,
                        int num_seqs, int max_q, int max_kv, cudaStream_t st);
int ksana_latent_prefill(const void* q, int ldq, int total_tokens, const void* kv, int ldkv, const void* rot, int ldr,
                         int rows, const int* cu_q, const int* kv_lens, int h, int d, int rd, int dv, float scale,
                         const void* gate, int ldg, void* out, int ldo, int seq_base, int num_seqs, int max_q,
                         cudaStream_t st);
long long ksana_recurrence_scratch(int tokens, int num_seqs, int max_q, int C);
int ksana_recurrence_prompts(const void* y, int ldy, const void* x, int ldx, float* state, const int* slots,
                             const int* cu_q, const int* kv_lens, const int* seq_of_token, const float* conv_w,
                             const float* conv_b, const void* gates, const float* gates_b, const float* rate, int C, int K,
                             int B, void* out, int ldo, int seq_base, int num_seqs, int tok_base, int tokens, int max_q,
                             float* scratch, cudaStream_t st);
int ksana_recurrence_step(const void* y, int ldy, const void* x, int ldx, float* state, const int* slots, const int* cu_q,
                          const int* kv_lens, const float* conv_w, const float* conv_b, const void* gates,
                          const float* gates_b, const float* rate, int C, int K, int B, void* out, int ldo, int seq_base,
                          int num_seqs, cudaStream_t st);
int ksana_recurrence_conv(const void* x, int ldx, const float* state, const int* slots, const int* cu_q,
                          const int* kv_lens, const int* seq_of_token, const float* conv_w, const float* conv_b, int C,
                          int K, void* u, int tok_base, int tokens, int kind, cudaStream_t st);
int ksana_recurrence_scan(const void* y, int ldy, const void* x, int ldx, float* state, const int* slots, const int* cu_q,
                          const int* kv_lens, const void* u, const float* z, const float* gates_b, const float* rate,
                          int C, int K, int B, void* out, int ldo, int seq_base, int num_seqs, int tok_base, int kind,
                          cudaStream_t st);
int ksana_gated_stream_norm(const void* x, int ldx, const void* xg, int ldxg, const void* rows, const int* pos,
                            const float* weights, int k, const void* y, int ldy, const float* ys, int ldys, const void* yg,
                            int ldyg, float scale, const float* in, float* stream, const void* w0, const void* w1, void* out,
                            int tokens, int H, float eps, int kind, cudaStream_t st);
int ksana_qk_row_norm_cache(void* q, int ldq, const void* k, int ldk, const void* v, int ldv, const int* slots, void* cache,
                            const float* qw, const float* kw, float eps, const int* positions, const float* rotary, int rd,
                            int tokens, int h, int hk, int d, int dv, int bs, int kind, cudaStream_t st);
int ksana_talking_any(const void* q, int ldq, const void* cache, const int* block_tables, int max_blocks, const int* cu_q,
                      const int* kv_lens, const int* seq_of_token, int h, int hk, int d, int dv, int bs, float scale,
                      const float* sink, const float* talk, float out_scale, const void* gate, int ldg, void* out, int ldo,
                      int tok_base, int tokens, int kind, cudaStream_t st);
long long ksana_talking_prefill_bytes(int h, int num_seqs, const int* cu_q_host, const int* kv_lens_host);
int ksana_talking_prefill(const void* q, int ldq, int total_tokens, const void* cache, int num_blocks,
                          const int* block_tables, int max_blocks, const int* cu_q, const int* kv_lens, int h, int hk, int d,
                          int dv, int bs, float scale, const float* sink, const float* talk, float out_scale,
                          const void* gate, int ldg, void* out, int ldo, int num_seqs, const int* cu_q_host,
                          const int* kv_lens_host, void* scratch, long long scratch_bytes, int* launches, cudaStream_t st);
long long ksana_talking_decode_bytes(int h, int num_seqs, int max_kv);
int ksana_talking_decode(const void* q, int ldq, const void* cache, int num_blocks, const int* block_tables, int max_blocks,
                         const int* cu_q, const int* kv_lens, int h, int hk, int d, int dv, int bs, float scale,
                         const float* sink, const float* talk, float out_scale, const void* gate, int ldg, void* out,
                         int ldo, int seq_base, int num_seqs, int max_kv, void* scratch, long long scratch_bytes,
                         cudaStream_t st);
int ksana_token_mix(const void* h, const float* mu, float* last, long long slot_pitch, long long slots_total,
                    const int* slots, const int* cu_q, const int* kv_lens, const int* seq_of_token, void* out, int tokens,
                    int W, int rows, int kind, cudaStream_t st);
int ksana_tanh_parts(const float* x, int n, void* out, int rows, int kind, cudaStream_t st);
int ksana_time_mix_recurrent(const void* r, int ldr, const void* k, int ldk, const void* v, int ldv, const float* z, int ldz,
                             const float* w0, const float* u, float* state, long long slot_pitch, const int* slots,
                             const int* cu_q, const int* kv_lens, int h, int d, void* out, int seq_base, int num_seqs,
                             int one_token, int kind, cudaStream_t st);
long long ksana_time_mix_scratch(int tokens, int num_seqs, int h, int d);
int ksana_time_mix_chunked(const void* r, int ldr, const void* k, int ldk, const void* v, int ldv, const float* z, int ldz,
                           const float* w0, const float* u, float* state, long long slot_pitch, const int* slots,
                           const int* cu_q, const int* kv_lens, int h, int d, void* out, int seq_base, int num_seqs,
                           int max_q, float* scratch, cudaStream_t st);
}

namespace {

// Scratch of weight-mixing attention in a step.
static long long talking_bytes(const KsanaMixerStep* s, const KsanaMixerLayer& w) {
  const long long p = ksana_talking_prefill_bytes(w.h, s->num_prefill, s->cu_q_host, s->kv_lens_host);
  const long long d = s->one_token ? ksana_talking_decode_bytes(w.h, s->num_decode, s->max_kv_decode) : 0;
  return p > d ? p : d;
}

// How latent attention uses its scratch in a step: contexts of prompts (latents, then keys and values) in rounds of at
// most expand_bytes, absorbed queries and weighted latents for the tokens from `first` on.
struct LatentPlan {
  bool expand;   // prompts run over keys and values written out per head
  int first;     // tokens from here on attend to the latents themselves
  long long prompt_bytes, bytes;
};
static bool latent_expands(const KsanaMixerLayer& w) {
  return !((w.arank | w.rot | w.adim | w.avdim) & 7) && w.adim <= 128 && w.avdim <= 128 && w.rot <= 64;
}
// sequences [lo, end) of one round
static int latent_round(const KsanaMixerModel* m, const KsanaMixerStep* s, const KsanaMixerLayer& w, int lo,
                        long long* rows) {
  const long long per_row = 2LL * w.ah * (w.adim + w.avdim);
  int hi = lo;
  *rows = 0;
  while (hi < s->num_prefill && (hi == lo || (*rows + s->kv_lens_host[hi]) * per_row <= m->expand_bytes))
    *rows += s->kv_lens_host[hi++];
  return hi;
}
static LatentPlan latent_plan(const KsanaMixerModel* m, const KsanaMixerStep* s, const KsanaMixerLayer& w) {
  LatentPlan p{latent_expands(w), 0, 0, 0};
  p.first = p.expand ? s->prefill_tokens : 0;
  long long most = 0;
  if (p.expand)
    for (int lo = 0; lo < s->num_prefill;) {
      long long rows;
      lo = latent_round(m, s, w, lo, &rows);
      if (rows > most) most = rows;
    }
  p.prompt_bytes = most * 2 * (w.arank + w.rot + static_cast<long long>(w.ah) * (w.adim + w.avdim));
  p.bytes = p.prompt_bytes + (s->total_tokens - p.first) * 2LL * w.ah * (2 * w.arank + w.rot);
  return p;
}

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

  // the same over hyper-connected streams: sublayer `sub` of `w` hands over y and / or routed rows; in_w and norm_w are the
  // next sublayer's
  bool hyper(int id, const KsanaMixerLayer& w, int sub, const void* y, bool routed, const float* in_w, const void* norm_w,
             bool first) {
    const int H = m->hidden;
    void* out = m->h_buf[pp];
    if (!step(id, ksana_hyper_norm(y, H, w.ls[sub], routed ? m->rows_out_buf : nullptr, m->pair_pos, m->expert_weights,
                                   routed ? w.top : 0, first ? s->start : residual, first, w.hc_mix[sub], w.hc_out[sub],
                                   residual, in_w, norm_w, out, s->total_tokens, H, m->streams, m->eps, 1, st)))
      return false;
    h = out;
    pp ^= 1;
    return true;
  }

  int head_gemm(const void* a, long long a_row, long long a_head, const void* w, void* c, long long c_row,
                long long c_head, int rows, int heads, int N, int K) {
    const int rc = ksana_gemm_bf16_batched(a, a_row, a_head, w, c, c_row, c_head, rows, heads, N, K, st);
    return rc == -1 ? ksana_head_gemm_any(a, a_row, a_head, w, c, c_row, c_head, rows, heads, N, K, 1, st) : rc;
  }

  bool latent(const KsanaMixerLayer& w, char* x, char* out) {
    const int T = s->total_tokens, ld = w.n_in, qd = w.adim + w.rot, nq = w.ah * qd, width = w.arank + w.rot;
    const LatentPlan p = latent_plan(m, s, w);
    if (p.bytes > m->lat_bytes) return step(21, -6);
    char* a = x + static_cast<size_t>(nq) * 2;
    const char* gate = w.head_gate ? a + static_cast<size_t>(width) * 2 : nullptr;
    char* buf = static_cast<char*>(m->lat_buf);
    // absorbed queries and weighted latents of `rows` tokens lie behind the prompts' part
    const int rows = T - p.first, ldc = w.ah * width, ldo = w.ah * w.arank;
    char *q_cat = buf + p.prompt_bytes, *o = q_cat + static_cast<size_t>(rows) * ldc * 2;
    if (!step(21, ksana_latent_append(x, ld, w.adim, q_cat, p.first, a, ld, w.anorm, m->eps, s->positions, w.rot_table,
                                      s->slot_mapping, w.kv, T, w.ah, w.arank, w.rot, 1, st)))
      return false;
    if (p.first > 0) {
      for (int lo = 0; lo < s->num_prefill;) {
        long long ctx;
        const int hi = latent_round(m, s, w, lo, &ctx);
        int max_kv = 0, max_q = 0;
        for (int b = lo; b < hi; ++b) {
          max_kv = s->kv_lens_host[b] > max_kv ? s->kv_lens_host[b] : max_kv;
          const int q = s->cu_q_host[b + 1] - s->cu_q_host[b];
          max_q = q > max_q ? q : max_q;
        }
        char* kv = buf + ctx * width * 2;
        const int n = w.ah * (w.adim + w.avdim), R = static_cast<int>(ctx);
        if (!step(22, ksana_latent_gather(w.kv, s->block_tables, s->max_blocks, s->kv_lens, lo, hi - lo, max_kv,
                                          m->block_size, width, buf, st)) ||
            !step(23, ksana_gemm_bf16(buf, w.a_expand, kv, nullptr, R, n, w.arank, width, w.arank, n, 0, 0, 0, m->gemm_ws,
                                      m->gemm_ws_floats, m->gemm_counters, m->n_counters, st)) ||
            !step(24, ksana_latent_prefill(x, ld, T, kv, n, buf + w.arank * 2, width, R, s->cu_q, s->kv_lens, w.ah, w.adim,
                                           w.rot, w.avdim, w.ascale, gate, ld, out, w.k_out, lo, hi - lo, max_q, st)))
          return false;
        lo = hi;
      }
    }
    if (rows == 0) return true;
    if (!step(26, head_gemm(x + static_cast<size_t>(p.first) * ld * 2, ld, qd, w.a_uk_t, q_cat, ldc, width, rows, w.ah,
                            w.arank, w.adim)))
      return false;
    // the kernels index tokens of the whole step
    const char* qc = q_cat - static_cast<size_t>(p.first) * ldc * 2;
    char* oc = o - static_cast<size_t>(p.first) * ldo * 2;
    int rc = -1;
    if (p.first == s->prefill_tokens)  // only the sequences behind the prompts
      rc = ksana_latent_decode(qc, ldc, T, w.kv, m->num_blocks, s->block_tables, s->max_blocks, s->cu_q, s->kv_lens, w.ah,
                               w.arank, w.rot, m->block_size, w.ascale, gate, ld, oc, ldo, s->num_prefill, s->num_decode,
                               s->max_q_decode, s->max_kv_decode, st);
    if (rc == -1)
      rc = ksana_window_attention_any(qc, ldc, w.kv, s->block_tables, s->max_blocks, s->cu_q, s->kv_lens, s->seq_of_token,
                                      w.ah, 1, width, w.arank, m->block_size, 0, 0, 1, w.ascale, nullptr, 0, 1.f, 0.f, 0,
                                      gate, ld, oc, ldo, p.first, rows, 1, st);
    if (!step(27, rc)) return false;
    return step(28, head_gemm(o, ldo, w.arank, w.a_uv, out + static_cast<size_t>(p.first) * w.k_out * 2, w.k_out, w.avdim,
                              rows, w.ah, w.avdim, w.arank));
  }

  bool recurrence(const KsanaMixerLayer& w, char* y, char* out) {
    const int ld = w.n_in, C = w.rc;
    char* x = y + static_cast<size_t>(C) * 2;
    auto general = [&](int id, int seq_base, int seqs, int tok_base, int tokens) {
      const long long need = static_cast<long long>(tokens) * C * 5 / 2 + 4;
      if (need > m->chunk_floats) return step(id, -6);
      float* z = m->chunk_buf;
      void* u = z + static_cast<long long>(tokens) * C * 2;
      const int part = C / w.rb;
      *launches += 2;
      if (int rc = ksana_recurrence_conv(x, ld, w.state, s->state_slots, s->cu_q, s->kv_lens, s->seq_of_token, w.conv_w,
                                         w.conv_b, C, w.rk, u, tok_base, tokens, 1, st))
        return step(id, rc);
      if (int rc = ksana_head_gemm_any(u, C, part, w.gates_by_block, z, 2LL * C, 2LL * part, tokens, w.rb, 2 * part, part,
                                       2, st))
        return step(id, rc);
      return step(id, ksana_recurrence_scan(y, ld, x, ld, w.state, s->state_slots, s->cu_q, s->kv_lens, u, z, w.gates_b,
                                            w.rate, C, w.rk, w.rb, out, w.k_out, seq_base, seqs, tok_base, 1, st));
    };
    if (s->num_prefill > 0) {
      int rc = -6;
      if (ksana_recurrence_scratch(s->prefill_tokens, s->num_prefill, s->max_q_prefill, C) <= m->chunk_floats)
        rc = ksana_recurrence_prompts(y, ld, x, ld, w.state, s->state_slots, s->cu_q, s->kv_lens, s->seq_of_token,
                                      w.conv_w, w.conv_b, w.gates, w.gates_b, w.rate, C, w.rk, w.rb, out, w.k_out, 0,
                                      s->num_prefill, 0, s->prefill_tokens, s->max_q_prefill, m->chunk_buf, st);
      if (rc == -1) {
        if (!general(29, 0, s->num_prefill, 0, s->prefill_tokens)) return false;
      } else {
        *launches += 2;
        if (!step(29, rc)) return false;
      }
    }
    if (s->num_decode > 0) {
      int rc = -1;
      if (s->one_token)
        rc = ksana_recurrence_step(y, ld, x, ld, w.state, s->state_slots, s->cu_q, s->kv_lens, w.conv_w, w.conv_b, w.gates,
                                   w.gates_b, w.rate, C, w.rk, w.rb, out, w.k_out, s->num_prefill, s->num_decode, st);
      if (rc == -1) return general(30, s->num_prefill, s->num_decode, s->prefill_tokens, s->total_tokens - s->prefill_tokens);
      if (!step(30, rc)) return false;
    }
    return true;
  }

  bool attention(const KsanaMixerLayer& w, char* x, void* out) {
    const int T = s->total_tokens, ld = w.n_in, nq = w.h * w.d, nk = w.reads ? 0 : w.hk * w.d;
    char *k = x + static_cast<size_t>(nq) * 2, *v = k + static_cast<size_t>(nk) * 2;
    const char* gate = w.head_gate ? v + (w.reads ? 0 : static_cast<size_t>(w.hk * w.dv) * 2) : nullptr;
    if (w.shared_kv) {  // the keys go to the cache in the launch that runs a parallel dense FFN's activation
      const int I = w.parallel ? w.inter : 0;
      if (!step(2, ksana_append_act(k, v, ld, s->slot_mapping, w.kv, T, w.hk, w.d, m->block_size,
                                    static_cast<char*>(out) + static_cast<size_t>(w.h * w.dv) * 2, w.k_out, I, w.gated, 1,
                                    st)))
        return false;
    } else if (!step(2, ksana_qk_norm_cache(x, ld, k, ld, v, ld, s->slot_mapping, w.kv, w.q_norm, w.k_norm, m->eps,
                                            s->positions, w.rot_table, w.rot, T, w.h, w.reads ? 0 : w.hk, w.d, w.dv,
                                            m->block_size, 1, st))) {
      return false;
    }
    auto general = [&](int first, int count) {
      return ksana_window_attention_any(x, ld, w.kv, s->block_tables, s->max_blocks, s->cu_q, s->kv_lens, s->seq_of_token,
                                        w.h, w.hk, w.d, w.dv, m->block_size, w.window, w.keep_first, w.shared_kv,
                                        w.scale, w.bias, w.bias_len, w.attn_out_scale, w.softcap, w.sink, gate, ld, out, w.k_out,
                                        first, count, 1, st);
    };
    if (s->num_prefill > 0) {
      int rc = ksana_window_prefill(x, ld, T, w.kv, m->num_blocks, s->block_tables, s->max_blocks, s->cu_q, s->kv_lens,
                                    w.h, w.hk, w.d, w.dv, m->block_size, w.window, w.keep_first, w.shared_kv, w.scale,
                                    w.bias, w.bias_len, w.attn_out_scale, w.softcap, w.sink, gate, ld, out, w.k_out, 0,
                                    s->num_prefill, s->max_q_prefill, st);
      if (rc == -1) rc = general(0, s->prefill_tokens);
      if (!step(3, rc)) return false;
    }
    if (s->num_decode > 0) {
      int rc = -1;
      if (s->one_token)
        rc = ksana_window_decode(x, ld, w.kv, m->num_blocks, s->block_tables, s->max_blocks, s->cu_q, s->kv_lens, w.h, w.hk, w.d, w.dv,
                                 m->block_size, w.window, w.keep_first, w.shared_kv, w.scale, w.bias, w.bias_len,
                                 w.attn_out_scale, w.softcap, w.sink, gate, ld, out, w.k_out, s->num_prefill,
                                 s->num_decode, s->max_kv_decode, st);
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
                                    w.lin_out_scale, 0, 1, st));
  }

  // experts of the tokens in `h`; their rows stay in sorted order for the norm that adds them up
  bool experts(const KsanaMixerLayer& w) {
    const int T = s->total_tokens, H = m->hidden, I = w.expert_inter, n = T * w.top;
    const int* offsets = m->sort_meta + w.experts;
    const int in_rows = w.experts_plain ? I : 2 * I;
    if (!step(15, gemm(h, H, w.w_router, nullptr, m->router_buf, w.router_rows, w.router_rows, 1))) return false;
    if (!step(16, ksana_moe_topk(m->router_buf, w.router_rows, w.b_router, T, w.experts, w.top, w.groups, w.keep_groups,
                                 w.scoring, w.router_scale, m->expert_ids, m->expert_weights, st)))
      return false;
    ++*launches;
    if (!step(17, ksana_moe_permute(h, H, m->expert_ids, T, w.top, H, 0, w.experts, m->sort_meta, m->pair_pos,
                                    m->pair_src, m->rows_buf, st)))
      return false;
    if (!step(18, ksana_moe_grouped_gemm(m->rows_buf, w.w_expert_gu, m->rows_gu_buf, offsets, w.experts, n, in_rows, H, st)))
      return false;
    int rc = w.experts_plain ? ksana_relu2(m->rows_gu_buf, I, m->rows_act_buf, n, I, 1, st)
             : w.limit > 0.f ? ksana_clamped_gate_mul(m->rows_gu_buf, m->rows_act_buf, n, I, w.limit, w.alpha, 1, st)
                           : ksana_silu_mul(m->rows_gu_buf, 2 * I, m->rows_act_buf, I, n, I, st);
    if (rc == -1) rc = ksana_silu_mul_any(m->rows_gu_buf, m->rows_act_buf, n, I, 1, st);
    if (!step(19, rc)) return false;
    return step(20, ksana_moe_grouped_gemm(m->rows_act_buf, w.w_expert_down, m->rows_out_buf, offsets, w.experts, n, H, I,
                                           st));
  }

  bool feed_forward(const KsanaMixerLayer& w) {
    const int T = s->total_tokens, H = m->hidden, I = w.inter;
    if (w.plain) {
      if (!step(11, gemm(h, H, w.w_gu, w.b_up, m->gu_buf, I, I))) return false;
      if (!step(12, ksana_relu2(m->gu_buf, I, m->act_buf, T, I, 1, st))) return false;
    } else if (w.w_gu_il != nullptr && T >= 384) {
      if (!step(11, ksana_gemm_bf16_geglu(h, w.w_gu_il, m->act_buf, T, 2 * I, H, H, H, I, st))) return false;
    } else {
      if (!step(11, gemm(h, H, w.w_gu, nullptr, m->gu_buf, 2 * I, 2 * I))) return false;
      if (!step(12, ksana_gelu_mul(m->gu_buf, 2 * I, m->act_buf, I, T, I, 1, st))) return false;
    }
    return step(13, gemm(m->act_buf, I, w.w_down, w.plain ? w.b_down : nullptr, m->proj_buf, H, H));
  }

  bool talking(const KsanaMixerLayer& w, char* x, void* out) {
    const int T = s->total_tokens, ld = w.n_in;
    char *k = x + static_cast<size_t>(w.h * w.d) * 2, *v = k + static_cast<size_t>(w.hk * w.d) * 2;
    const char* gate = w.out_gate ? v + static_cast<size_t>(w.hk * w.dv) * 2 : nullptr;
    auto append = w.qk_norm_all ? ksana_qk_row_norm_cache : ksana_qk_norm_cache;
    if (!step(2, append(x, ld, k, ld, v, ld, s->slot_mapping, w.kv, w.q_norm, w.k_norm, m->eps, s->positions, w.rot_table,
                        w.rot, T, w.h, w.hk, w.d, w.dv, m->block_size, 1, st)))
      return false;
    auto general = [&](int first, int count) {
      return ksana_talking_any(x, ld, w.kv, s->block_tables, s->max_blocks, s->cu_q, s->kv_lens, s->seq_of_token, w.h, w.hk,
                               w.d, w.dv, m->block_size, w.scale, w.talk_sink, w.talk_mix, w.attn_out_scale, gate, ld, out,
                               w.k_out, first, count, 1, st);
    };
    if (s->num_prefill > 0) {
      int n = 0;
      int rc = ksana_talking_prefill(x, ld, T, w.kv, m->num_blocks, s->block_tables, s->max_blocks, s->cu_q, s->kv_lens, w.h,
                                     w.hk, w.d, w.dv, m->block_size, w.scale, w.talk_sink, w.talk_mix, w.attn_out_scale, gate,
                                     ld, out, w.k_out, s->num_prefill, s->cu_q_host, s->kv_lens_host, m->lat_buf,
                                     m->lat_bytes, &n, st);
      if (rc == -1) rc = general(0, s->prefill_tokens); else *launches += n - 1;
      if (!step(31, rc)) return false;
    }
    if (s->num_decode > 0) {
      int rc = -1;
      if (s->one_token) {
        rc = ksana_talking_decode(x, ld, w.kv, m->num_blocks, s->block_tables, s->max_blocks, s->cu_q, s->kv_lens, w.h, w.hk,
                                  w.d, w.dv, m->block_size, w.scale, w.talk_sink, w.talk_mix, w.attn_out_scale, gate, ld, out,
                                  w.k_out, s->num_prefill, s->num_decode, s->max_kv_decode, m->lat_buf, m->lat_bytes, st);
        if (rc == 0) ++*launches;
      }
      if (rc == -1) rc = general(s->prefill_tokens, T - s->prefill_tokens);
      if (!step(32, rc)) return false;
    }
    return true;
  }

  bool time_mix(const KsanaMixerLayer& w, char* out) {
    const int T = s->total_tokens, H = m->hidden, n = w.mh * w.md, ld = w.mpad;
    const long long pitch = static_cast<long long>(n) * w.md + H;  // of a state slot: the heads' states, the last token
    if (!step(33, ksana_token_mix(h, w.mu, w.state + pitch - H, pitch, 1, s->state_slots, s->cu_q, s->kv_lens,
                                  s->seq_of_token, m->mixes_buf, T, H, 5, 1, st)))
      return false;
    const char* mixes = static_cast<const char*>(m->mixes_buf);
    char* rkvg = static_cast<char*>(m->rkvg_buf);
    const size_t in = static_cast<size_t>(T) * H * 2, to = static_cast<size_t>(T) * ld * 2;
    for (int i = 0; i < 4; ++i)
      if (!step(34, gemm(mixes + i * in, H, static_cast<const char*>(w.w_mix) + static_cast<size_t>(i) * ld * H * 2, nullptr,
                         rkvg + i * to, ld, ld)))
        return false;
    if (!step(35, gemm(mixes + 4 * in, H, w.w_decay1, nullptr, m->rank_buf, w.mrank, w.mrank, 1))) return false;
    if (!step(36, ksana_tanh_parts(m->rank_buf, w.mrank, m->tanh_buf, T, 1, st))) return false;
    if (!step(37, gemm(m->tanh_buf, 2 * w.mrank, w.w_decay2, nullptr, m->decay_buf, ld, ld, 1))) return false;
    const char *r = rkvg, *k = r + to, *v = k + to, *g = v + to;
    int n_long = s->num_long;
    if (n_long > 0) {
      int rc = -1;
      if (ksana_time_mix_scratch(s->long_tokens, n_long, w.mh, w.md) <= m->chunk_floats)
        rc = ksana_time_mix_chunked(r, ld, k, ld, v, ld, m->decay_buf, ld, w.w_decay0, w.bonus, w.state, pitch, s->state_slots,
                                    s->cu_q, s->kv_lens, w.mh, w.md, m->o_buf, 0, n_long, s->max_q_prefill, m->chunk_buf, st);
      if (rc == -1) {
        n_long = 0;  // not a size of the chunked form
      } else {
        *launches += 2;
        if (!step(38, rc)) return false;
      }
    }
    const int base[2] = {n_long, s->num_prefill}, count[2] = {s->num_prefill - n_long, s->num_decode};
    for (int i = 0; i < 2; ++i)
      if (count[i] > 0 &&
          !step(39, ksana_time_mix_recurrent(r, ld, k, ld, v, ld, m->decay_buf, ld, w.w_decay0, w.bonus, w.state, pitch,
                                             s->state_slots, s->cu_q, s->kv_lens, w.mh, w.md, m->o_buf, base[i], count[i],
                                             i == 1 && s->one_token, 1, st)))
        return false;
    return step(40, ksana_gated_norm(m->o_buf, g, ld, w.mix_norm, out, w.k_out, T, w.mh, w.md, m->eps, 0, w.mix_out_scale, 1,
                                     1, st));
  }

  bool gated_layer(const KsanaMixerLayer& w) {
    const int T = s->total_tokens, H = m->hidden;
    char *x = static_cast<char*>(m->in_buf), *mix = static_cast<char*>(m->mix_buf);
    const char* h0 = static_cast<const char*>(h);
    if (!step(1, gemm(h, H, w.w_in, w.b_in, x, w.n_in, w.n_in))) return false;
    const int used = w.h * w.dv + w.mh * w.md;
    if (used < w.k_out &&
        cudaMemset2DAsync(mix + static_cast<size_t>(used) * 2, static_cast<size_t>(w.k_out) * 2, 0,
                          static_cast<size_t>(w.k_out - used) * 2, T, st) != cudaSuccess)
      return step(8, -5);
    if (!talking(w, x, mix)) return false;
    if (w.mh > 0 && !time_mix(w, mix + static_cast<size_t>(w.h * w.dv) * 2)) return false;
    if (!step(9, gemm(mix, w.k_out, w.w_out, w.b_out, m->proj_buf, H, H))) return false;
    const int attn_in = w.h * w.d + w.hk * (w.d + w.dv) + (w.out_gate ? w.h * w.dv : 0), n = H + w.shared_ff;
    if (w.experts > 0) {
      h = h0 + static_cast<size_t>(T) * H * 2;
      if (!experts(w)) return false;
      if (!step(41, gemm(h, H, w.w_ff_in, w.b_ff_in, m->gu_buf, n, n))) return false;
      if (!step(42, ksana_relu2(static_cast<char*>(m->gu_buf) + static_cast<size_t>(H) * 2, n, m->act_buf, T, w.shared_ff, 1, st)))
        return false;
      if (!step(43, gemm(m->act_buf, w.shared_ff, w.w_shared_down, nullptr, m->shared_buf, H, H))) return false;
    }
    const bool ff = w.experts > 0;
    void* out = m->h_buf[pp];
    if (!step(44, ksana_gated_stream_norm(m->proj_buf, H, x + static_cast<size_t>(attn_in) * 2, w.n_in,
                                          ff ? m->rows_out_buf : nullptr, m->pair_pos, m->expert_weights, w.top,
                                          ff ? m->shared_buf : nullptr, H, ff ? m->router_buf + w.experts : nullptr,
                                          w.router_rows, ff ? m->gu_buf : nullptr, n, m->residual_scale, residual, residual,
                                          w.next_ln, w.next_ln2, out, T, H, m->eps, 1, st)))
      return false;
    h = out;
    pp ^= 1;
    return true;
  }

  bool layer(const KsanaMixerLayer& w, bool first) {
    if (w.gated_residual) return gated_layer(w);
    const int T = s->total_tokens, H = m->hidden;
    char* x = static_cast<char*>(m->in_buf);
    char* mix = static_cast<char*>(m->mix_buf);
    if (!step(1, gemm(h, H, w.w_in, w.b_in, x, w.n_in, w.n_in))) return false;
    const int used = w.h * w.dv + w.ah * w.avdim + w.lh * w.ldv + w.rc + (w.parallel ? w.inter : 0);
    if (used < w.k_out &&
        cudaMemset2DAsync(mix + static_cast<size_t>(used) * 2, static_cast<size_t>(w.k_out) * 2, 0,
                          static_cast<size_t>(w.k_out - used) * 2, T, st) != cudaSuccess)
      return step(8, -5);
    if (w.h > 0 && !attention(w, x, mix)) return false;
    const size_t attn_in = w.h > 0 ? static_cast<size_t>(w.h * w.d + w.hk * (w.d + (w.shared_kv ? 0 : w.dv))) * 2 : 0;
    if (w.lh > 0 && !linear(w, x + attn_in, mix + static_cast<size_t>(w.h * w.dv) * 2)) return false;
    if (w.ah > 0 && !latent(w, x, mix)) return false;
    if (w.rc > 0 && !recurrence(w, x, mix)) return false;
    if (!step(9, gemm(mix, w.k_out, w.w_out, w.b_out, m->proj_buf, H, H))) return false;
    if (m->streams > 0) {
      const bool more = w.ln2 != nullptr;
      if (!hyper(10, w, 0, m->proj_buf, false, more ? w.hc_in[1] : w.next_in, more ? w.ln2 : w.next_ln, first)) return false;
      if (!more) return true;
      if (w.experts > 0) return experts(w) && hyper(14, w, 1, nullptr, true, w.next_in, w.next_ln, false);
      return feed_forward(w) && hyper(14, w, 1, m->proj_buf, false, w.next_in, w.next_ln, false);
    }
    if (w.experts > 0 && !experts(w)) return false;
    if (w.ln2 != nullptr && (!norm(10, m->proj_buf, w.ln2) || !feed_forward(w))) return false;
    return norm(14, m->proj_buf, w.next_ln, w.experts > 0, &w);
  }
};

}  // namespace

KSANA_API long long ksana_mixer_latent_bytes(const KsanaMixerModel* m, const KsanaMixerStep* s, int layers) {
  long long most = 0;
  for (int i = 0; i < layers; ++i)
    if (m->layers[i].talk) {
      const long long n = talking_bytes(s, m->layers[i]);
      if (n > most) most = n;
    } else if (m->layers[i].ah > 0) {
      const long long n = latent_plan(m, s, m->layers[i]).bytes;
      if (n > most) most = n;
    }
  return most;
}

KSANA_API int ksana_mixer_forward(const KsanaMixerModel* m, const KsanaMixerStep* s, const void* h, float* residual,
                                  int first, int last, void** out_h, int* fail_code, int* launches, cudaStream_t stream) {
  *fail_code = 0;
  *launches = 0;
  Exec ex{m, s, residual, launches, fail_code, stream};
  ex.h = h;
  for (int i = first; i < last && s->total_tokens > 0; ++i)
    if (!ex.layer(m->layers[i], i == 0)) return (i + 1) * 100 + ex.failed;
  *out_h = const_cast<void*>(ex.h);
  return 0;
}
