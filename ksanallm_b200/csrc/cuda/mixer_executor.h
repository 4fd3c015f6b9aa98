// Native forward pass of layers with mixers of their own sizes (windowed attention and / or linear attention, latent
// attention, a gated recurrence, weight-mixing attention beside time mixing; a norm over a 32-bit residual stream, or over
// several hyper-connected ones; a dense or routed FFN behind or beside the mixers), driven from ONE call per step. A layer that runs several times is listed once
// per run. Mirrored with ctypes on the Python side.
#pragma once
#include <cuda_runtime.h>

extern "C" {

struct KsanaMixerLayer {
  // weights, bf16
  const void* w_in;      // [n_in, H]: attention q, k, v, head gates (or latent q, latent, head gates, or the recurrence's
                         // y, x), linear attention q, k, v, gate, then a parallel dense FFN's input
  const void* b_in;      // optional bias [n_in]
  const void* w_out;     // [H, k_out]: attention columns, linear-attention columns, a parallel dense FFN's, zero padding
  const void* b_out;     // optional bias [H]
  const void* ln2;       // norm before the FFN (null: the layer has none, or it reads the mixers' norm)
  const void* w_gu;      // [2 I, H] gate rows, then up rows; plain: [I, H]
  const void* b_up;      // plain: optional bias [I]
  const void* b_down;    // plain: optional bias [H]
  const void* w_gu_il;   // optional copy of w_gu, gate / up rows interleaved in groups of 16: prompt-sized steps then run
                         // the activation as the GEMM's epilogue
  const void* w_down;    // [H, I]
  const void* next_ln;   // next layer's first norm, or the final norm
  int n_in, k_out, inter;
  int plain;             // FFN behind the mixers: squared ReLU instead of gated GELU
  // FFN beside the mixers: dense of width `inter` inside w_in / w_out, or routed experts (experts > 0)
  int parallel, gated;
  int experts, top, expert_inter, router_rows, groups, keep_groups;
  float limit, alpha;           // limit > 0: clamped gates
  const void* w_router;         // [router_rows, H], rows from `experts` on are padding
  const float* b_router;        // optional [experts]
  const void* w_expert_gu;      // [experts, 2 expert_inter, H]
  const void* w_expert_down;    // [experts, H, expert_inter]
  // what the stream takes between this layer and the next norm
  const float* next_vec;        // optional [H]
  int next_start;               // add the embedding output
  // softmax attention (h == 0: none)
  int h, hk, d, dv, window, keep_first, shared_kv, bias_len;
  float scale, attn_out_scale, softcap;
  int sink, head_gate, reads;  // reads: another layer's keys and values, nothing is appended
  int rot;                     // rotated dimensions (of latent attention: its shared part)
  const float* rot_table;
  const float* q_norm;
  const float* k_norm;
  const float* bias;     // [h, bias_len]
  void* kv;              // this layer's cache
  // linear attention (lh == 0: none)
  int lh, ld, ldv, rd, act, gate;
  float key_scale, lin_out_scale;
  const float* decay;
  const float* rotary;
  const float* norm_w;   // null: per-head norm without weight
  float* state;          // this layer's state pool
  // latent attention (ah == 0: none)
  int ah, adim, avdim, arank;
  float ascale;
  const float* anorm;
  const void* a_uk_t;    // [ah, arank, adim]
  const void* a_uv;      // [ah, avdim, arank]
  const void* a_expand;  // [ah (adim + avdim), arank]
  // gated recurrence (rc == 0: none)
  int rc, rk, rb;
  const float* conv_w;
  const float* conv_b;
  const void* gates;           // [2, rb, rc / rb, rc / rb]
  const void* gates_by_block;  // [rb, 2 rc / rb, rc / rb]
  const float* gates_b;
  const float* rate;
  // hyper-connections of the two sublayers, and their layer scales
  const float* ls[2];
  const float* hc_in[2];
  const float* hc_mix[2];
  const float* hc_out[2];
  const float* next_in;        // how the next layer (or the final norm) reads the streams
  // gated residual: mixers and experts side by side, over norms of their own (h_buf: two planes [T, H])
  int gated_residual, experts_plain, scoring, shared_ff;  // scoring: of the router, 1 sigmoid
  float router_scale;
  const void* next_ln2;        // the next layer's second norm (null: it has one)
  const void* w_ff_in;         // [H + shared_ff, H]: the experts' residual gate, the shared expert's input
  const void* b_ff_in;
  const void* w_shared_down;   // [H, shared_ff]
  // weight-mixing attention
  int talk, out_gate, qk_norm_all;
  const float* talk_mix;       // [h, h]
  const float* talk_sink;      // [h]
  // time mixing (mh == 0: none)
  int mh, md, mrank, mpad;     // mpad: rows of one projection (mh * md filled up)
  float mix_out_scale;
  const float* mu;             // [5, H]
  const void* w_mix;           // [4, mpad, H]: r, k, v, gate
  const void* w_decay1;        // [mrank, H]
  const void* w_decay2;        // [mpad, 2 mrank]
  const float* w_decay0;       // [mh * md]
  const float* bonus;          // [mh * md]
  const float* mix_norm;       // [mh * md]
};

struct KsanaMixerModel {
  int hidden, block_size, num_blocks, center;  // center: LayerNorm, else RMS norm
  int streams;                                 // 0: one residual stream
  float eps, residual_scale;                   // residual_scale: of gated sublayers
  // scratch for max_tokens rows
  void* in_buf;    // [T, max n_in]
  void* mix_buf;   // [T, max k_out]
  void* o_buf;     // [T, max lh * ldv or mh * md]
  void* gu_buf;    // [T, 2 max I]
  void* act_buf;   // [T, max I]
  void* proj_buf;  // [T, H]
  void* h_buf[2];  // [T, H]
  // routed experts: [T, max router_rows], [T, max top] (ids, weights), [T max top] (sorted row of a pair, pair of a sorted
  // row), the sort's counters, and rows in sorted order [T max top, H | 2 I | I | H]
  float* router_buf;
  int* expert_ids;
  float* expert_weights;
  int* pair_pos;
  int* pair_src;
  int* sort_meta;
  void* rows_buf;
  void* rows_gu_buf;
  void* rows_act_buf;
  void* rows_out_buf;
  float* chunk_buf;
  long long chunk_floats;
  // gated layers: [T, H] (shared expert), time mixing's [5][T, H], [4][T, mpad], [T, mrank] fp32, [T, 2 mrank], [T, mpad] fp32
  void* shared_buf;
  void* mixes_buf;
  void* rkvg_buf;
  float* rank_buf;
  void* tanh_buf;
  float* decay_buf;
  void* lat_buf;           // scratch of latent and of weight-mixing attention
  long long lat_bytes, expand_bytes;  // expand_bytes: keys and values that prompts have written out at a time
  float* gemm_ws;
  long long gemm_ws_floats;
  unsigned int* gemm_counters;
  int n_counters;
  const KsanaMixerLayer* layers;
};

struct KsanaMixerStep {
  const int* positions;
  const int* slot_mapping;
  const int* seq_of_token;
  const int* block_tables;
  const int* cu_q;
  const int* kv_lens;
  const int* state_slots;
  const float* start;    // the embedding output [T, H] (layers with next_start)
  int total_tokens, max_blocks;
  int num_prefill, num_decode, prefill_tokens;
  int max_q_prefill, max_kv_decode;
  int one_token;         // every decode sequence has exactly one new token
  int num_long;          // leading prompt portions long enough for the chunked form of linear attention
  int long_tokens;       // their tokens
  int max_q_decode;
  const int* cu_q_host;
  const int* kv_lens_host;
};

// h: normalised input of layer `first` ([T, H] bf16), residual: [T, H] fp32 stream, updated in place. *out_h receives
// the pointer of the normalised output. Returns 0, or (layer + 1) * 100 + step on failure with the failing call's code
// in *fail_code.
// Bytes of lat_buf that a step needs (the largest layer's).
long long ksana_mixer_latent_bytes(const KsanaMixerModel* m, const KsanaMixerStep* s, int layers);

int ksana_mixer_forward(const KsanaMixerModel* m, const KsanaMixerStep* s, const void* h, float* residual, int first,
                        int last, void** out_h, int* fail_code, int* launches, cudaStream_t stream);
}
