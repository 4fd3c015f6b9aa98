"""Operator front door.

CUDA tensors go to the hand-written sm_100a kernels (``ops.cuda``; a missing kernel library on a GPU
box is an error, never a silent fallback). CPU tensors go to the fp32 PyTorch restatements in
``ops.reference`` that also serve as the kernels' test oracle.
"""
from __future__ import annotations

from typing import Optional

import torch

from . import reference as ref


def _cuda():
    from . import cuda as _c
    return _c


def _mixer():
    from . import cuda_mixer as _c
    return _c


def rms_norm(x, weight, eps, residual=None):
    if x.is_cuda:
        return _cuda().rms_norm(x, weight, eps, residual)
    return ref.rms_norm(x, weight, eps, residual)


def layer_norm(x, weight, bias, eps, residual=None, out_dtype=None):
    if x.is_cuda:
        return _mixer().layer_norm(x, weight, bias, eps, residual, out_dtype)
    return ref.layer_norm(x, weight, bias, eps, residual, out_dtype)


def stream_norm(x, weight, eps, center, stream_in, stream_out=None, out_dtype=None, add_rows=None, add_vec=None,
                routed=None):
    """The 32-bit residual stream takes ``x`` (and more) and is normalised; see ``reference.stream_norm``."""
    f = _mixer() if stream_in.is_cuda else ref
    return f.stream_norm(x, weight, eps, center, stream_in, stream_out, out_dtype, add_rows, add_vec, routed)


def hyper_norm(x, scale, routed, streams, mix, out_w, streams_out, in_w, weight, eps, out_dtype):
    """Residual streams take a sublayer's result and the next sublayer's input is normalised; see
    ``reference.hyper_norm``."""
    f = _mixer() if streams.is_cuda else ref
    return f.hyper_norm(x, scale, routed, streams, mix, out_w, streams_out, in_w, weight, eps, out_dtype)


def _library_baseline() -> bool:
    """KSANA_LIBRARY_BASELINE=1 routes dense GEMMs to cuBLAS (torch.matmul): the measured stand-in for the
    reference's cuBLAS + NCCL build, never the default."""
    import os
    return os.environ.get("KSANA_LIBRARY_BASELINE", "0") == "1"


def linear(x, weight, bias=None, out_dtype=None):
    """``out_dtype`` float32: the accumulator leaves unrounded."""
    if x.is_cuda:
        if _library_baseline():
            y = torch.nn.functional.linear(x, weight, bias)
            return y if out_dtype is None else y.to(out_dtype)
        return _cuda().linear(x, weight, bias, out_dtype)
    return ref.linear(x, weight, bias, out_dtype)


def linear_fp8_block(x, wq, w_scale_inv, bias=None, sfb=None, pow2=False):
    """``pow2``: the weight's block scales are powers of two; the activations then get power-of-two group scales
    too and (CUDA, ``sfb`` = the packed scale bytes) large products run on the scaled tensor-core path."""
    if x.is_cuda:
        return _cuda().linear_fp8_block(x, wq, w_scale_inv, bias, sfb, pow2)
    return ref.linear_fp8_block(x, wq, w_scale_inv, bias, ue8m0=pow2)


def linear_int4(x, packed, scales, zeros, bias=None, group=128, sz=None):
    if x.is_cuda:
        return _cuda().linear_int4(x, packed, scales, zeros, bias, group, sz=sz)
    return ref.linear_int4(x, packed, scales, zeros, bias, group)


def silu_and_mul(x):
    if x.is_cuda:
        return _cuda().silu_and_mul(x)
    return ref.silu_and_mul(x)


def gelu_and_mul(x):
    if x.is_cuda:
        return _mixer().gelu_and_mul(x)
    return ref.gelu_and_mul(x)


def activation(x, kind):
    if x.is_cuda and kind == "gelu_tanh":
        return _mixer().gelu(x)
    if x.is_cuda and kind == "relu2":
        return _mixer().relu2(x)
    return ref.activation(x, kind)


def embedding(ids, table, scale=1.0, out_dtype=None, positions=None, pos_table=None):
    """``pos_table``: learned position vectors, added unscaled."""
    if ids.is_cuda and out_dtype is not None:
        return _mixer().embedding(ids, table, scale, out_dtype, positions, pos_table)
    if ids.is_cuda and pos_table is None:
        return _cuda().embedding(ids, table, scale)
    return ref.embedding(ids, table, scale, out_dtype, positions, pos_table)


def rope_qknorm_cache(q, k, v, positions, cos_sin, slot_mapping, kv_cache, q_norm_w=None, k_norm_w=None,
                      eps=1e-6, interleaved=False, rotary_dim=0, k_scale=1.0, v_scale=1.0, norm_after_rope=False):
    if norm_after_rope and q_norm_w is not None:
        # the fused kernel normalises before rotating: this order goes through the reference implementation
        return ref.rope_qknorm_cache(q, k, v, positions, cos_sin, slot_mapping, kv_cache, q_norm_w, k_norm_w, eps,
                                     interleaved, rotary_dim, k_scale, v_scale, True)
    if q.is_cuda:
        return _cuda().rope_qknorm_cache(q, k, v, positions, cos_sin, slot_mapping, kv_cache, q_norm_w, k_norm_w,
                                         eps, interleaved, rotary_dim, k_scale, v_scale)
    return ref.rope_qknorm_cache(q, k, v, positions, cos_sin, slot_mapping, kv_cache, q_norm_w, k_norm_w,
                                 eps, interleaved, rotary_dim, k_scale, v_scale)


def paged_attention(q, kv_cache, meta, scale, alibi_slopes=None, k_scale=1.0, v_scale=1.0, window=0):
    """``meta`` is the step's :class:`~ksanallm_b200.engine.step_input.StepInput`."""
    if q.is_cuda:
        return _cuda().paged_attention(q, kv_cache, meta, scale, alibi_slopes, k_scale, v_scale, window)
    return ref.paged_attention(q, kv_cache, meta.block_tables, meta.cu_q, meta.kv_lens, scale, alibi_slopes,
                               k_scale, v_scale, window)


def qk_norm_cache(q, k, v, slot_mapping, cache, block_size, q_norm, k_norm, eps, positions=None, rotary=None,
                  norm_all=False, halves=False):
    f = _mixer() if q.is_cuda else ref
    return f.qk_norm_cache(q, k, v, slot_mapping, cache, block_size, q_norm, k_norm, eps, positions, rotary, norm_all,
                           halves)


def talking_attention(q, cache, meta, block_size, kv_heads, vdim, scale, sink, talk, out_scale, out, gate=None):
    """Writes heads * vdim columns of ``out`` [T, ...] (a column slice is fine); see ``reference.talking_attention``."""
    if q.is_cuda:
        from . import cuda_talking
        cuda_talking.talking_attention(q, cache, meta, block_size, kv_heads, vdim, scale, sink, talk, out_scale, out, gate)
        return
    out.copy_(ref.talking_attention(q, cache, meta.block_tables, meta.cu_q, meta.kv_lens, block_size, kv_heads, vdim, scale,
                                    sink, talk, out_scale, gate).flatten(1))


def token_mix(h, mu, state, meta):
    """``state`` [slots, 1, 1, n]: the previous token's vector is the last W numbers of a slot."""
    if h.is_cuda:
        from . import cuda_timemix
        return cuda_timemix.token_mix(h, mu, state, meta)
    return ref.token_mix(h, mu, state.flatten(1)[:, -h.shape[1]:], meta.state_slots, meta.cu_q, meta.kv_lens)


def tanh_parts(x, dtype):
    if x.is_cuda:
        from . import cuda_timemix
        return cuda_timemix.tanh_parts(x, dtype)
    return ref.tanh_parts(x, dtype)


def time_mix(r, k, v, z, w0, u, state, meta):
    """``state`` as in :func:`token_mix`: the heads' states are the first h * d * d numbers of a slot."""
    if r.is_cuda:
        from . import cuda_timemix
        return cuda_timemix.time_mix(r, k, v, z, w0, u, state, meta)
    h, d = u.shape
    S = state.flatten(1)[:, :h * d * d].unflatten(1, (h, d, d))
    return ref.time_mix(r, k, v, z, w0, u, S, meta.state_slots, meta.cu_q, meta.kv_lens)


def gated_stream_norm(x, x_gate, routed, y, y_scale, y_gate, scale, stream_in, stream_out, weights, eps, out_dtype):
    f = ref
    if stream_in.is_cuda:
        f = _mixer()
    return f.gated_stream_norm(x, x_gate, routed, y, y_scale, y_gate, scale, stream_in, stream_out, weights, eps, out_dtype)


def latent_attention(q, a, norm_w, eps, rotary, cache, meta, block_size, w, scale, gate, out):
    """Rotation, cache append and attention; ``w``: :class:`~ksanallm_b200.models.mixers.LatentWeights`. Writes
    heads * vdim columns of ``out``."""
    if q.is_cuda:
        from . import cuda_latent
        cuda_latent.latent_attention(q, a, norm_w, eps, rotary, cache, meta, block_size, w, scale, gate, out)
        return
    ref.latent_append(q, a, norm_w, eps, meta.positions, rotary, meta.slot_mapping, cache, block_size)
    out.copy_(ref.latent_attention(q, cache, meta.block_tables, meta.cu_q, meta.kv_lens, block_size, w.uk, w.uv, scale,
                                   gate).flatten(1))


def gated_recurrence(y, x, state, meta, w, out):
    """``w``: :class:`~ksanallm_b200.models.mixers.RecurrenceWeights`. Writes ``out`` [T, C] (a column slice is fine)."""
    if x.is_cuda:
        from . import cuda_recurrence
        cuda_recurrence.gated_recurrence(y, x, state, meta, w, out)
        return
    out.copy_(ref.gated_recurrence(y, x, state, meta.state_slots, meta.cu_q, meta.kv_lens, w.conv, w.conv_b, w.gates,
                                   w.gates_b, w.rate))


def append_act(k, u, slot_mapping, cache, block_size, out, gated=False):
    """Keys to a cache of keys alone and / or a GELU feed-forward's activation; see ``reference.append_act``."""
    f = _mixer() if (k if k is not None else u).is_cuda else ref
    f.append_act(k, u, slot_mapping, cache, block_size, out, gated)


def window_attention(q, cache, meta, block_size, kv_heads, vdim, scale, window, bias, out_scale, out, keep_first=0,
                     softcap=0.0, sink=False, gate=None):
    """Writes heads * vdim columns of ``out`` [T, ...] (a column slice is fine). Whether the cache holds values of their
    own or the keys are the values shows in its width."""
    if q.is_cuda:
        _mixer().window_attention(q, cache, meta, block_size, kv_heads, vdim, scale, window, bias, out_scale, out,
                                  keep_first, softcap, sink, gate)
        return
    out.copy_(ref.window_attention(q, cache, meta.block_tables, meta.cu_q, meta.kv_lens, block_size, kv_heads, vdim,
                                   scale, window, bias, out_scale, keep_first, softcap, sink, gate).flatten(1))


def linear_attention(q, k, v, state, meta, decay, act, rotary, key_scale):
    if q.is_cuda:
        return _mixer().linear_attention(q, k, v, state, meta, decay, act, rotary, key_scale)
    return ref.linear_attention(q, k, v, state, meta.state_slots, meta.cu_q, meta.kv_lens, meta.positions, decay, act,
                                rotary, key_scale)


def gated_norm(o, g, weight, eps, gate, out_scale, out, per_head=False):
    if o.is_cuda:
        _mixer().gated_norm(o, g, weight, eps, gate, out_scale, out, per_head)
        return
    out.copy_(ref.gated_norm(o, g, weight, eps, gate, out_scale, per_head))


def softcap(logits, cap):
    if logits.is_cuda:
        return _mixer().softcap(logits, cap)
    return ref.softcap(logits, cap)


def mla_cache_append(latent, k_rope, slot_mapping, cache):
    if latent.is_cuda:
        return _cuda().mla_cache_append(latent, k_rope, slot_mapping, cache)
    return ref.mla_cache_append(latent, k_rope, slot_mapping, cache)


def mla_paged_attention(q_latent, q_rope, cache, meta, scale):
    if q_latent.is_cuda:
        return _cuda().mla_paged_attention(q_latent, q_rope, cache, meta, scale)
    return ref.mla_paged_attention(q_latent, q_rope, cache, meta.block_tables, meta.cu_q, meta.kv_lens, scale)


def moe_route(logits, top_k, scoring="softmax", norm_topk=False, n_group=1, topk_group=1, routed_scale=1.0,
              correction_bias=None):
    if logits.is_cuda:
        return _cuda().moe_route(logits, top_k, scoring, norm_topk, n_group, topk_group, routed_scale, correction_bias)
    return ref.moe_route(logits, top_k, scoring, norm_topk, n_group, topk_group, routed_scale, correction_bias)


def moe_topk(logits, experts, top_k, bias=None, groups=1, keep=1, scoring="softmax", scale=1.0):
    if logits.is_cuda:
        from . import cuda_moe
        return cuda_moe.moe_topk(logits, experts, top_k, bias, groups, keep, scoring, scale)
    return ref.moe_topk(logits, experts, top_k, bias, groups, keep, scoring, scale)


def moe_expert_rows(x, ids, w_gate_up, w_down, limit=0.0, alpha=1.0, plain=False):
    if x.is_cuda:
        from . import cuda_moe
        return cuda_moe.expert_pipeline(x, ids, w_gate_up, w_down, 0, limit, alpha, plain)
    return ref.moe_expert_rows(x, ids, w_gate_up, w_down, limit, alpha, plain)


def moe_experts(x, ids, weights, w_gate_up, w_down, expert_offset=0):
    if x.is_cuda:
        return _cuda().moe_experts(x, ids, weights, w_gate_up, w_down, expert_offset)
    return ref.moe_experts(x, ids, weights, w_gate_up, w_down, expert_offset)


def argmax(logits):
    if logits.is_cuda:
        return _cuda().argmax(logits)
    return ref.argmax(logits)


def sample(logits, temperature, top_k, top_p, uniform):
    if logits.is_cuda:
        return _cuda().sample(logits, temperature, top_k, top_p, uniform)
    return ref.sample(logits, temperature, top_k, top_p, uniform)
