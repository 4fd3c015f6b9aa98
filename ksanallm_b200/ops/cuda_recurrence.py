"""Gated linear recurrence behind a short convolution (csrc/cuda/gated_recurrence.cu)."""
from __future__ import annotations

import torch

from .cuda import _check, _ptr, _stream, lib
from .cuda_latent import head_gemm
from .cuda_mixer import _KIND


def gated_recurrence(y, x, state, meta, w, out: torch.Tensor) -> None:
    """See ``reference.gated_recurrence``; ``w``: :class:`~ksanallm_b200.models.mixers.RecurrenceWeights`. bf16 prompts go
    through chunks on the tensor cores, bf16 single tokens through one launch; fp32 and other sizes through the general
    kernels."""
    T, C = x.shape
    K, B = w.conv.shape[1], w.gates.shape[1]
    assert x.stride(1) == y.stride(1) == out.stride(1) == 1 and state.is_contiguous()
    n_pre, n_dec, pre_tokens = meta.num_prefill, meta.num_decode, meta.num_prefill_tokens
    rows = (_ptr(y), y.stride(0), _ptr(x), x.stride(0), _ptr(state), _ptr(meta.state_slots), _ptr(meta.cu_q),
            _ptr(meta.kv_lens))
    maps = (_ptr(w.conv_t), _ptr(w.conv_b), _ptr(w.gates), _ptr(w.gates_b), _ptr(w.rate), C, K, B, _ptr(out), out.stride(0))

    def general(seq_base: int, seqs: int, tok_base: int, tokens: int) -> None:
        if not seqs or not tokens:
            return
        kind = _KIND[x.dtype]
        u = torch.empty(tokens, C, dtype=x.dtype, device=x.device)
        _check(lib().ksana_recurrence_conv(_ptr(x), x.stride(0), _ptr(state), _ptr(meta.state_slots), _ptr(meta.cu_q),
                                           _ptr(meta.kv_lens), _ptr(meta.seq_of_token), _ptr(w.conv_t), _ptr(w.conv_b), C,
                                           K, _ptr(u), tok_base, tokens, kind, _stream()), "recurrence_conv")
        z = torch.empty(tokens, B, 2 * (C // B), dtype=torch.float32, device=x.device)
        head_gemm(u.view(tokens, B, C // B), w.gates_by_block, z)
        _check(lib().ksana_recurrence_scan(*rows, _ptr(u), _ptr(z), _ptr(w.gates_b), _ptr(w.rate), C, K, B, _ptr(out),
                                           out.stride(0), seq_base, seqs, tok_base, kind, _stream()), "recurrence_scan")

    if x.dtype != torch.bfloat16:
        return general(0, meta.num_seqs, 0, T)
    if n_pre:
        cu = meta.cu_q_host
        max_q = int((cu[1:n_pre + 1] - cu[:n_pre]).max())
        scratch = torch.empty(lib().ksana_recurrence_scratch(pre_tokens, n_pre, max_q, C), dtype=torch.float32,
                              device=x.device)
        code = lib().ksana_recurrence_prompts(*rows, _ptr(meta.seq_of_token), *maps, 0, n_pre, 0, pre_tokens, max_q,
                                              _ptr(scratch), _stream())
        if code == -1:
            general(0, n_pre, 0, pre_tokens)
        else:
            _check(code, "recurrence_prompts")
    if n_dec:
        code = -1
        if meta.num_decode_tokens == n_dec:
            code = lib().ksana_recurrence_step(*rows, *maps, n_pre, n_dec, _stream())
        if code == -1:
            general(n_pre, n_dec, pre_tokens, T - pre_tokens)
        else:
            _check(code, "recurrence_step")
