"""Attention whose softmax weights are mixed across heads (csrc/cuda/talking_attention.cu, talking_prefill.cu,
talking_decode.cu)."""
from __future__ import annotations

import ctypes

import torch

from .cuda import _check, _ptr, _stream, lib
from .cuda_mixer import _KIND, _packed_heads


def talking_attention(q, cache, meta, block_size: int, kv_heads: int, vdim: int, scale: float, sink, talk,
                      out_scale: float, out: torch.Tensor, gate=None) -> None:
    """See ``reference.talking_attention``. bf16 prompts take the tensor-core kernels, bf16 single tokens the two streams over
    the cache; sizes those do not have, and fp32, take the general kernel."""
    T, h, d = q.shape
    _packed_heads(q)
    assert out.stride(1) == 1 and sink.dtype == talk.dtype == torch.float32 and talk.is_contiguous()
    assert gate is None or gate.dtype == q.dtype and gate.stride(1) == 1
    sizes = (h, kv_heads, d, vdim, block_size, float(scale), _ptr(sink), _ptr(talk), float(out_scale), _ptr(gate),
             gate.stride(0) if gate is not None else 0)
    tables = (_ptr(meta.block_tables), meta.max_blocks, _ptr(meta.cu_q), _ptr(meta.kv_lens))

    def general(first: int, count: int) -> None:
        if count:
            _check(lib().ksana_talking_any(_ptr(q), q.stride(0), _ptr(cache), *tables, _ptr(meta.seq_of_token), *sizes,
                                           _ptr(out), out.stride(0), first, count, _KIND[q.dtype], _stream()), "talking_any")

    if q.dtype != torch.bfloat16:
        return general(0, T)
    n_pre, n_dec, pre_tokens = meta.num_prefill, meta.num_decode, meta.num_prefill_tokens
    cu, kl = meta.cu_q_host, meta.kv_lens_host
    if n_pre:
        n = lib().ksana_talking_prefill_bytes(h, n_pre, cu.ctypes.data, kl.ctypes.data)
        scratch = torch.empty(n, dtype=torch.uint8, device=q.device)
        launches = ctypes.c_int()
        code = lib().ksana_talking_prefill(
            _ptr(q), q.stride(0), T, _ptr(cache), cache.shape[0], *tables, *sizes, _ptr(out), out.stride(0), n_pre,
            cu.ctypes.data, kl.ctypes.data, _ptr(scratch), n, ctypes.byref(launches), _stream())
        if code == -1:
            general(0, pre_tokens)
        else:
            _check(code, "talking_prefill")
    if n_dec:
        code = -1
        if meta.num_decode_tokens == n_dec:
            top = int(kl[n_pre:].max())
            n = lib().ksana_talking_decode_bytes(h, n_dec, top)
            scratch = torch.empty(n, dtype=torch.uint8, device=q.device)
            code = lib().ksana_talking_decode(_ptr(q), q.stride(0), _ptr(cache), cache.shape[0], *tables, *sizes, _ptr(out),
                                              out.stride(0), n_pre, n_dec, top, _ptr(scratch), n, _stream())
        if code == -1:
            general(pre_tokens, T - pre_tokens)
        else:
            _check(code, "talking_decode")
