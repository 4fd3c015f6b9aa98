"""Attention whose softmax weights are mixed across heads (csrc/cuda/talking_attention.cu)."""
from __future__ import annotations

import torch

from .cuda import _check, _ptr, _stream, lib
from .cuda_mixer import _KIND, _packed_heads


def talking_attention(q, cache, meta, block_size: int, kv_heads: int, vdim: int, scale: float, sink, talk,
                      out_scale: float, out: torch.Tensor, gate=None) -> None:
    """See ``reference.talking_attention``."""
    T, h, d = q.shape
    _packed_heads(q)
    assert out.stride(1) == 1 and sink.dtype == talk.dtype == torch.float32 and talk.is_contiguous()
    assert gate is None or gate.dtype == q.dtype and gate.stride(1) == 1
    sizes = (h, kv_heads, d, vdim, block_size, float(scale), _ptr(sink), _ptr(talk), float(out_scale), _ptr(gate),
             gate.stride(0) if gate is not None else 0)
    _check(lib().ksana_talking_any(
        _ptr(q), q.stride(0), _ptr(cache), _ptr(meta.block_tables), meta.max_blocks, _ptr(meta.cu_q), _ptr(meta.kv_lens),
        _ptr(meta.seq_of_token), *sizes, _ptr(out), out.stride(0), 0, T, _KIND[q.dtype], _stream()), "talking_any")
