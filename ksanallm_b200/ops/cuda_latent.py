"""Latent attention over pages of 16 tokens (csrc/cuda/latent_attention.cu, window_attention.cu, gemm_batched.cu)."""
from __future__ import annotations

import torch

from .cuda import _check, _ptr, _stream, lib
from .cuda_mixer import _KIND, window_attention


def head_gemm(a: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """out[t, b, :] = a[t, b, :] @ w[b]^T for views a [T, B, K], out [T, B, N] with contiguous last dimensions, w [B, N, K]
    contiguous; bf16 (out may be fp32) or all fp32. Sizes the tensor-core kernel takes go there."""
    T, B, K = a.shape
    N = w.shape[1]
    args = (_ptr(a), a.stride(0), a.stride(1), _ptr(w), _ptr(out), out.stride(0), out.stride(1), T, B, N, K)
    code = -1
    if out.dtype == torch.bfloat16:
        code = lib().ksana_gemm_bf16_batched(*args, _stream())
    if code == -1:
        kind = 0 if a.dtype == torch.float32 else 1 if out.dtype == torch.bfloat16 else 2
        code = lib().ksana_head_gemm_any(*args, kind, _stream())
    _check(code, "head_gemm")
    return out


def latent_attention(q, a, norm_w, eps: float, rotary, cache, meta, block_size: int, w, scale: float, gate,
                     out: torch.Tensor) -> None:
    """See ``reference.latent_append`` and ``reference.latent_attention``."""
    T, h, qd = q.shape
    rank, dim, vdim = w.rank, w.dim, w.vdim
    rot = qd - dim
    assert q.stride(2) == 1 and q.stride(1) == qd and a.stride(1) == 1 and out.stride(1) == 1 and cache.is_contiguous()
    q_cat = torch.empty(T, h, rank + rot, dtype=q.dtype, device=q.device)
    _check(lib().ksana_latent_append(_ptr(q), q.stride(0), dim, _ptr(q_cat), 0, _ptr(a), a.stride(0), _ptr(norm_w),
                                     float(eps), _ptr(meta.positions), _ptr(rotary), _ptr(meta.slot_mapping),
                                     _ptr(cache), T, h, rank, rot, _KIND[q.dtype], _stream()), "latent_append")
    head_gemm(q[..., :dim], w.uk_t, q_cat[..., :rank])
    o = torch.empty(T, h * rank, dtype=q.dtype, device=q.device)
    _check(lib().ksana_window_attention_any(
        _ptr(q_cat), q_cat.stride(0), _ptr(cache), _ptr(meta.block_tables), meta.max_blocks, _ptr(meta.cu_q),
        _ptr(meta.kv_lens), _ptr(meta.seq_of_token), h, 1, rank + rot, rank, block_size, 0, 0, 1, float(scale), None, 0,
        1.0, 0.0, 0, _ptr(gate), gate.stride(0) if gate is not None else 0, _ptr(o), o.stride(0), 0, T, _KIND[q.dtype],
        _stream()), "latent_attention_any")
    head_gemm(o.view(T, h, rank), w.uv, out.unflatten(1, (h, vdim)))
