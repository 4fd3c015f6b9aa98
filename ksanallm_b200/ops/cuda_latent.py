"""Latent attention over pages of 16 tokens (csrc/cuda/latent_attention.cu, window_attention.cu, gemm_batched.cu)."""
from __future__ import annotations

import torch

from .cuda import _check, _ptr, _stream, gemm_bf16, lib
from .cuda_mixer import _KIND


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


# Keys and values that prompts have written out at a time: more contexts than this go in several rounds.
EXPAND_BYTES = 1 << 30


def _prompts(q, cache, meta, block_size: int, w, scale: float, gate, out) -> bool:
    """The step's prompt portions over keys and values written out per head. False: sizes the kernel does not take."""
    T, h, qd = q.shape
    rank, dim, vdim = w.rank, w.dim, w.vdim
    rot, width = qd - dim, rank + qd - dim
    if q.dtype != torch.bfloat16 or (rank | rot | dim | vdim) % 8 or dim > 128 or vdim > 128 or rot > 64:
        return False
    n_pre, cu, kl = meta.num_prefill, meta.cu_q_host, meta.kv_lens_host
    per_row = 2 * h * (dim + vdim)
    lo = 0
    while lo < n_pre:
        hi, rows = lo, 0
        while hi < n_pre and (hi == lo or (rows + int(kl[hi])) * per_row <= EXPAND_BYTES):
            rows += int(kl[hi])
            hi += 1
        lat = torch.empty(rows, width, dtype=q.dtype, device=q.device)
        _check(lib().ksana_latent_gather(_ptr(cache), _ptr(meta.block_tables), meta.max_blocks, _ptr(meta.kv_lens), lo,
                                         hi - lo, int(kl[lo:hi].max()), block_size, width, _ptr(lat), _stream()),
               "latent_gather")
        kv = gemm_bf16(lat[:, :rank], w.expand)
        code = lib().ksana_latent_prefill(
            _ptr(q), q.stride(0), T, _ptr(kv), kv.stride(0), lat.data_ptr() + 2 * rank, width, rows, _ptr(meta.cu_q),
            _ptr(meta.kv_lens), h, dim, rot, vdim, float(scale), _ptr(gate), gate.stride(0) if gate is not None else 0,
            _ptr(out), out.stride(0), lo, hi - lo, int((cu[lo + 1:hi + 1] - cu[lo:hi]).max()), _stream())
        if code == -1:
            return False
        _check(code, "latent_prefill")
        lo = hi
    return True


def latent_attention(q, a, norm_w, eps: float, rotary, cache, meta, block_size: int, w, scale: float, gate,
                     out: torch.Tensor) -> None:
    """See ``reference.latent_append`` and ``reference.latent_attention``. bf16 prompts attend to keys and values that are
    written out of the latents per head; single tokens, fp32 and other sizes to the latents themselves."""
    T, h, qd = q.shape
    rank, dim, vdim = w.rank, w.dim, w.vdim
    rot = qd - dim
    assert q.stride(2) == 1 and q.stride(1) == qd and a.stride(1) == 1 and out.stride(1) == 1 and cache.is_contiguous()
    n_pre, n_dec = meta.num_prefill, meta.num_decode
    first = meta.num_prefill_tokens if q.dtype == torch.bfloat16 and n_pre else 0  # tokens from here on: absorbed queries
    q_cat = torch.empty(T - first, h, rank + rot, dtype=q.dtype, device=q.device)
    _check(lib().ksana_latent_append(_ptr(q), q.stride(0), dim, _ptr(q_cat), first, _ptr(a), a.stride(0), _ptr(norm_w),
                                     float(eps), _ptr(meta.positions), _ptr(rotary), _ptr(meta.slot_mapping),
                                     _ptr(cache), T, h, rank, rot, _KIND[q.dtype], _stream()), "latent_append")
    if first and not _prompts(q, cache, meta, block_size, w, scale, gate, out):
        q_cat = torch.empty(T, h, rank + rot, dtype=q.dtype, device=q.device)
        q_cat[..., rank:] = q[..., dim:]
        first = 0
    if first == T:
        return
    head_gemm(q[first:, :, :dim], w.uk_t, q_cat[..., :rank])
    o = torch.empty(T - first, h * rank, dtype=q.dtype, device=q.device)
    # the kernels index tokens of the whole step
    at = [x.data_ptr() - first * x.stride(0) * x.element_size() for x in (q_cat, o)]
    gates = (_ptr(gate), gate.stride(0) if gate is not None else 0)
    code = -1
    if q.dtype == torch.bfloat16 and first == meta.num_prefill_tokens:  # only the sequences behind the prompts
        cu = meta.cu_q_host[n_pre:]
        code = lib().ksana_latent_decode(
            at[0], q_cat.stride(0), T, _ptr(cache), cache.shape[0], _ptr(meta.block_tables), meta.max_blocks,
            _ptr(meta.cu_q), _ptr(meta.kv_lens), h, rank, rot, block_size, float(scale), *gates, at[1], o.stride(0), n_pre,
            n_dec, int((cu[1:] - cu[:-1]).max()), int(meta.kv_lens_host[n_pre:].max()), _stream())
    if code == -1:
        code = lib().ksana_window_attention_any(
            at[0], q_cat.stride(0), _ptr(cache), _ptr(meta.block_tables), meta.max_blocks, _ptr(meta.cu_q),
            _ptr(meta.kv_lens), _ptr(meta.seq_of_token), h, 1, rank + rot, rank, block_size, 0, 0, 1, float(scale), None, 0,
            1.0, 0.0, 0, *gates, at[1], o.stride(0), first, T - first, _KIND[q.dtype], _stream())
    _check(code, "latent_attention")
    head_gemm(o.view(T - first, h, rank), w.uv, out[first:].unflatten(1, (h, vdim)))
