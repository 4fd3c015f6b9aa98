"""Gated linear recurrence behind a short convolution (csrc/cuda/gated_recurrence.cu)."""
from __future__ import annotations

import torch

from .cuda import _check, _ptr, _stream, lib
from .cuda_latent import head_gemm
from .cuda_mixer import _KIND


def gated_recurrence(y, x, state, meta, w, out: torch.Tensor) -> None:
    """See ``reference.gated_recurrence``; ``w``: :class:`~ksanallm_b200.models.mixers.RecurrenceWeights`."""
    T, C = x.shape
    K, B = w.conv.shape[1], w.gates.shape[1]
    kind = _KIND[x.dtype]
    assert x.stride(1) == y.stride(1) == out.stride(1) == 1 and state.is_contiguous()
    u = torch.empty(T, C, dtype=x.dtype, device=x.device)
    _check(lib().ksana_recurrence_conv(_ptr(x), x.stride(0), _ptr(state), _ptr(meta.state_slots), _ptr(meta.cu_q),
                                       _ptr(meta.kv_lens), _ptr(meta.seq_of_token), _ptr(w.conv), _ptr(w.conv_b), C, K,
                                       _ptr(u), 0, T, kind, _stream()), "recurrence_conv")
    z = torch.empty(T, B, 2 * (C // B), dtype=torch.float32, device=x.device)
    head_gemm(u.view(T, B, C // B), w.gates_by_block, z)
    _check(lib().ksana_recurrence_scan(_ptr(y), y.stride(0), _ptr(x), x.stride(0), _ptr(state), _ptr(meta.state_slots),
                                       _ptr(meta.cu_q), _ptr(meta.kv_lens), _ptr(u), _ptr(z), _ptr(w.gates_b),
                                       _ptr(w.rate), C, K, B, _ptr(out), out.stride(0), 0, meta.num_seqs, 0, kind,
                                       _stream()), "recurrence_scan")
