"""Time mixing with token-dependent decays (csrc/cuda/time_mix.cu)."""
from __future__ import annotations

import torch

from .cuda import _check, _ptr, _stream, lib
from .cuda_mixer import _KIND


def token_mix(h, mu, state, meta) -> torch.Tensor:
    """See ``reference.token_mix``; ``state`` [slots, 1, 1, n], its last W numbers being the previous token's vector."""
    T, W = h.shape
    assert h.is_contiguous() and mu.is_contiguous() and state.is_contiguous()
    n = state.shape[-1]
    out = torch.empty(mu.shape[0], T, W, dtype=h.dtype, device=h.device)
    _check(lib().ksana_token_mix(_ptr(h), _ptr(mu), _ptr(state) + 4 * (n - W), n, state.shape[0], _ptr(meta.state_slots),
                                 _ptr(meta.cu_q), _ptr(meta.kv_lens), _ptr(meta.seq_of_token), _ptr(out), T, W, mu.shape[0],
                                 _KIND[h.dtype], _stream()), "token_mix")
    return out


def tanh_parts(x, dtype) -> torch.Tensor:
    T, n = x.shape
    x = x.contiguous()
    out = torch.empty(T, 2 * n if dtype == torch.bfloat16 else n, dtype=dtype, device=x.device)
    _check(lib().ksana_tanh_parts(_ptr(x), n, _ptr(out), T, _KIND[dtype], _stream()), "tanh_parts")
    return out


def time_mix(r, k, v, z, w0, u, state, meta) -> torch.Tensor:
    """See ``reference.time_mix``; ``state`` [slots, 1, 1, n] starts with the heads' states."""
    T, (h, d) = r.shape[0], u.shape
    assert r.stride(1) == k.stride(1) == v.stride(1) == z.stride(1) == 1 and z.dtype == torch.float32
    assert state.is_contiguous()
    out = torch.empty(T, h, d, dtype=r.dtype, device=r.device)
    n_pre, n_dec = meta.num_prefill, meta.num_decode
    head = (_ptr(r), r.stride(0), _ptr(k), k.stride(0), _ptr(v), v.stride(0), _ptr(z), z.stride(0), _ptr(w0), _ptr(u),
            _ptr(state), state.shape[-1], _ptr(meta.state_slots), _ptr(meta.cu_q), _ptr(meta.kv_lens), h, d, _ptr(out))
    one = n_dec > 0 and meta.num_decode_tokens == n_dec
    for base, count, single in ((0, n_pre, 0), (n_pre, n_dec, int(one))):
        if count:
            _check(lib().ksana_time_mix_recurrent(*head, base, count, single, _KIND[r.dtype], _stream()),
                   "time_mix_recurrent")
    return out
