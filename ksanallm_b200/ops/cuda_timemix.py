"""Time mixing with token-dependent decays (csrc/cuda/time_mix.cu)."""
from __future__ import annotations

import torch

from .cuda import _check, _ptr, _stream, lib
from .cuda_mixer import _KIND, long_portions


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
    """See ``reference.time_mix``; ``state`` [slots, 1, 1, n] starts with the heads' states. Long bf16 portions of prompts go
    through chunks on the tensor cores, everything else token by token."""
    T, (h, d) = r.shape[0], u.shape
    assert r.stride(1) == k.stride(1) == v.stride(1) == z.stride(1) == 1 and z.dtype == torch.float32
    assert state.is_contiguous()
    out = torch.empty(T, h, d, dtype=r.dtype, device=r.device)
    n_pre, n_dec = meta.num_prefill, meta.num_decode
    head = (_ptr(r), r.stride(0), _ptr(k), k.stride(0), _ptr(v), v.stride(0), _ptr(z), z.stride(0), _ptr(w0), _ptr(u),
            _ptr(state), state.shape[-1], _ptr(meta.state_slots), _ptr(meta.cu_q), _ptr(meta.kv_lens), h, d, _ptr(out))
    n_long = long_portions(meta) if r.dtype == torch.bfloat16 else 0
    if n_long:
        cu = meta.cu_q_host
        scratch = torch.empty(lib().ksana_time_mix_scratch(int(cu[n_long]), n_long, h, d), dtype=torch.float32,
                              device=r.device)
        code = lib().ksana_time_mix_chunked(*head, 0, n_long, int((cu[1:n_long + 1] - cu[:n_long]).max()), _ptr(scratch),
                                            _stream())
        if code == -1:
            n_long = 0
        else:
            _check(code, "time_mix_chunked")
    one = n_dec > 0 and meta.num_decode_tokens == n_dec
    for base, count, single in ((n_long, n_pre - n_long, 0), (n_pre, n_dec, int(one))):
        if count:
            _check(lib().ksana_time_mix_recurrent(*head, base, count, single, _KIND[r.dtype], _stream()),
                   "time_mix_recurrent")
    return out
