"""ctypes wrappers of the kernels behind layers with mixers of their own sizes (csrc/cuda/mixer_elementwise.cu,
window_attention.cu, linear_attention.cu). bf16 and fp32 storage; everything is computed in 32-bit floats."""
from __future__ import annotations

from typing import Optional

import torch

from .cuda import _check, _ptr, _stream, lib

_KIND = {torch.float32: 0, torch.bfloat16: 1}


def _rows(x: torch.Tensor) -> torch.Tensor:
    """[rows, H] view with a contiguous last dimension."""
    x = x.reshape(-1, x.shape[-1])
    return x if x.stride(1) == 1 else x.contiguous()


def layer_norm(x, weight, bias, eps: float, residual: Optional[torch.Tensor] = None, out_dtype=None) -> torch.Tensor:
    x2 = _rows(x)
    out = torch.empty(x2.shape, dtype=out_dtype or x.dtype, device=x.device)
    r2 = residual.view(-1, x2.shape[1]) if residual is not None else None
    rk = _KIND[r2.dtype] if r2 is not None else (0 if x.dtype == torch.float32 else _KIND[out.dtype])
    kinds = _KIND[x.dtype] | rk << 1 | _KIND[weight.dtype] << 2 | _KIND[out.dtype] << 3
    if bias is not None:
        bias = bias.to(weight.dtype)
    _check(lib().ksana_layer_norm(_ptr(x2), x2.stride(0), _ptr(r2), r2.stride(0) if r2 is not None else 0, _ptr(weight),
                                  _ptr(bias), _ptr(out), out.stride(0), x2.shape[0], x2.shape[1], float(eps), kinds,
                                  _stream()), "layer_norm")
    return out.view(x.shape)


def stream_norm(x, weight, eps: float, center: bool, stream_in, stream_out=None, out_dtype=None, add_rows=None,
                add_vec=None, routed=None) -> torch.Tensor:
    T, H = stream_in.shape
    out = torch.empty(T, H, dtype=out_dtype or stream_in.dtype, device=stream_in.device)
    y, pos, wts = routed if routed is not None else (None, None, None)
    assert stream_in.is_contiguous() and (stream_out is None or stream_out.is_contiguous())
    assert all(t is None or t.is_contiguous() for t in (add_rows, add_vec, y, pos, wts))
    xk = x if x is not None else y
    kinds = (_KIND[xk.dtype] if xk is not None else 0) | _KIND[stream_in.dtype] << 1 | _KIND[weight.dtype] << 2 | \
        _KIND[out.dtype] << 3
    assert x is None or x.stride(1) == 1
    _check(lib().ksana_stream_norm(_ptr(x), x.stride(0) if x is not None else 0, _ptr(stream_in), _ptr(stream_out), H,
                                   _ptr(weight), None, _ptr(out), H, T, H, float(eps), kinds, int(center),
                                   _ptr(add_rows), _ptr(add_vec), _ptr(y), _ptr(pos), _ptr(wts),
                                   wts.shape[1] if wts is not None else 0, _stream()), "stream_norm")
    return out


def hyper_norm(x, scale, routed, streams, mix, out_w, streams_out, in_w, weight, eps: float, out_dtype) -> torch.Tensor:
    S, H = in_w.shape[0], weight.shape[0]
    T = streams.shape[0]
    rows, pos, wts = routed if routed is not None else (None, None, None)
    assert streams.is_contiguous() and streams.dtype == torch.float32 and weight.dtype == out_dtype
    assert x is None or x.stride(1) == 1 and x.dtype == out_dtype
    assert all(t is None or t.is_contiguous() for t in (scale, rows, pos, wts, mix, out_w, streams_out, in_w))
    out = torch.empty(T, H, dtype=out_dtype, device=streams.device)
    _check(lib().ksana_hyper_norm(_ptr(x), x.stride(0) if x is not None else 0, _ptr(scale), _ptr(rows), _ptr(pos),
                                  _ptr(wts), wts.shape[1] if wts is not None else 0, _ptr(streams),
                                  int(streams.dim() == 2), _ptr(mix), _ptr(out_w), _ptr(streams_out), _ptr(in_w),
                                  _ptr(weight), _ptr(out), T, H, S, float(eps), _KIND[out_dtype], _stream()),
           "hyper_norm")
    return out


def relu2(x: torch.Tensor) -> torch.Tensor:
    x2 = _rows(x)
    out = torch.empty(x2.shape, dtype=x.dtype, device=x.device)
    _check(lib().ksana_relu2(_ptr(x2), x2.stride(0), _ptr(out), x2.shape[0], x2.shape[1], _KIND[x.dtype], _stream()),
           "relu2")
    return out.view(x.shape)


def gated_stream_norm(x, x_gate, routed, y, y_scale, y_gate, scale: float, stream_in, stream_out, weights, eps: float,
                      out_dtype) -> torch.Tensor:
    T, H = stream_in.shape
    out = torch.empty(len(weights), T, H, dtype=out_dtype, device=stream_in.device)
    rows, pos, wts = routed if routed is not None else (None, None, None)
    assert stream_in.is_contiguous() and (stream_out is None or stream_out.is_contiguous()) and len(weights) in (1, 2)
    assert all(t is None or t.is_contiguous() for t in (rows, pos, wts))
    assert all(t is None or t.stride(1) == 1 and t.dtype == out_dtype for t in (x, x_gate, y, y_gate))
    assert all(w.dtype == out_dtype and w.is_contiguous() for w in weights)

    def ld(t):
        return t.stride(0) if t is not None else 0
    _check(lib().ksana_gated_stream_norm(
        _ptr(x), ld(x), _ptr(x_gate), ld(x_gate), _ptr(rows), _ptr(pos), _ptr(wts), wts.shape[1] if wts is not None else 0,
        _ptr(y), ld(y), _ptr(y_scale), ld(y_scale), _ptr(y_gate), ld(y_gate), float(scale), _ptr(stream_in),
        _ptr(stream_out), _ptr(weights[0]), _ptr(weights[1]) if len(weights) > 1 else None, _ptr(out), T, H, float(eps),
        _KIND[out_dtype], _stream()), "gated_stream_norm")
    return out


def clamped_gate_mul(x: torch.Tensor, limit: float, alpha: float) -> torch.Tensor:
    T, two_i = x.shape
    assert x.is_contiguous()
    out = torch.empty(T, two_i // 2, dtype=x.dtype, device=x.device)
    _check(lib().ksana_clamped_gate_mul(_ptr(x), _ptr(out), T, two_i // 2, float(limit), float(alpha), _KIND[x.dtype],
                                        _stream()), "clamped_gate_mul")
    return out


def embedding(ids, table, scale: float, out_dtype, positions=None, pos_table=None) -> torch.Tensor:
    assert out_dtype == torch.float32 and table.is_contiguous()
    assert pos_table is None or pos_table.is_contiguous() and pos_table.dtype == table.dtype
    T, H = ids.numel(), table.shape[1]
    out = torch.empty(T, H, dtype=torch.float32, device=table.device)
    _check(lib().ksana_embedding_f32(_ptr(ids), _ptr(table), _ptr(out), T, H, table.shape[0], float(scale),
                                     _ptr(positions) if pos_table is not None else None, _ptr(pos_table),
                                     pos_table.shape[0] if pos_table is not None else 0, _KIND[table.dtype],
                                     _stream()), "embedding_f32")
    return out


def gelu_and_mul(x: torch.Tensor) -> torch.Tensor:
    T, two_i = x.shape
    out = torch.empty(T, two_i // 2, dtype=x.dtype, device=x.device)
    _check(lib().ksana_gelu_mul(_ptr(x), x.stride(0), _ptr(out), out.stride(0), T, two_i // 2, _KIND[x.dtype],
                                _stream()), "gelu_mul")
    return out


def append_act(k, u, slot_mapping, cache, block_size: int, out, gated: bool = False) -> None:
    """k and u are column slices of one matrix (or one of them is None)."""
    T = (k if k is not None else u).shape[0]
    hk, d = (k.shape[1], k.shape[2]) if k is not None else (0, 8)
    ld = u.stride(0) if u is not None else k.stride(0)
    dt = k.dtype if k is not None else u.dtype
    if k is not None:
        _packed_heads(k)
        assert cache.is_contiguous() and cache.dtype == dt
    if u is not None:
        assert u.stride(1) == 1 and (T == 1 or k is None or k.stride(0) == ld)
        assert out.stride(1) == 1 and out.dtype == dt
    cols = 0 if u is None else u.shape[1] // 2 if gated else u.shape[1]
    _check(lib().ksana_append_act(_ptr(k), _ptr(u), ld, _ptr(slot_mapping), _ptr(cache), T, hk, d, block_size, _ptr(out),
                                  out.stride(0) if u is not None else 0, cols, int(gated), _KIND[dt], _stream()),
           "append_act")


def gelu(x: torch.Tensor) -> torch.Tensor:
    x2 = _rows(x)
    out = torch.empty(x2.shape, dtype=x.dtype, device=x.device)
    append_act(None, x2, None, None, 1, out)
    return out.view(x.shape)


def _packed_heads(x: torch.Tensor) -> torch.Tensor:
    assert x.stride(2) == 1 and (x.shape[1] == 1 or x.stride(1) == x.shape[2])
    return x


def qk_norm_cache(q, k, v, slot_mapping, cache, block_size: int, q_norm, k_norm, eps: float, positions=None,
                  rotary=None, norm_all: bool = False, halves: bool = False) -> None:
    T, h, d = q.shape
    if norm_all or halves:
        assert norm_all and halves and k is not None and q_norm is not None
    hk, dv = (v.shape[1], v.shape[2]) if v is not None else (0, 0)
    for x in (q, k, v):
        if x is not None:
            _packed_heads(x)
    assert cache.dtype == q.dtype and cache.is_contiguous()
    fn = lib().ksana_qk_row_norm_cache if norm_all else lib().ksana_qk_norm_cache
    _check(fn(_ptr(q), q.stride(0), _ptr(k), k.stride(0) if k is not None else 0, _ptr(v),
              v.stride(0) if v is not None else 0, _ptr(slot_mapping), _ptr(cache), _ptr(q_norm), _ptr(k_norm), float(eps),
              _ptr(positions) if rotary is not None else None, _ptr(rotary),
              rotary.shape[1] if rotary is not None else 0, T, h, hk, d, dv, block_size, _KIND[q.dtype], _stream()),
           "qk_norm_cache")


def window_attention(q, cache, meta, block_size: int, kv_heads: int, vdim: int, scale: float, window: int, bias,
                     out_scale: float, out: torch.Tensor, keep_first: int = 0, softcap: float = 0.0, sink: bool = False,
                     gate=None) -> None:
    """bf16 prompts take the tensor-core kernel, bf16 single tokens the cache-streaming one; sizes those do not have,
    and fp32, take the general kernel."""
    T, h, d = q.shape
    _packed_heads(q)
    assert out.stride(1) == 1
    n_pre, n_dec, pre_tokens = meta.num_prefill, meta.num_decode, meta.num_prefill_tokens
    blen = bias.shape[1] if bias is not None else 0
    shared = int(cache.shape[1] == kv_heads * block_size * d)
    sizes = (h, kv_heads, d, vdim, block_size, window, keep_first, shared, float(scale), _ptr(bias), blen,
             float(out_scale), float(softcap), int(sink), _ptr(gate), gate.stride(0) if gate is not None else 0)
    assert gate is None or gate.dtype == q.dtype and gate.stride(1) == 1

    def general(first: int, count: int) -> None:
        if count:
            _check(lib().ksana_window_attention_any(
                _ptr(q), q.stride(0), _ptr(cache), _ptr(meta.block_tables), meta.max_blocks, _ptr(meta.cu_q),
                _ptr(meta.kv_lens), _ptr(meta.seq_of_token), *sizes, _ptr(out), out.stride(0), first, count,
                _KIND[q.dtype], _stream()), "window_attention_any")

    if q.dtype != torch.bfloat16:
        return general(0, T)
    cu = meta.cu_q_host
    if n_pre:
        max_q = int((cu[1:n_pre + 1] - cu[:n_pre]).max())
        code = lib().ksana_window_prefill(_ptr(q), q.stride(0), T, _ptr(cache), cache.shape[0], _ptr(meta.block_tables),
                                          meta.max_blocks, _ptr(meta.cu_q), _ptr(meta.kv_lens), *sizes, _ptr(out),
                                          out.stride(0), 0, n_pre, max_q, _stream())
        if code == -1:
            general(0, pre_tokens)
        else:
            _check(code, "window_prefill")
    if n_dec:
        code = -1
        if meta.num_decode_tokens == n_dec:
            code = lib().ksana_window_decode(_ptr(q), q.stride(0), _ptr(cache), cache.shape[0], _ptr(meta.block_tables),
                                             meta.max_blocks, _ptr(meta.cu_q), _ptr(meta.kv_lens), *sizes, _ptr(out), out.stride(0),
                                             n_pre, n_dec, int(meta.kv_lens_host[n_pre:].max()), _stream())
        if code == -1:
            general(pre_tokens, T - pre_tokens)
        else:
            _check(code, "window_decode")


# Prompt portions of more tokens than this go through the chunked form of linear attention.
LINEAR_CHUNK_MIN_TOKENS = 16


def long_portions(meta) -> int:
    """How many leading prompt portions of the step go through the chunked form (a step lists them longest first; a
    shorter one ahead of a longer one goes along)."""
    n_pre = meta.num_prefill
    lens = meta.cu_q_host[1:n_pre + 1] - meta.cu_q_host[:n_pre]
    above = (lens > LINEAR_CHUNK_MIN_TOKENS).nonzero()[0]
    return int(above[-1]) + 1 if len(above) else 0


def linear_attention(q, k, v, state, meta, decay, act: str, rotary, key_scale: float) -> torch.Tensor:
    T, h, d = q.shape
    dv = v.shape[2]
    for x in (q, k, v):
        _packed_heads(x)
    out = torch.empty(T, h, dv, dtype=q.dtype, device=q.device)
    rd = rotary.shape[1] if rotary is not None else 0
    n_pre, n_dec = meta.num_prefill, meta.num_decode
    head = (_ptr(q), q.stride(0), _ptr(k), k.stride(0), _ptr(v), v.stride(0), _ptr(state), _ptr(meta.state_slots),
            _ptr(meta.cu_q), _ptr(meta.kv_lens), _ptr(meta.positions), _ptr(decay), _ptr(rotary), rd,
            1 if act == "silu" else 0, float(key_scale), h, d, dv, _ptr(out))
    n_long = long_portions(meta) if q.dtype == torch.bfloat16 else 0
    if n_long:
        cu = meta.cu_q_host
        scratch = torch.empty(lib().ksana_linear_chunk_scratch(int(cu[n_long]), n_long, h, d, dv), dtype=torch.float32,
                              device=q.device)
        code = lib().ksana_linear_chunked(*head, 0, n_long, int((cu[1:n_long + 1] - cu[:n_long]).max()), _ptr(scratch),
                                          _stream())
        if code == -1:
            n_long = 0
        else:
            _check(code, "linear_chunked")
    one = n_dec > 0 and meta.num_decode_tokens == n_dec
    for base, count, single in ((n_long, n_pre - n_long, 0), (n_pre, n_dec, 1 if one else 0)):
        if count:
            _check(lib().ksana_linear_recurrent(*head, base, count, single, _KIND[q.dtype], _stream()),
                   "linear_recurrent")
    return out


def gated_norm(o, g, weight, eps: float, gate: str, out_scale: float, out: torch.Tensor, per_head: bool = False) -> None:
    T, h, dv = o.shape
    assert o.is_contiguous() and g.stride(1) == 1 and out.stride(1) == 1
    _check(lib().ksana_gated_norm(_ptr(o), _ptr(g), g.stride(0), _ptr(weight), _ptr(out), out.stride(0), T, h, dv,
                                  float(eps), 1 if gate == "sigmoid" else 0, float(out_scale), int(per_head),
                                  _KIND[o.dtype], _stream()), "gated_norm")


def softcap(logits: torch.Tensor, cap: float) -> torch.Tensor:
    rows, n = logits.shape
    x = logits.float()
    if x.stride(1) != 1:
        x = x.contiguous()
    out = torch.empty(rows, n, dtype=torch.float32, device=x.device)
    _check(lib().ksana_softcap(_ptr(x), x.stride(0), _ptr(out), rows, n, float(cap), _stream()), "softcap")
    return out
