"""Binding of the native dense-layer executor (csrc/cuda/dense_executor.cu): the whole decoder stack of a step is
launched by one C call instead of ~8 Python-level kernel wrappers per layer.

Eligible models: dense (no MoE / MLA) RMSNorm + RoPE decoders with a gated SiLU FFN, bf16 weights or 128 x 128
block-scaled e4m3 weights (all four linears of every layer alike), head_dim 128 and the 16-token KV block, on one GPU or tensor-parallel with the single-kernel fused GEMM + reduce-scatter path. Anything
else keeps the Python layer code in models/transformer.py (same kernels, launched one by one).
"""
from __future__ import annotations

import ctypes
import os
from typing import List, Optional

import numpy as np
import torch

from ..ops import cuda as kcuda
from ..ops import cuda_latent

P, I, F, LL = ctypes.c_void_p, ctypes.c_int, ctypes.c_float, ctypes.c_longlong


class _Layer(ctypes.Structure):
    _fields_ = [(n, P) for n in ("wqkv", "bqkv", "wo", "ln2", "wgu", "wdown", "next_ln", "q_norm", "k_norm",
                                 "kv_cache", "sqkv", "so", "sgu", "sdown", "fqkv", "fo", "fgu", "fdown", "wgu_il")]


class _Model(ctypes.Structure):
    _fields_ = [("hidden", I), ("heads", I), ("kv_heads", I), ("head_dim", I), ("inter", I), ("n_layers", I),
                ("eps", F), ("rotary_dim", I), ("rope_interleaved", I), ("block_size", I), ("num_blocks", I),
                ("kv_kind", I), ("attn_scale", F), ("k_scale", F), ("v_scale", F), ("rope_cache", P),
                ("rank", I), ("ws", I), ("rows_cap", I), ("comm_ctas", I), ("recv", P), ("hbuf", P), ("sig", P),
                ("hbuf_mc", P), ("partial", P), ("partial_mc", P), ("two_kernel_max_tokens", I), ("ll_recv", P), ("ll_recv2", P),
                ("ll_recv2_mc", P), ("ll_half_words", LL), ("ll_rows_cap", I), ("ll_max_tokens", I),
                ("ll_one_shot", I), ("qkv_buf", P), ("attn_buf", P), ("gu_buf", P), ("act_buf", P), ("proj_buf", P),
                ("h_buf", P * 2), ("gemm_ws", P), ("gemm_ws_floats", LL), ("gemm_counters", P), ("n_counters", I),
                ("attn_ws", P), ("attn_ws_floats", LL), ("sig_words", I), ("a8_buf", P), ("sa_buf", P), ("a8_cols", I),
                ("fp8_pow2", I), ("mx_min_rows", I), ("layers", P)]


class _Step(ctypes.Structure):
    _fields_ = [("positions", P), ("slot_mapping", P), ("block_tables", P), ("cu_q", P), ("kv_lens", P),
                ("total_tokens", I), ("num_prefill", I), ("num_decode", I), ("max_blocks", I), ("max_q_prefill", I),
                ("max_q_decode", I), ("max_kv_decode", I), ("split_seq", I), ("split_row", I), ("num_prefill_b", I),
                ("num_decode_b", I), ("max_q_prefill_b", I), ("max_q_decode_b", I), ("max_kv_decode_b", I)]


def _p(t: Optional[torch.Tensor]):
    return None if t is None else t.data_ptr()


class DenseExecutor:
    @staticmethod
    def eligible(model) -> bool:
        cfg, tp = model.cfg, model.tp
        if os.environ.get("KSANA_DISABLE_NATIVE_EXECUTOR", "0") == "1" or os.environ.get("KSANA_LIBRARY_BASELINE") == "1":
            return False
        if model.device.type != "cuda" or model.dtype != torch.bfloat16 or not model.layers or model.norm_w is None:
            return False
        if getattr(model, "num_cache_layers", len(model.layers)) != len(model.layers):
            return False  # cross-layer KV sharing
        if (cfg.use_mla or cfg.norm_type != "rmsnorm" or cfg.residual_scale != 1.0 or cfg.head_dim != 128 or
                cfg.position_encoding not in ("rope", "none") or not cfg.gated_mlp or
                cfg.hidden_act not in ("silu", "swish") or cfg.sliding_window or
                cfg.qk_norm_after_rope or cfg.qk_l2_norm or cfg.cla_share_factor or cfg.rope_layers or cfg.attn_temperature_tuning):
            return False
        for layer in model.layers:
            if layer.is_moe or not hasattr(layer.attn, "qkv"):
                return False
            lins = (layer.attn.qkv, layer.attn.o_proj, layer.ffn.up, layer.ffn.down)
            kind = model.layers[0].attn.qkv.kind
            if kind not in ("dense", "fp8_block") or any(l.kind != kind for l in lins):
                return False
            if layer.attn.o_proj.bias is not None:
                return False
            if kind == "fp8_block":
                if tp.size > 1 and (tp.fused is None or tp.fused.partial is None):
                    return False
                for l in lins:
                    w, sc = l.weight, l.scale_inv
                    if (w.shape[1] % 128 or w.shape[0] % 8 or not w.is_contiguous() or sc.dtype != torch.float32 or
                            not sc.is_contiguous() or tuple(sc.shape) != ((w.shape[0] + 127) // 128, w.shape[1] // 128)):
                        return False
            if layer.ffn.up.bias is not None or layer.ffn.down.bias is not None or layer.attn.alibi is not None:
                return False
            if layer.ln2 is None or getattr(layer, "ln2_b", None) is not None:
                return False
            if layer.attn.k_scale != 1.0 or layer.attn.v_scale != 1.0:
                return False  # per-layer fp8 KV scales: Python layer path
        if tp.size > 1:
            fc = tp.fused
            if fc is None or not fc.single_kernel or fc.hidden % 256 or fc.hidden > 9216 or fc.hidden != cfg.hidden_size:
                return False
        return True

    def __init__(self, model):
        self.model = model
        cfg, tp = model.cfg, model.tp
        self.tp = tp
        self.H = cfg.hidden_size
        a0 = model.layers[0].attn
        self.h, self.hk, self.d = a0.h, a0.hk, a0.d
        self.inter = model.layers[0].ffn.down.weight.shape[1]
        n = len(model.layers)
        self._layers = (_Layer * n)()
        # power-of-two scales only if every fp8 weight has them: the activation quantiser is chosen per model
        pow2 = all(getattr(l, "pow2", False) for layer in model.layers
                   for l in (layer.attn.qkv, layer.attn.o_proj, layer.ffn.up, layer.ffn.down))
        for i, layer in enumerate(model.layers):
            L = self._layers[i]
            nxt = model.layers[i + 1].ln1 if i + 1 < n else model.norm_w
            L.wqkv, L.bqkv = _p(layer.attn.qkv.weight), _p(layer.attn.qkv.bias)
            L.wo, L.ln2 = _p(layer.attn.o_proj.weight), _p(layer.ln2)
            L.wgu, L.wdown = _p(layer.ffn.up.weight), _p(layer.ffn.down.weight)
            L.next_ln = _p(nxt)
            L.q_norm, L.k_norm = _p(layer.attn.q_norm), _p(layer.attn.k_norm)
            L.kv_cache = None
            if layer.attn.qkv.kind == "fp8_block":
                L.sqkv, L.so = _p(layer.attn.qkv.scale_inv), _p(layer.attn.o_proj.scale_inv)
                L.sgu, L.sdown = _p(layer.ffn.up.scale_inv), _p(layer.ffn.down.scale_inv)
                if pow2:
                    L.fqkv, L.fo = _p(layer.attn.qkv.sfb()), _p(layer.attn.o_proj.sfb())
                    L.fgu, L.fdown = _p(layer.ffn.up.sfb()), _p(layer.ffn.down.sfb())
        self.fp8 = model.layers[0].attn.qkv.kind == "fp8_block"
        # KSANA_FUSED_SWIGLU=1: keep a second copy of every gate_up weight with gate / up rows interleaved in groups of
        # 16, so prefill-sized steps run SiLU-mul as the GEMM's epilogue (costs the memory of the gate_up weights again)
        self._wgu_il = []
        if os.environ.get("KSANA_FUSED_SWIGLU", "0") == "1" and not self.fp8 and self.inter % 16 == 0:
            for i, layer in enumerate(model.layers):
                w = layer.ffn.up.weight
                I_ = w.shape[0] // 2
                il = torch.stack((w[:I_].view(I_ // 16, 16, -1), w[I_:].view(I_ // 16, 16, -1)), 1).reshape(w.shape)
                self._wgu_il.append(il.contiguous())
                self._layers[i].wgu_il = self._wgu_il[-1].data_ptr()
        m = self._m = _Model()
        m.hidden, m.heads, m.kv_heads, m.head_dim, m.inter, m.n_layers = self.H, self.h, self.hk, self.d, self.inter, n
        m.eps = float(cfg.rms_norm_eps)
        m.rotary_dim = int(cfg.rotary_dim or cfg.head_dim)
        m.rope_interleaved = 1 if cfg.rope_interleaved else 0
        m.attn_scale = float(a0.scale)
        m.k_scale = m.v_scale = 1.0
        m.rope_cache = _p(model.rope_cache)
        m.rank, m.ws = tp.rank, tp.size
        if tp.size > 1:
            fc = tp.fused
            m.rows_cap, m.comm_ctas = fc.rows_cap, fc.comm_ctas
            m.recv = ctypes.cast(fc._recv_ptrs, P)
            m.hbuf = ctypes.cast(fc._hbuf_ptrs, P)
            m.sig = ctypes.cast(fc._sig_ptrs, P)
            m.hbuf_mc = fc.hbuf_mc or None
            m.partial = ctypes.cast(fc._partial_ptrs, P)
            m.partial_mc = fc.partial_mc or None
            m.two_kernel_max_tokens = fc.two_kernel_max_tokens
            m.sig_words = fc.sig_words
            m.ll_recv = ctypes.cast(fc._ll_recv_ptrs, P)
            m.ll_recv2 = ctypes.cast(fc._ll_recv2_ptrs, P)
            m.ll_recv2_mc = fc.ll_recv2_mc or None
            m.ll_half_words = fc.ll_half_words
            m.ll_rows_cap, m.ll_max_tokens, m.ll_one_shot = fc.ll_rows_cap, fc.ll_max_tokens, int(fc.ll_one_shot)
        ws = kcuda.workspace(model.device)
        self._ws = ws
        m.gemm_ws, m.gemm_ws_floats = _p(ws.gemm_ws), ws.gemm_ws.numel()
        m.gemm_counters, m.n_counters = _p(ws.gemm_counters), ws.gemm_counters.numel()
        m.attn_ws, m.attn_ws_floats = _p(ws.attn_ws), ws.attn_ws.numel()
        m.layers = ctypes.cast(self._layers, P)
        if self.fp8:
            from ..ops import cuda_fp8
            m.fp8_pow2, m.mx_min_rows = int(pow2), cuda_fp8.MXF8_MIN_ROWS
        self.cap = 0
        self.overlap_min_tokens = int(os.environ.get("KSANA_OVERLAP_MIN_TOKENS", "1024"))
        self._bufs: List[torch.Tensor] = []
        self._kv_key = None
        self._step = _Step()
        lib = kcuda.lib()
        lib.ksana_dense_forward.argtypes = [P, P, P, P, I, I, P, P, P, P, P]
        lib.ksana_dense_forward.restype = I
        self._fn = lib.ksana_dense_forward
        self._out = P()
        self._fail = I()
        self._launches = I()

    def _ensure(self, T: int) -> None:
        if T <= self.cap:
            return
        cap = (max(T, 1024) + 1023) // 1024 * 1024
        dev, bf = self.model.device, torch.bfloat16
        nqkv = (self.h + 2 * self.hk) * self.d
        mk = lambda cols: torch.empty(cap, cols, dtype=bf, device=dev)  # noqa: E731
        qkv, attn, gu, act = mk(nqkv), mk(self.h * self.d), mk(2 * self.inter), mk(self.inter)
        self._bufs = [qkv, attn, gu, act]
        m = self._m
        if self.fp8:
            cols = max(self.H, self.h * self.d, self.inter)
            a8 = torch.empty(cap, cols, dtype=torch.uint8, device=dev)
            sa = torch.empty(cap + 256, cols // 128, dtype=torch.float32, device=dev)
            self._bufs += [a8, sa]
            m.a8_buf, m.sa_buf, m.a8_cols = _p(a8), _p(sa), cols
        m.qkv_buf, m.attn_buf, m.gu_buf, m.act_buf = _p(qkv), _p(attn), _p(gu), _p(act)
        if self.tp.size == 1:
            proj, h0, h1 = mk(self.H), mk(self.H), mk(self.H)
            self._bufs += [proj, h0, h1]
            m.proj_buf = _p(proj)
            m.h_buf[0], m.h_buf[1] = _p(h0), _p(h1)
            self._h = (h0, h1)
        self.cap = cap

    def _bind_kv(self, kv_caches) -> None:
        # every layer's pointer is part of the key: a new cache (a second engine on the same model) may start at the
        # address the old one had while its other layers, or its block count, differ
        key = tuple(c.data_ptr() for c in kv_caches) + tuple(kv_caches[0].shape)
        if key == self._kv_key:
            return
        for i in range(len(self.model.layers)):
            self._layers[i].kv_cache = kv_caches[i].data_ptr()
        c = kv_caches[0]
        m = self._m
        m.num_blocks, m.block_size = c.shape[0], c.shape[3]
        m.kv_kind = 0 if c.dtype == torch.bfloat16 else 1
        self._kv_key = key

    def can_run(self, meta, kv_caches, n_layers: int) -> bool:
        T = meta.total_tokens
        if T == 0 or n_layers == 0 or kv_caches[0].dim() != 5 or kv_caches[0].shape[3] != 16:
            return False
        if getattr(meta, "mrope_positions", None) is not None:
            return False
        if kv_caches[0].dtype != torch.bfloat16 and meta.num_prefill:
            return False  # fp8 cache prefill chunks take the dequantising path
        if self.tp.size > 1:
            fc = self.tp.fused
            return T <= min(8192, fc.max_tokens)
        return True

    def _overlap_split(self, cu, n_seq: int, T: int) -> int:
        """Sequence index at which a prefill-sized tensor-parallel step is cut into two half-batches that run on two
        streams (the collectives of one half overlap the compute of the other); 0: run the step as one batch."""
        fc = self.tp.fused if self.tp.size > 1 else None
        if fc is None or n_seq < 2 or T < self.overlap_min_tokens or fc.partial is None:
            return 0
        split = int(np.abs(cu[1:n_seq] - T // 2).argmin()) + 1
        rows_a = int(cu[split])
        if min(rows_a, T - rows_a) < max(256, T // 4):
            return 0
        return split

    def forward(self, meta, kv_caches, h: torch.Tensor, residual: torch.Tensor, n_layers: int) -> torch.Tensor:
        """h: normalised input of layer 0, residual: the residual stream (both [T, H], contiguous); returns the
        normalised output of layer ``n_layers - 1`` (a view of an internal buffer, valid until the next call)."""
        T = meta.total_tokens
        self._ensure(T)
        self._bind_kv(kv_caches)
        s = self._step
        s.positions, s.slot_mapping = meta.positions.data_ptr(), meta.slot_mapping.data_ptr()
        s.block_tables, s.cu_q, s.kv_lens = meta.block_tables.data_ptr(), meta.cu_q.data_ptr(), meta.kv_lens.data_ptr()
        n_pre, n_dec = meta.num_prefill, meta.num_decode
        s.total_tokens, s.num_prefill, s.num_decode, s.max_blocks = T, n_pre, n_dec, meta.max_blocks
        cu, kl = meta.cu_q_host, meta.kv_lens_host

        def maxima(lo, hi):
            """(prefill count, decode count, max q prefill, max q decode, max kv decode) of sequences [lo, hi)."""
            p_hi = min(hi, n_pre)
            q = cu[lo + 1:hi + 1] - cu[lo:hi]
            n_p, n_d = max(p_hi - lo, 0), hi - max(lo, n_pre)
            mq_p = int(q[:n_p].max()) if n_p > 0 else 0
            mq_d = int(q[n_p:].max()) if n_d > 0 else 0
            mkv = int(kl[max(lo, n_pre):hi].max()) if n_d > 0 else 0
            return n_p, max(n_d, 0), mq_p, mq_d, mkv

        n_seq = n_pre + n_dec
        split = self._overlap_split(cu, n_seq, T)
        s.split_seq, s.split_row = split, int(cu[split]) if split else 0
        s.num_prefill, s.num_decode, s.max_q_prefill, s.max_q_decode, s.max_kv_decode = maxima(0, split or n_seq)
        if split:
            (s.num_prefill_b, s.num_decode_b, s.max_q_prefill_b, s.max_q_decode_b,
             s.max_kv_decode_b) = maxima(split, n_seq)
        fc = self.tp.fused if self.tp.size > 1 else None
        epoch = (ctypes.c_uint * 2)(0, 0)
        if fc is not None:
            epoch[0], epoch[1] = fc.epoch & 0xFFFFFFFF, fc.ll_seq & 0xFFFFFFFF
            self._m.two_kernel_max_tokens = fc.two_kernel_max_tokens
            self._m.ll_max_tokens = fc.ll_max_tokens
        rc = self._fn(ctypes.byref(self._m), ctypes.byref(s), h.data_ptr(), residual.data_ptr(), 0, n_layers,
                      epoch, ctypes.byref(self._out), ctypes.byref(self._fail),
                      ctypes.byref(self._launches), torch.cuda.current_stream().cuda_stream)
        kcuda.launch_count += self._launches.value
        if fc is not None:
            # every collective of the stack took its epoch (and buffer half) from the shared counters
            fc.epoch, fc.ll_seq = epoch[0], epoch[1]
        if rc != 0:
            raise RuntimeError(f"native dense forward failed at layer {rc // 100 - 1}, step {rc % 100}, "
                               f"code {self._fail.value}")
        if fc is not None:
            return fc.hbuf[:T]
        out = self._out.value
        return (self._h[0] if out == self._h[0].data_ptr() else self._h[1])[:T]


# ---- layers with mixers of their own sizes (csrc/cuda/mixer_executor.cu) ---------------------------------------------

class _MixerLayer(ctypes.Structure):
    _fields_ = [(n, P) for n in ("w_in", "b_in", "w_out", "b_out", "ln2", "w_gu", "b_up", "b_down", "w_gu_il", "w_down",
                                 "next_ln")] + \
        [(n, I) for n in ("n_in", "k_out", "inter", "plain", "parallel", "gated", "experts", "top", "expert_inter",
                          "router_rows", "groups", "keep_groups")] + [("limit", F), ("alpha", F)] + \
        [(n, P) for n in ("w_router", "b_router", "w_expert_gu", "w_expert_down", "next_vec")] + \
        [(n, I) for n in ("next_start", "h", "hk", "d", "dv", "window", "keep_first", "shared_kv", "bias_len")] + \
        [("scale", F), ("attn_out_scale", F), ("softcap", F)] + [(n, I) for n in ("sink", "head_gate", "reads", "rot")] + \
        [(n, P) for n in ("rot_table", "q_norm", "k_norm", "bias", "kv")] + \
        [(n, I) for n in ("lh", "ld", "ldv", "rd", "act", "gate")] + \
        [("key_scale", F), ("lin_out_scale", F), ("decay", P), ("rotary", P), ("norm_w", P), ("state", P)] + \
        [(n, I) for n in ("ah", "adim", "avdim", "arank")] + [("ascale", F)] + \
        [(n, P) for n in ("anorm", "a_uk_t", "a_uv", "a_expand")] + [(n, I) for n in ("rc", "rk", "rb")] + \
        [(n, P) for n in ("conv_w", "conv_b", "gates", "gates_by_block", "gates_b", "rate")] + \
        [(n, P * 2) for n in ("ls", "hc_in", "hc_mix", "hc_out")] + [("next_in", P)] + \
        [(n, I) for n in ("gated_residual", "experts_plain", "scoring", "shared_ff")] + [("router_scale", F)] + \
        [(n, P) for n in ("next_ln2", "w_ff_in", "b_ff_in", "w_shared_down")] + \
        [(n, I) for n in ("talk", "out_gate", "qk_norm_all")] + [("talk_mix", P), ("talk_sink", P)] + \
        [(n, I) for n in ("mh", "md", "mrank", "mpad")] + [("mix_out_scale", F)] + \
        [(n, P) for n in ("mu", "w_mix", "w_decay1", "w_decay2", "w_decay0", "bonus", "mix_norm")]


class _MixerModel(ctypes.Structure):
    _fields_ = [("hidden", I), ("block_size", I), ("num_blocks", I), ("center", I), ("streams", I), ("eps", F), ("residual_scale", F), ("in_buf", P),
                ("mix_buf", P), ("o_buf", P), ("gu_buf", P), ("act_buf", P), ("proj_buf", P), ("h_buf", P * 2)] + \
               [(n, P) for n in ("router_buf", "expert_ids", "expert_weights", "pair_pos", "pair_src", "sort_meta",
                                 "rows_buf", "rows_gu_buf", "rows_act_buf", "rows_out_buf")] + \
               [("chunk_buf", P), ("chunk_floats", LL)] + \
               [(n, P) for n in ("shared_buf", "mixes_buf", "rkvg_buf", "rank_buf", "tanh_buf", "decay_buf")] + \
               [("lat_buf", P), ("lat_bytes", LL), ("expand_bytes", LL), ("gemm_ws", P), ("gemm_ws_floats", LL), ("gemm_counters", P), ("n_counters", I),
                ("layers", P)]


class _MixerStep(ctypes.Structure):
    _fields_ = [(n, P) for n in ("positions", "slot_mapping", "seq_of_token", "block_tables", "cu_q", "kv_lens",
                                 "state_slots", "start")] + \
        [(n, I) for n in ("total_tokens", "max_blocks", "num_prefill", "num_decode", "prefill_tokens", "max_q_prefill",
                          "max_kv_decode", "one_token", "num_long", "long_tokens",
                          "max_q_decode")] + [("cu_q_host", P), ("kv_lens_host", P)]


class MixerExecutor:
    """The one-call-per-step path of bf16 models whose layers are :class:`~ksanallm_b200.models.mixers.MixerLayer`."""

    @staticmethod
    def eligible(model) -> bool:
        if os.environ.get("KSANA_DISABLE_NATIVE_EXECUTOR", "0") == "1" or os.environ.get("KSANA_LIBRARY_BASELINE") == "1":
            return False
        if model.device.type != "cuda" or model.dtype != torch.bfloat16 or not model.layers or model.norm_w is None:
            return False
        for layer in model.layers:
            lins = [x for x in (layer.ff_in, layer.shared_down) if x is not None]
            lins += [layer.in_proj, layer.o_proj] + ([layer.ffn.up, layer.ffn.down] if layer.ffn is not None else [])
            if any(lin.kind != "dense" or lin.pre is not None or lin.weight.dtype != torch.bfloat16 or
                   not lin.weight.is_contiguous() or lin.weight.shape[0] % 8 or lin.weight.shape[1] % 8 for lin in lins):
                return False
            f = layer.ffn
            if f is not None and (f.gated, f.act) != (False, "relu2") and (
                    f.up.bias is not None or f.down.bias is not None or not f.gated or f.act != "gelu_tanh"):
                return False
            e = layer.experts
            if layer.spec.gated_residual and model.cfg.hidden_size % 8:
                return False
            if e is not None:
                H, two_i = model.cfg.hidden_size, e.w_gate_up.shape[1] * (2 if layer.spec.moe.plain else 1)
                if e.perm is not None or e._eplb_counts is not None or e.gate_w.dtype != torch.bfloat16 or H % 8 or \
                        two_i % 16 or any(t.dtype != torch.bfloat16 or not t.is_contiguous()
                                          for t in (e.gate_w, e.w_gate_up, e.w_down)) or layer.spec.moe.experts > 2048:
                    return False
        return True

    def __init__(self, model):
        self.model = model
        n = len(model.layers)
        self._layers = (_MixerLayer * n)()
        self._wgu_il = {}
        for i, layer in enumerate(model.layers):
            L = self._layers[i]
            nxt = model.layers[i + 1].ln1 if i + 1 < n else model.norm_w
            L.w_in, L.b_in, L.w_out = _p(layer.in_proj.weight), _p(layer.in_proj.bias), _p(layer.o_proj.weight)
            L.n_in, L.k_out = layer.in_proj.weight.shape[0], layer.o_proj.weight.shape[1]
            L.b_out, L.next_ln = _p(layer.o_proj.bias), _p(nxt)
            for j, c in enumerate(layer.hyper):
                L.hc_in[j], L.hc_mix[j], L.hc_out[j] = _p(c.inp), _p(c.mix), _p(c.out)
                L.ls[j] = _p((layer.ls1, layer.ls2)[j])
            if layer.hyper:
                L.next_in = _p(model.layers[i + 1].hyper[0].inp if i + 1 < n else model.stream_sum)
            L.parallel, L.gated = int(layer.spec.parallel), int(layer.spec.gated)
            if layer.parallel_ff:
                L.inter = layer.parallel_ff
            if layer.experts is not None:
                e, s = layer.experts, layer.spec.moe
                L.experts, L.top, L.expert_inter = s.experts, s.top, e.w_down.shape[2]
                L.groups, L.keep_groups, L.limit, L.alpha = s.groups, s.keep, s.limit, s.alpha
                L.experts_plain, L.scoring, L.router_scale = int(s.plain), int(s.scoring == "sigmoid"), s.scale
                L.ln2 = _p(layer.ln2)
                L.router_rows, L.w_router, L.b_router = e.gate_w.shape[0], _p(e.gate_w), _p(e.logit_bias)
                L.w_expert_gu, L.w_expert_down = _p(e.w_gate_up), _p(e.w_down)
            start = model.layers[i + 1].pass_start if i + 1 < n else None
            if start is not None:
                L.next_vec, L.next_start = _p(start.step), int(start.add_start)
            if layer.ffn is not None:
                L.ln2, L.w_gu, L.w_down = _p(layer.ln2), _p(layer.ffn.up.weight), _p(layer.ffn.down.weight)
                L.inter = layer.ffn.down.weight.shape[1]
                L.plain, L.b_up, L.b_down = int(not layer.ffn.gated), _p(layer.ffn.up.bias), _p(layer.ffn.down.bias)
                if layer.ffn.gated and os.environ.get("KSANA_FUSED_SWIGLU", "0") == "1" and L.inter % 16 == 0:  # see DenseExecutor
                    key = layer.ffn.up.weight.data_ptr()  # (the runs of a looped layer share one copy)
                    if key not in self._wgu_il:
                        self._wgu_il[key] = kcuda.interleave_gate_up(layer.ffn.up.weight)
                    L.w_gu_il = _p(self._wgu_il[key])
            if layer.attn is not None:
                a, s = layer.attn, layer.attn.spec
                L.h, L.hk, L.d, L.dv, L.window = s.heads, s.kv_heads, s.dim, s.vdim, s.window
                L.scale, L.attn_out_scale = s.scale, s.out_scale
                L.keep_first, L.shared_kv = s.keep_first, int(s.shared_kv)
                L.q_norm, L.k_norm = _p(a.q_norm), _p(a.k_norm)
                L.softcap, L.sink, L.head_gate = s.softcap, int(s.sink), int(s.head_gate)
                L.reads, L.rot = int(s.kv_from is not None), s.rot.dims if s.rot else 0
                L.talk, L.out_gate, L.qk_norm_all = int(s.talk), int(s.out_gate), int(s.qk_norm_all)
                L.talk_mix, L.talk_sink = _p(a.talk), _p(a.sink)
            L.gated_residual = int(layer.spec.gated_residual)
            if L.gated_residual:
                L.next_ln2 = _p(model.layers[i + 1].ln2 if i + 1 < n else None)
                if layer.ff_in is not None:
                    L.w_ff_in, L.b_ff_in = _p(layer.ff_in.weight), _p(layer.ff_in.bias)
                    L.w_shared_down, L.shared_ff = _p(layer.shared_down.weight), layer.shared_down.in_features
            if layer.timemix is not None:
                a, s = layer.timemix, layer.timemix.spec
                L.mh, L.md, L.mpad, L.mrank = s.heads, s.dim, a.proj.shape[1], a.w1.shape[0]
                L.mix_out_scale, L.mu, L.w_mix = s.out_scale, _p(a.mu), _p(a.proj)
                L.w_decay1, L.w_decay2, L.w_decay0, L.bonus, L.mix_norm = _p(a.w1), _p(a.w2), _p(a.w0), _p(a.u), _p(a.norm)
            if layer.latent is not None:
                a, s = layer.latent, layer.latent.spec
                L.ah, L.adim, L.avdim, L.arank, L.rot, L.ascale = s.heads, s.dim, s.vdim, s.rank, s.rot_dim, s.scale
                L.head_gate, L.anorm = int(s.head_gate), _p(a.norm)
                L.a_uk_t, L.a_uv, L.a_expand = _p(a.w.uk_t), _p(a.w.uv), _p(a.w.expand)
            if layer.recurrence is not None:
                a, s = layer.recurrence.w, layer.recurrence.spec
                L.rc, L.rk, L.rb = s.width, s.taps, s.blocks
                L.conv_w, L.conv_b, L.gates, L.gates_by_block = _p(a.conv_t), _p(a.conv_b), _p(a.gates), _p(a.gates_by_block)
                L.gates_b, L.rate = _p(a.gates_b), _p(a.rate)
            if layer.linear is not None:
                a, s = layer.linear, layer.linear.spec
                L.lh, L.ld, L.ldv, L.rd = s.heads, s.dim, s.vdim, s.rot_dims
                L.act, L.gate = int(s.act == "silu"), int(s.gate == "sigmoid")
                L.key_scale, L.lin_out_scale = s.key_scale, s.out_scale
                L.decay, L.norm_w = _p(a.decay), _p(a.norm)
        m = self._m = _MixerModel()
        m.hidden, m.eps = model.cfg.hidden_size, float(model.cfg.rms_norm_eps)
        m.residual_scale = float(model.cfg.residual_scale)
        m.center, m.streams = int(model.cfg.norm_type == "layernorm"), model.cfg.streams
        m.expand_bytes = cuda_latent.EXPAND_BYTES
        ws = self._ws = kcuda.workspace(model.device)
        m.gemm_ws, m.gemm_ws_floats = _p(ws.gemm_ws), ws.gemm_ws.numel()
        m.gemm_counters, m.n_counters = _p(ws.gemm_counters), ws.gemm_counters.numel()
        m.layers = ctypes.cast(self._layers, P)
        self.cap, self._bufs, self._chunk, self._latent = 0, [], None, None
        self._rec_width = max(x.rc for x in self._layers)
        self._key = self._tables = None
        self._step = _MixerStep()
        self._fn = kcuda.lib().ksana_mixer_forward
        self._fn.argtypes, self._fn.restype = [P, P, P, P, I, I, P, P, P, P], I
        self._lat_fn = kcuda.lib().ksana_mixer_latent_bytes
        self._lat_fn.argtypes, self._lat_fn.restype = [P, P, I], LL
        self._out, self._fail, self._launches = P(), I(), I()

    def _ensure(self, T: int) -> None:
        if T <= self.cap:
            return
        cap = (max(T, 1024) + 1023) // 1024 * 1024
        L, H = self._layers, self._m.hidden
        cols = [max(max(f(x) for x in L), 8) for f in (
            lambda x: x.n_in, lambda x: x.k_out, lambda x: max(x.lh * x.ldv, x.mh * x.md),
            lambda x: H + x.shared_ff if x.shared_ff else 0 if x.parallel else 2 * x.inter,
            lambda x: x.shared_ff if x.shared_ff else 0 if x.parallel else x.inter)]
        planes = 2 if any(x.gated_residual for x in L) else 1
        cols += [H] + [H * planes] * 2
        dev = self.model.device
        self._bufs = [torch.empty(cap, c, dtype=torch.bfloat16, device=dev) for c in cols]
        m = self._m
        m.in_buf, m.mix_buf, m.o_buf, m.gu_buf, m.act_buf, m.proj_buf, m.h_buf[0], m.h_buf[1] = (_p(b) for b in self._bufs)
        if planes > 1:
            pad, rank = (max(f(x) for x in L) for f in (lambda x: x.mpad, lambda x: x.mrank))
            self._gated = [torch.empty(cap, c, dtype=t, device=dev) for c, t in (
                (H, torch.bfloat16), (5 * H, torch.bfloat16), (4 * pad, torch.bfloat16), (rank, torch.float32),
                (2 * rank, torch.bfloat16), (pad, torch.float32))]
            m.shared_buf, m.mixes_buf, m.rkvg_buf, m.rank_buf, m.tanh_buf, m.decay_buf = (_p(b) for b in self._gated)
        routed = [x for x in L if x.experts]
        if routed:
            top = max(x.top for x in routed)
            self._routed = [torch.empty(cap, max(x.router_rows for x in routed), dtype=torch.float32, device=dev)]
            self._routed += [torch.empty(cap, top, dtype=t, device=dev)
                             for t in (torch.int32, torch.float32, torch.int32, torch.int32)]
            self._routed.append(torch.zeros(3 * max(x.experts for x in routed) + 2, dtype=torch.int32, device=dev))
            self._routed += [torch.empty(cap * top, c, dtype=torch.bfloat16, device=dev)
                             for c in (H, max(2 * x.expert_inter for x in routed), max(x.expert_inter for x in routed), H)]
            for name, b in zip(("router_buf", "expert_ids", "expert_weights", "pair_pos", "pair_src", "sort_meta",
                                "rows_buf", "rows_gu_buf", "rows_act_buf", "rows_out_buf"), self._routed):
                setattr(m, name, _p(b))
        self.cap = cap

    def _bind(self, caches) -> None:
        # the position tables grow with the longest sequence an engine asks for: they are part of the key
        tables = [(layer.attn.bias if layer.attn else None,
                   next((x.rotary() for x in (layer.linear, layer.attn, layer.latent) if x and x.rotary() is not None), None))
                  for layer in self.model.layers]
        key = tuple((c.kv.data_ptr(), c.kv.shape, c.state.data_ptr(), _p(b), _p(r)) for c, (b, r) in zip(caches, tables))
        if key == self._key:
            return
        m = self._m
        m.block_size = 1
        for L, c, layer, (bias, rotary) in zip(self._layers, caches, self.model.layers, tables):
            L.kv, L.state, L.bias, L.rotary = _p(c.kv), _p(c.state), _p(bias), _p(rotary)
            L.rot_table = L.rotary if L.rot else None
            L.bias_len = bias.shape[1] if bias is not None else 0
            m.num_blocks = c.kv.shape[0]
            if layer.kv_width():
                m.block_size = c.kv.shape[1] // layer.kv_width()
        self._key, self._tables = key, tables

    def _chunk_floats(self, need: int) -> None:
        if need > self._m.chunk_floats:
            self._chunk = torch.empty(need, dtype=torch.float32, device=self.model.device)
            self._m.chunk_buf, self._m.chunk_floats = _p(self._chunk), need

    def can_run(self, meta, caches, n_layers: int) -> bool:
        return meta.total_tokens > 0 and (meta.state_slots is not None or not self.model.cfg.has_state)

    def forward(self, meta, caches, h: torch.Tensor, residual: torch.Tensor, n_layers: int) -> torch.Tensor:
        """As DenseExecutor.forward; ``residual`` is the 32-bit stream."""
        from ..ops.cuda_mixer import long_portions
        T = meta.total_tokens
        self._ensure(T)
        self._bind(caches)
        s, m = self._step, self._m
        s.positions, s.slot_mapping, s.seq_of_token = _p(meta.positions), _p(meta.slot_mapping), _p(meta.seq_of_token)
        s.block_tables, s.cu_q, s.kv_lens = _p(meta.block_tables), _p(meta.cu_q), _p(meta.kv_lens)
        s.state_slots, s.total_tokens, s.max_blocks = _p(meta.state_slots), T, meta.max_blocks
        s.start = _p(meta.start)
        n_pre, n_dec, cu = meta.num_prefill, meta.num_decode, meta.cu_q_host
        s.num_prefill, s.num_decode, s.prefill_tokens = n_pre, n_dec, meta.num_prefill_tokens
        s.max_q_prefill = int((cu[1:n_pre + 1] - cu[:n_pre]).max()) if n_pre else 0
        s.max_kv_decode = int(meta.kv_lens_host[n_pre:].max()) if n_dec else 0
        s.one_token = int(T - s.prefill_tokens == n_dec)
        s.max_q_decode = int((cu[n_pre + 1:] - cu[n_pre:-1]).max()) if n_dec else 0
        s.num_long = long_portions(meta) if any(x.lh or x.mh for x in self._layers) else 0
        s.long_tokens = int(cu[s.num_long])
        if s.num_long:
            self._chunk_floats(max((s.long_tokens // 128 + s.num_long) * x.lh * x.ld * x.ldv for x in self._layers))
            self._chunk_floats(max(kcuda.lib().ksana_time_mix_scratch(s.long_tokens, s.num_long, x.mh, x.md)
                                   for x in self._layers))
        if self._rec_width:  # chunks of prompts, or the gates' products where the general kernels run
            self._chunk_floats(max(T * self._rec_width * 5 // 2 + 4, kcuda.lib().ksana_recurrence_scratch(
                s.prefill_tokens, n_pre, s.max_q_prefill, self._rec_width)))
        s.cu_q_host, s.kv_lens_host = cu.ctypes.data, meta.kv_lens_host.ctypes.data
        need = self._lat_fn(ctypes.byref(m), ctypes.byref(s), n_layers)
        if need > m.lat_bytes:
            self._latent = torch.empty(need, dtype=torch.uint8, device=self.model.device)
            m.lat_buf, m.lat_bytes = _p(self._latent), need
        rc = self._fn(ctypes.byref(m), ctypes.byref(s), h.data_ptr(), residual.data_ptr(), 0, n_layers,
                      ctypes.byref(self._out), ctypes.byref(self._fail), ctypes.byref(self._launches),
                      torch.cuda.current_stream().cuda_stream)
        kcuda.launch_count += self._launches.value
        if rc != 0:
            raise RuntimeError(f"native mixer forward failed at layer {rc // 100 - 1}, step {rc % 100}, "
                               f"code {self._fail.value}")
        out = self._bufs[6 if self._out.value == self._bufs[6].data_ptr() else 7]
        return out.view(-1)[:T * m.hidden].view(T, m.hidden)
