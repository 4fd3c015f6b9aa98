"""Layers whose sequence mixers have sizes of their own, described by :class:`LayerSpec`: softmax attention over a
window or everything (with rotation, a learned distance bias, first tokens that stay visible, values that are the keys,
capped scores, a sink, a gate per head, another layer's keys and values, or weights that are mixed across heads), latent
attention, a gated linear recurrence, linear attention with a fixed decay per head, and time mixing with token-dependent
decays, the last two alone or beside attention.

All mixers of a layer read the same normalised input, so their input projections are one GEMM and their outputs go
into one buffer that a single output projection reads. A dense feed-forward that reads that input too (``parallel``) is
part of the same two GEMMs. A layer's cache is the pair (paged keys / values or latents, state pool); either is an empty
tensor where the layer does not have that mixer. A layer that runs several times has one :class:`MixerLayer` per run, over
the same weights.

Where the model has ``streams``, the residual is [T, streams, H] and each sublayer has a :class:`HyperConnection`. Where
a layer's sublayers are gated into the residual (``gated_residual``), its normalised input is [1 or 2, T, H]: one norm for the
mixers, one for the feed-forward.
"""
from __future__ import annotations

from dataclasses import replace
from typing import Dict, NamedTuple, Optional, Tuple

import torch

from .. import ops
from ..config.model_config import (AttentionSpec, LatentAttentionSpec, LayerSpec, LinearAttentionSpec, ModelConfig,
                                   RecurrenceSpec, RotarySpec, TimeMixSpec)
from ..ops import reference as ref
from .layers import DenseFFN, LinearW, MoEFFN


class LayerCache(NamedTuple):
    # [num_blocks, kv_heads * block_size * (dim + vdim)], without the values where they are the keys, or
    # [num_blocks, block_size * (rank + rot_dim)] of latents
    kv: torch.Tensor
    state: torch.Tensor  # [num_slots, *state_shape] fp32


class RotaryTables:
    """cos / sin rows of every rotation the model's layers use, grown to the longest position needed."""

    def __init__(self, device):
        self.device = device
        self.length = 0
        self._specs: Dict[str, RotarySpec] = {}
        self._tables: Dict[str, torch.Tensor] = {}

    def _build(self, key: str) -> None:
        r = self._specs[key]
        self._tables[key] = ref.rotary_table(r.dims, r.base, max(self.length, 1), self.device, r.scaling)

    def reserve(self, length: int) -> None:
        if length > self.length:
            self.length = length
            for key in self._tables:
                self._build(key)

    def get(self, spec: RotarySpec) -> torch.Tensor:
        key = repr(spec)
        if key not in self._tables:
            self._specs[key] = spec
            self._build(key)
        return self._tables[key]


class WindowedAttention:
    def __init__(self, cfg: ModelConfig, spec: AttentionSpec, w: Dict[str, torch.Tensor], prefix: str,
                 tables: RotaryTables):
        self.spec, self.eps, self.tables = spec, cfg.rms_norm_eps, tables
        self.nq, self.nk = spec.heads * spec.dim, spec.kv_heads * spec.dim
        self.nv = 0 if spec.shared_kv else spec.kv_heads * spec.vdim
        if spec.shared_kv and (spec.qk_norm or spec.qkv_bias or spec.rot or spec.head_gate or spec.kv_from is not None):
            raise NotImplementedError("keys that are the values are cached as projected")
        self.page = self.nk + self.nv  # cache elements per token
        if spec.kv_from is not None:
            self.nk = self.nv = 0
        self.width = spec.heads * spec.vdim
        self.rows = self.nq + self.nk + self.nv + (spec.heads if spec.head_gate else self.width if spec.out_gate else 0)
        if spec.talk and (spec.window or spec.bias_max or spec.shared_kv or spec.softcap or spec.sink or spec.head_gate):
            raise NotImplementedError("weights are mixed across heads in attention to all keys with plain scores")
        self.talk, self.sink = w.get(prefix + ".talk"), w.get(prefix + ".sink")
        self.q_norm, self.k_norm = w.get(prefix + ".q_norm"), w.get(prefix + ".k_norm")
        self.rel = w.get(prefix + ".rel")
        self.bias: Optional[torch.Tensor] = None  # [heads, reach]: the bias of every distance a query can see

    def reserve(self, length: int) -> None:
        reach = length if self.spec.keep_first else min(self.spec.window or length, length)
        if self.rel is not None and (self.bias is None or self.bias.shape[1] < reach):
            self.bias = ref.distance_bias(self.rel, self.spec.bias_max, reach)

    def rotary(self) -> Optional[torch.Tensor]:
        return self.tables.get(self.spec.rot) if self.spec.rot is not None else None

    def run(self, x: torch.Tensor, meta, kv: torch.Tensor, out: torch.Tensor,
            ff: Optional[Tuple[torch.Tensor, torch.Tensor, bool]] = None) -> None:
        """x [T, rows] = the projected (q | k | v); writes heads * vdim columns of ``out``. ``ff`` = (input, output,
        gated) of a feed-forward's activation that runs in the launch of the cache append (keys = values only)."""
        s = self.spec
        q = x[:, :self.nq].unflatten(1, (s.heads, s.dim))
        k = x[:, self.nq:self.nq + self.nk].unflatten(1, (s.kv_heads, s.dim)) if self.nk else None
        end = self.nq + self.nk + self.nv
        bs = kv.shape[1] // self.page
        if s.shared_kv:
            u, act, gated = ff if ff is not None else (None, None, False)
            ops.append_act(k, u, meta.slot_mapping, kv, bs, act, gated)
        else:
            v = x[:, self.nq + self.nk:end].unflatten(1, (s.kv_heads, s.vdim)) if self.nk else None
            if k is not None or s.rot is not None or self.q_norm is not None:
                ops.qk_norm_cache(q, k, v, meta.slot_mapping, kv, bs, self.q_norm, self.k_norm, self.eps, meta.positions,
                                  self.rotary(), s.qk_norm_all, s.rot is not None and s.rot.halves)
        if s.talk:
            ops.talking_attention(q, kv, meta, bs, s.kv_heads, s.vdim, s.scale, self.sink, self.talk, s.out_scale, out,
                                  x[:, end:end + self.width] if s.out_gate else None)
            return
        ops.window_attention(q, kv, meta, bs, s.kv_heads, s.vdim, s.scale, s.window, self.bias, s.out_scale, out,
                             s.keep_first, s.softcap, s.sink, x[:, end:end + s.heads] if s.head_gate else None)


class LatentWeights:
    """The maps from the latent to keys and values, in the layouts its kernels want."""

    def __init__(self, uk: torch.Tensor, uv: torch.Tensor):
        self.uk, self.uv = uk, uv                             # [h, dim, rank], [h, vdim, rank]
        self.h, self.dim, self.rank = uk.shape
        self.vdim = uv.shape[1]
        self.uk_t = uk.transpose(1, 2).contiguous()           # [h, rank, dim]: absorbed into the query
        # [h * (dim + vdim), rank]: all heads' keys, then all heads' values, written out by one GEMM
        self.expand = torch.cat((uk.reshape(-1, self.rank), uv.reshape(-1, self.rank)), 0).contiguous()


class LatentAttention:
    def __init__(self, cfg: ModelConfig, spec: LatentAttentionSpec, w: Dict[str, torch.Tensor], prefix: str,
                 tables: RotaryTables):
        self.spec, self.eps, self.tables = spec, cfg.rms_norm_eps, tables
        self.nq, self.na = spec.heads * (spec.dim + spec.rot_dim), spec.rank + spec.rot_dim
        self.rows = self.nq + self.na + (spec.heads if spec.head_gate else 0)
        self.width = spec.heads * spec.vdim
        self.norm = w[prefix + ".latent_norm"]
        self.w = LatentWeights(w[prefix + ".w_uk"], w[prefix + ".w_uv"])

    def reserve(self, length: int) -> None:
        pass

    def rotary(self) -> torch.Tensor:
        return self.tables.get(self.spec.rot)

    def run(self, x: torch.Tensor, meta, kv: torch.Tensor, out: torch.Tensor) -> None:
        """x [T, rows] = the projected (q | latent, rotated key part | gate); writes heads * vdim columns of ``out``."""
        s = self.spec
        q = x[:, :self.nq].unflatten(1, (s.heads, s.dim + s.rot_dim))
        bs = kv.shape[1] // s.width
        gate = x[:, self.nq + self.na:self.nq + self.na + s.heads] if s.head_gate else None
        ops.latent_attention(q, x[:, self.nq:self.nq + self.na], self.norm, self.eps, self.rotary(), kv, meta, bs, self.w,
                             s.scale, gate, out)


class RecurrenceWeights:
    """What a gated recurrence needs behind its input projections."""

    def __init__(self, w: Dict[str, torch.Tensor], prefix: str, decay_scale: float):
        self.conv, self.conv_b = w[prefix + ".conv"], w[prefix + ".conv_b"]        # [C, K], [C] fp32
        self.gates, self.gates_b = w[prefix + ".gates"], w[prefix + ".gates_b"]    # [2, B, C / B, C / B], [2, C] fp32
        self.conv_t = self.conv.t().contiguous()                                   # [K, C]: one load for neighbours
        lam = w[prefix + ".lam"].double()
        self.rate = (decay_scale * torch.nn.functional.softplus(lam, threshold=100)).float()  # [C]
        self.gates_by_block = torch.cat((self.gates[0], self.gates[1]), 1).contiguous()  # [B, 2 C / B, C / B]


class GatedRecurrence:
    def __init__(self, cfg: ModelConfig, spec: RecurrenceSpec, w: Dict[str, torch.Tensor], prefix: str):
        self.spec = spec
        self.rows, self.width = 2 * spec.width, spec.width
        self.w = RecurrenceWeights(w, prefix, spec.decay_scale)

    def run(self, x: torch.Tensor, meta, state: torch.Tensor, out: torch.Tensor) -> None:
        """x [T, rows] = the projected (y | x); writes ``width`` columns of ``out``."""
        C = self.spec.width
        ops.gated_recurrence(x[:, :C], x[:, C:2 * C], state, meta, self.w, out)


class DecayedLinearAttention:
    def __init__(self, cfg: ModelConfig, spec: LinearAttentionSpec, w: Dict[str, torch.Tensor], prefix: str, device,
                 tables: RotaryTables):
        self.spec, self.eps, self.tables = spec, cfg.rms_norm_eps, tables
        self.nq, self.nv = spec.heads * spec.dim, spec.heads * spec.vdim
        self.rows = 2 * self.nq + 2 * self.nv
        self.width = self.nv
        self.decay = torch.tensor(spec.decay, dtype=torch.float64).float().to(device)
        self.norm = w[prefix + ".norm"] if spec.norm == "concat" else None

    def rotary(self) -> Optional[torch.Tensor]:
        return self.tables.get(RotarySpec(self.spec.rot_dims, self.spec.rot_base)) if self.spec.rot_dims else None

    def run(self, x: torch.Tensor, meta, state: torch.Tensor, out: torch.Tensor) -> None:
        """x [T, rows] = the projected (q | k | v | gate); writes heads * vdim columns of ``out``."""
        s = self.spec
        q = x[:, :self.nq].unflatten(1, (s.heads, s.dim))
        k = x[:, self.nq:2 * self.nq].unflatten(1, (s.heads, s.dim))
        v = x[:, 2 * self.nq:2 * self.nq + self.nv].unflatten(1, (s.heads, s.vdim))
        g = x[:, 2 * self.nq + self.nv:]
        o = ops.linear_attention(q, k, v, state, meta, self.decay, s.act, self.rotary(), s.key_scale)
        ops.gated_norm(o, g, self.norm, self.eps, s.gate, s.out_scale, out)


class TimeMixing:
    def __init__(self, cfg: ModelConfig, spec: TimeMixSpec, w: Dict[str, torch.Tensor], prefix: str):
        self.spec, self.eps = spec, cfg.rms_norm_eps
        self.rows, self.width = 0, spec.heads * spec.dim
        self.mu, self.proj = w[prefix + ".mu"], w[prefix + ".mix_proj"]  # [5, W] fp32 (r, k, v, gate, decay), [4, n, W]
        self.w1, self.w2, self.w0 = w[prefix + ".w1"], w[prefix + ".w2"], w[prefix + ".w0"]
        self.u, self.norm = w[prefix + ".u"].contiguous(), w[prefix + ".norm"]

    def run(self, h: torch.Tensor, meta, state: torch.Tensor, out: torch.Tensor) -> None:
        """h [T, W] = the mixer's input; writes heads * dim columns of ``out``."""
        n = self.width
        m = ops.token_mix(h, self.mu, state, meta)
        r, k, v, g = (ops.linear(m[i], self.proj[i])[:, :n] for i in range(4))
        t = ops.tanh_parts(ops.linear(m[4], self.w1, None, torch.float32), h.dtype)
        z = ops.linear(t, self.w2, None, torch.float32)[:, :n]
        o = ops.time_mix(r, k, v, z, self.w0, self.u, state, meta)
        ops.gated_norm(o, g, self.norm, self.eps, "silu", self.spec.out_scale, out, per_head=True)


class PassStart(NamedTuple):
    """What the stream takes ahead of one pass of a loop."""
    step: torch.Tensor      # [H] fp32, the pass's learned vector
    add_start: bool         # also the embedding output: every pass but the first


class HyperConnection:
    """How one sublayer reads the residual streams and what they become: u = sum_s inp[s] x_s;
    x_t <- sum_s mix[s, t] x_s + out[t] y."""

    def __init__(self, w: Dict[str, torch.Tensor], prefix: str):
        self.inp, self.out, self.mix = (w[f"{prefix}.{n}"].contiguous() for n in ("in", "out", "mix"))


class MixerLayer:
    """One run of a layer: x <- x + mixers(norm1(x)); x <- x + ff(norm2(x)) unless the layer has no feed-forward; or, in
    parallel, h = norm1(x); x <- x + (mixers(h) + ff(h)); or, with a gated residual, x <- x + scale * (mixers(norm1(x)) *
    gate1 + ff(norm2(x)) * gate2)."""

    def __init__(self, cfg: ModelConfig, w: Dict[str, torch.Tensor], idx: int, tp, tables: RotaryTables,
                 number: Optional[int] = None):
        """``number``: this run starts that pass of the loop."""
        if tp.size > 1:
            raise NotImplementedError("models described layer by layer run on one GPU (tensor_para_size 1)")
        p = f"model.layers.{idx}"
        spec: LayerSpec = cfg.layers[idx]
        self.cfg, self.tp, self.idx, self.spec = cfg, tp, idx, spec
        self.is_moe = spec.moe is not None
        self.pass_start = PassStart(w["model.loop.step"][number].contiguous(), number > 0) if number is not None else None
        self.ln1, self.ln1_b = w[p + ".input_layernorm.weight"], None
        self.ln2, self.ln2_b = w.get(p + ".post_attention_layernorm.weight"), None
        self.in_proj, self.o_proj = LinearW(w, p + ".mixer.in_proj"), LinearW(w, p + ".mixer.o_proj")
        device = self.ln1.device
        self.attn = WindowedAttention(cfg, spec.attn, w, p + ".mixer", tables) if spec.attn else None
        self.latent = LatentAttention(cfg, spec.latent, w, p + ".mixer", tables) if spec.latent else None
        self.recurrence = GatedRecurrence(cfg, spec.recurrence, w, p + ".mixer") if spec.recurrence else None
        self.timemix = TimeMixing(cfg, spec.timemix, w, p + ".mixer") if spec.timemix else None
        self.linear = DecayedLinearAttention(cfg, spec.linear, w, p + ".mixer", device, tables) if spec.linear else None
        self.hyper = [HyperConnection(w, f"{p}.hc{n}") for n in ((1, 2) if spec.has_ff else (1,))] if cfg.streams else []
        self.ls1, self.ls2 = (w.get(f"{p}.ls{n}") if spec.layer_scale else None for n in (1, 2))
        if spec.layer_scale and not cfg.streams:
            raise NotImplementedError("scales per layer come with residual streams")
        self.ffn = None
        if spec.ff and not spec.parallel:
            self.ffn = DenseFFN(replace(cfg, layers=[], hidden_act=spec.ff_act or cfg.hidden_act, gated_mlp=spec.gated), w,
                                p + ".mlp", tp)
        self.experts = None
        if spec.moe is not None:
            m = spec.moe
            self.experts = MoEFFN(replace(cfg, layers=[], num_experts=m.experts, num_experts_per_tok=m.top,
                                          moe_intermediate_size=m.ff, scoring_func="topk_" + m.scoring, n_group=m.groups,
                                          topk_group=m.keep, routed_scaling_factor=m.scale, num_shared_experts=0), w,
                                  p + ".mlp", tp)
            if m.router_bias and self.experts.logit_bias is None:
                raise KeyError(f"missing {p}.mlp.gate.bias")
            if self.experts.q4 is not None or self.experts.s_gate_up is not None:
                raise NotImplementedError("routed experts of models described layer by layer are not quantised")
        # a gated layer's feed-forward: residual gate and shared expert's input as one projection, the shared expert's output
        self.ff_in = self.shared_down = None
        if spec.gated_residual:
            if spec.ff or not spec.parallel or cfg.loop is not None or cfg.streams or spec.attn is None:
                raise NotImplementedError("gated residuals join attention and routed experts that run side by side")
            if spec.moe is not None:
                if not spec.moe.shared_ff:
                    raise NotImplementedError("routed experts of a gated layer come with a shared one")
                self.ff_in = LinearW(w, p + ".mlp.in_proj")
                self.shared_down = LinearW(w, p + ".mlp.shared_expert.down_proj")
        elif spec.timemix is not None or spec.moe is not None and spec.moe.shared_ff:
            raise NotImplementedError("time mixing and shared experts are part of layers with a gated residual")
        self.parallel_ff = spec.ff if spec.parallel else 0
        if self.parallel_ff and (self.linear is not None or self.attn is None or not spec.attn.shared_kv):
            raise NotImplementedError("a dense feed-forward runs beside attention whose values are its keys")
        if self.experts is not None and spec.parallel == bool(cfg.streams):
            raise NotImplementedError("routed experts run beside the mixers, or behind them over several streams")

    # ---- per-sequence memory ---------------------------------------------------------------------------------
    def kv_width(self) -> int:
        """Cache elements per token."""
        return self.spec.kv_width

    def state_shape(self):
        return self.spec.state_shape or (0, 0, 0)

    def kv_from(self) -> Optional[int]:
        """The layer whose cache this one reads (None: its own)."""
        return self.spec.attn.kv_from if self.spec.attn is not None else None

    def reserve(self, length: int) -> None:
        if self.attn is not None:
            self.attn.reserve(length)

    # ---- forward ---------------------------------------------------------------------------------------------
    def _norm(self, y, wgt, residual, **more):
        """The stream takes ``y`` (and ``more``); returns the normalised sum."""
        return ops.stream_norm(y, wgt, self.cfg.rms_norm_eps, self.cfg.norm_type == "layernorm", residual, residual,
                               self.ln1.dtype, **more)

    def start(self, x: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
        """First layer of the model: (its normalised input, the stream) from the embedding output, which stays as it is.
        With several streams all of them equal it until the first sublayer's result arrives: nothing is copied."""
        if self.spec.gated_residual:
            residual = torch.empty_like(x)
            h = ops.gated_stream_norm(None, None, None, None, None, None, self.cfg.residual_scale, x, residual, self.norms(),
                                      self.cfg.rms_norm_eps, self.ln1.dtype)
            return h, residual
        if self.hyper:
            h = ops.hyper_norm(None, None, None, x, None, None, None, self.hyper[0].inp, self.ln1, self.cfg.rms_norm_eps,
                               self.ln1.dtype)
            return h, torch.empty(x.shape[0], self.cfg.streams, x.shape[1], dtype=torch.float32, device=x.device)
        residual = torch.empty_like(x)
        h = ops.stream_norm(None, self.ln1, self.cfg.rms_norm_eps, self.cfg.norm_type == "layernorm", x, residual,
                            self.ln1.dtype, add_vec=self.pass_start.step if self.pass_start else None)
        return h, residual

    def norms(self):
        """A gated layer's norm weights: the mixers', then the feed-forward's if there is one."""
        return [self.ln1, self.ln2] if self.ln2 is not None else [self.ln1]

    def _gated(self, h: torch.Tensor, residual: torch.Tensor, meta, cache: LayerCache, next_norms):
        H, attn = residual.shape[1], self.attn
        x = self.in_proj(h[0])
        K, n = self.o_proj.in_features, attn.width + (self.timemix.width if self.timemix else 0)
        buf = torch.empty(h.shape[1], K, dtype=h.dtype, device=h.device)
        if K > n:
            buf[:, n:].zero_()
        attn.run(x[:, :attn.rows], meta, cache.kv, buf[:, :attn.width])
        if self.timemix is not None:
            self.timemix.run(h[0], meta, cache.state, buf[:, attn.width:n])
        routed = y = y_scale = y_gate = None
        if self.experts is not None:
            m = self.spec.moe
            z = ops.linear(h[1], self.experts.gate_w, None, torch.float32)
            routed = self.experts.rows(h[1], m.limit, m.alpha, m.plain, z)
            f = self.ff_in(h[1])
            y_scale, y_gate = z[:, m.experts], f[:, :H]
            y = self.shared_down(ops.activation(f[:, H:], "relu2"))
        return ops.gated_stream_norm(self.o_proj(buf), x[:, attn.rows:attn.rows + H], routed, y, y_scale, y_gate,
                                     self.cfg.residual_scale, residual, residual, next_norms, self.cfg.rms_norm_eps,
                                     self.ln1.dtype)

    def mix(self, h: torch.Tensor, meta, cache: LayerCache) -> torch.Tensor:
        x = self.in_proj(h)
        widths = [m.width for m in (self.attn, self.latent, self.linear, self.recurrence) if m is not None]
        widths.append(self.parallel_ff)
        K, used = self.o_proj.in_features, sum(widths)
        buf = torch.empty(h.shape[0], K, dtype=h.dtype, device=h.device)
        if K > used:
            buf[:, used:].zero_()  # padding of the output projection's input
        if self.parallel_ff:
            n = self.parallel_ff * (2 if self.spec.gated else 1)
            ff = (x[:, self.attn.rows:self.attn.rows + n], buf[:, widths[0]:used], self.spec.gated)
            self.attn.run(x[:, :self.attn.rows], meta, cache.kv, buf[:, :widths[0]], ff)
            return buf
        row = col = 0
        for m, mem in ((self.attn, cache.kv), (self.latent, cache.kv), (self.linear, cache.state),
                       (self.recurrence, cache.state)):
            if m is not None:
                m.run(x[:, row:row + m.rows], meta, mem, buf[:, col:col + m.width])
                row, col = row + m.rows, col + m.width
        return buf

    def _streams(self, h: torch.Tensor, residual: torch.Tensor, meta, cache: LayerCache, next_norm, next_in):
        eps, dtype = self.cfg.rms_norm_eps, self.ln1.dtype
        y = self.o_proj(self.mix(h, meta, cache))
        old = meta.start if self.idx == 0 else residual  # ahead of the first result all streams are the embedding output
        c = self.hyper[0]
        if not self.spec.has_ff:
            return ops.hyper_norm(y, self.ls1, None, old, c.mix, c.out, residual, next_in, next_norm, eps, dtype)
        h = ops.hyper_norm(y, self.ls1, None, old, c.mix, c.out, residual, self.hyper[1].inp, self.ln2, eps, dtype)
        y = routed = None
        if self.experts is not None:
            routed = self.experts.rows(h, self.spec.moe.limit, self.spec.moe.alpha)
        else:
            y = self.ffn.down(self.ffn.core(h))
        c = self.hyper[1]
        return ops.hyper_norm(y, self.ls2, routed, residual, c.mix, c.out, residual, next_in, next_norm, eps, dtype)

    def forward(self, h: torch.Tensor, residual: torch.Tensor, meta, cache: LayerCache, next_norm, next_norm_b=None,
                pass_start: Optional[PassStart] = None, next_in: Optional[torch.Tensor] = None,
                next_norm2: Optional[torch.Tensor] = None):
        """Same contract as DecoderLayer.forward: consumes the normalised input, returns the next layer's.
        ``pass_start``: the next run's, if it starts a pass; the embedding output is ``meta.start``. ``next_in``: how the
        next sublayer reads the streams, where there are several. ``next_norm2``: a gated next layer's second norm."""
        if self.spec.gated_residual:
            h = self._gated(h, residual, meta, cache, [next_norm] if next_norm2 is None else [next_norm, next_norm2])
            return h
        if self.hyper:
            return self._streams(h, residual, meta, cache, next_norm, next_in)
        y = self.o_proj(self.mix(h, meta, cache))
        if self.ffn is not None:
            h = self._norm(y, self.ln2, residual)
            y = self.ffn.down(self.ffn.core(h))
        if next_norm is None:
            assert self.experts is None  # (only a pipeline stage ends without a norm)
            residual.add_(y)
            return residual
        more = {}
        if self.experts is not None:
            more["routed"] = self.experts.rows(h)
        if pass_start is not None:
            more.update(add_vec=pass_start.step, add_rows=meta.start if pass_start.add_start else None)
        return self._norm(y, next_norm, residual, **more)
