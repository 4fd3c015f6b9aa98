"""Layers whose sequence mixers have sizes of their own, described by :class:`LayerSpec`: softmax attention over a
window with a learned distance bias, and linear attention with a fixed decay per head, alone or side by side.

Both mixers of a layer read the same normalised input, so their input projections are one GEMM and their outputs go
into one buffer that a single output projection reads. A layer's cache is the pair (paged keys / values, state pool);
either is an empty tensor where the layer does not have that mixer.
"""
from __future__ import annotations

from typing import Dict, NamedTuple, Optional

import torch

from .. import ops
from ..config.model_config import AttentionSpec, LayerSpec, LinearAttentionSpec, ModelConfig
from ..ops import reference as ref
from .layers import DenseFFN, LinearW


class LayerCache(NamedTuple):
    kv: torch.Tensor     # [num_blocks, kv_heads * block_size * (dim + vdim)]
    state: torch.Tensor  # [num_slots, heads, dim, vdim] fp32


class RotaryTables:
    """cos / sin rows of every (dims, base) pair the model's layers use, grown to the longest position needed."""

    def __init__(self, device):
        self.device = device
        self.length = 0
        self._tables: Dict[tuple, torch.Tensor] = {}

    def reserve(self, length: int) -> None:
        if length > self.length:
            self.length = length
            for dims, base in self._tables:
                self._tables[(dims, base)] = ref.rotary_table(dims, base, length, self.device)

    def get(self, dims: int, base: float) -> torch.Tensor:
        t = self._tables.get((dims, base))
        if t is None:
            t = self._tables[(dims, base)] = ref.rotary_table(dims, base, max(self.length, 1), self.device)
        return t


class WindowedAttention:
    def __init__(self, cfg: ModelConfig, spec: AttentionSpec, w: Dict[str, torch.Tensor], prefix: str):
        self.spec, self.eps = spec, cfg.rms_norm_eps
        self.nq, self.nk, self.nv = spec.heads * spec.dim, spec.kv_heads * spec.dim, spec.kv_heads * spec.vdim
        self.rows = self.nq + self.nk + self.nv
        self.width = spec.heads * spec.vdim
        self.q_norm, self.k_norm = w.get(prefix + ".q_norm"), w.get(prefix + ".k_norm")
        self.rel = w.get(prefix + ".rel")
        self.bias: Optional[torch.Tensor] = None  # [heads, reach]: the bias of every distance a query can see

    def reserve(self, length: int) -> None:
        reach = min(self.spec.window or length, length)
        if self.rel is not None and (self.bias is None or self.bias.shape[1] < reach):
            self.bias = ref.distance_bias(self.rel, self.spec.bias_max, reach)

    def run(self, x: torch.Tensor, meta, kv: torch.Tensor, out: torch.Tensor) -> None:
        """x [T, rows] = the projected (q | k | v); writes heads * vdim columns of ``out``."""
        s, T = self.spec, x.shape[0]
        q = x[:, :self.nq].unflatten(1, (s.heads, s.dim))
        k = x[:, self.nq:self.nq + self.nk].unflatten(1, (s.kv_heads, s.dim))
        v = x[:, self.nq + self.nk:].unflatten(1, (s.kv_heads, s.vdim))
        bs = kv.shape[1] // (s.kv_heads * (s.dim + s.vdim))
        ops.qk_norm_cache(q, k, v, meta.slot_mapping, kv, bs, self.q_norm, self.k_norm, self.eps)
        ops.window_attention(q, kv, meta, bs, s.kv_heads, s.vdim, s.scale, s.window, self.bias, s.out_scale, out)


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
        return self.tables.get(self.spec.rot_dims, self.spec.rot_base) if self.spec.rot_dims else None

    def run(self, x: torch.Tensor, meta, state: torch.Tensor, out: torch.Tensor) -> None:
        """x [T, rows] = the projected (q | k | v | gate); writes heads * vdim columns of ``out``."""
        s = self.spec
        q = x[:, :self.nq].unflatten(1, (s.heads, s.dim))
        k = x[:, self.nq:2 * self.nq].unflatten(1, (s.heads, s.dim))
        v = x[:, 2 * self.nq:2 * self.nq + self.nv].unflatten(1, (s.heads, s.vdim))
        g = x[:, 2 * self.nq + self.nv:]
        o = ops.linear_attention(q, k, v, state, meta, self.decay, s.act, self.rotary(), s.key_scale)
        ops.gated_norm(o, g, self.norm, self.eps, s.gate, s.out_scale, out)


class MixerLayer:
    """x <- x + mixers(norm1(x)); x <- x + ff(norm2(x)) unless the layer has no feed-forward."""

    def __init__(self, cfg: ModelConfig, w: Dict[str, torch.Tensor], idx: int, tp, tables: RotaryTables):
        if tp.size > 1:
            raise NotImplementedError("models with recurrent layers run on one GPU (tensor_para_size 1)")
        p = f"model.layers.{idx}"
        spec: LayerSpec = cfg.layers[idx]
        self.cfg, self.tp, self.idx, self.spec = cfg, tp, idx, spec
        self.is_moe = False
        self.ln1, self.ln1_b = w[p + ".input_layernorm.weight"], None
        self.ln2, self.ln2_b = w.get(p + ".post_attention_layernorm.weight"), None
        self.in_proj, self.o_proj = LinearW(w, p + ".mixer.in_proj"), LinearW(w, p + ".mixer.o_proj")
        device = self.ln1.device
        self.attn = WindowedAttention(cfg, spec.attn, w, p + ".mixer") if spec.attn else None
        self.linear = DecayedLinearAttention(cfg, spec.linear, w, p + ".mixer", device, tables) if spec.linear else None
        self.ffn = DenseFFN(cfg, w, p + ".mlp", tp) if spec.ff else None

    # ---- per-sequence memory ---------------------------------------------------------------------------------
    def kv_width(self) -> int:
        """Cache elements per token."""
        a = self.spec.attn
        return a.kv_heads * (a.dim + a.vdim) if a else 0

    def state_shape(self):
        return self.spec.state_shape or (0, 0, 0)

    def reserve(self, length: int) -> None:
        if self.attn is not None:
            self.attn.reserve(length)

    # ---- forward ---------------------------------------------------------------------------------------------
    def _norm(self, x, wgt, bias, residual):
        return ops.layer_norm(x, wgt, bias, self.cfg.rms_norm_eps, residual, self.ln1.dtype)

    def mix(self, h: torch.Tensor, meta, cache: LayerCache) -> torch.Tensor:
        x = self.in_proj(h)
        widths = [m.width for m in (self.attn, self.linear) if m is not None]
        K = self.o_proj.in_features
        buf = torch.empty(h.shape[0], K, dtype=h.dtype, device=h.device)
        if K > sum(widths):
            buf[:, sum(widths):].zero_()  # padding of the output projection's input
        row = col = 0
        for m, mem in ((self.attn, cache.kv), (self.linear, cache.state)):
            if m is not None:
                m.run(x[:, row:row + m.rows], meta, mem, buf[:, col:col + m.width])
                row, col = row + m.rows, col + m.width
        return buf

    def forward(self, h: torch.Tensor, residual: torch.Tensor, meta, cache: LayerCache, next_norm, next_norm_b=None):
        """Same contract as DecoderLayer.forward: consumes the normalised input, returns the next layer's."""
        y = self.o_proj(self.mix(h, meta, cache))
        if self.ffn is not None:
            h = self._norm(y, self.ln2, None, residual)
            y = self.ffn.down(self.ffn.core(h))
        if next_norm is None:
            residual.add_(y)
            return residual
        return self._norm(y, next_norm, next_norm_b, residual)
