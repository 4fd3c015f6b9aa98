"""HF ``config.json`` -> ModelConfig.

One normalised description for every supported architecture family (dense Llama-like, Qwen
variants, MoE variants, DeepSeek MLA+MoE, GPT-style post-norm, ChatGLM, Baichuan, InternLM2 ...).
Reference: src/ksana_llm/utils/config/model_config_parser.cpp (field extraction and
``quantization_config`` parsing, :75-113), model_config.h:222-327 (fields), and the
model-type dispatch of src/ksana_llm/runtime/model_instance.cpp:50-145.
"""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple


@dataclass
class RopeScaling:
    type: str = "default"  # default | linear | dynamic | llama3 | yarn | mrope | internlm2_dynamic
    factor: float = 1.0
    original_max_position_embeddings: int = 0
    low_freq_factor: float = 1.0
    high_freq_factor: float = 4.0
    beta_fast: float = 32.0
    beta_slow: float = 1.0
    mscale: float = 1.0
    mscale_all_dim: float = 0.0
    mrope_section: List[int] = field(default_factory=list)
    alpha: float = 0.0  # dynamic-NTK "alpha" flavour
    attention_factor: float = 0.0  # YaRN: magnitude of cos and sin as given (0: from factor and mscale)


@dataclass
class QuantConfig:
    method: str = "none"  # none | fp8 | fp8_block | gptq | awq | w4a8_awq
    bits: int = 16
    group_size: int = 128
    desc_act: bool = False
    weight_block_size: List[int] = field(default_factory=list)  # [128, 128] for block-scaled fp8
    zero_point: bool = False
    modules_to_not_convert: List[str] = field(default_factory=list)


@dataclass
class RotarySpec:
    """Rotation of the leading ``dims`` dimensions of q and k, neighbouring entries (2i, 2i + 1) being a pair, or the
    entries i and i + dims / 2 (``halves``)."""
    dims: int
    base: float
    scaling: RopeScaling = field(default_factory=RopeScaling)
    halves: bool = False


@dataclass
class AttentionSpec:
    """A softmax-attention mixer of one layer with sizes of its own."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0          # keys a position sees, itself included (0: all earlier ones)
    keep_first: int = 0      # the first tokens of the sequence stay visible however far behind the window they are
    shared_kv: bool = False  # the values are the keys: no value projection, one vector per token in the cache
    bias_max: float = 0.0    # learned distance bias: distance at which its log-spaced buckets end (0: no bias)
    qkv_bias: bool = False
    qk_norm: bool = False    # per-head RMS norm of q and k
    out_scale: float = 1.0   # factor on the mixer's output
    rot: Optional[RotarySpec] = None
    softcap: float = 0.0     # score <- cap * tanh(score / cap), 0: off
    sink: bool = False       # the softmax's denominator has one more term exp(0)
    head_gate: bool = False  # each head's output times the sigmoid of a number of its own, projected from the mixer's input
    o_bias: bool = False
    kv_from: Optional[int] = None  # reads the keys and values of that earlier layer: no projections, no cache of its own
    qk_norm_all: bool = False  # RMS norm of q (and of k) over all heads together, ahead of the rotation
    # every head's softmax weights become a learned mix of all heads' weights (talking heads); the softmax's denominator
    # has one more term exp(s) with a learned s per head
    talk: bool = False
    out_gate: bool = False  # the heads' output times sigmoid of a projection of the mixer's input, number by number


@dataclass
class LatentAttentionSpec:
    """Attention over a cached latent of ``rank`` numbers per token (RMS-normed) and one rotated key part shared by all
    heads; keys of ``dim`` unrotated dimensions and values are linear maps of the latent, per head."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    rank: int
    scale: float
    rot: RotarySpec = None
    head_gate: bool = False

    @property
    def width(self) -> int:
        """Cache elements per token."""
        return self.rank + self.rot_dim


@dataclass
class RecurrenceSpec:
    """A gated linear recurrence per channel behind a short causal convolution, times a GELU branch:
    log a = -decay_scale * r * softplus(lam), S <- a S + sqrt(1 - a^2) i u, the gates r and i being block-diagonal maps
    of u."""
    width: int
    blocks: int
    taps: int
    decay_scale: float = 8.0


@dataclass
class LinearAttentionSpec:
    """A linear-attention mixer with a fixed decay per head: S <- decay S + k v^T, o = S^T q."""
    heads: int
    dim: int
    vdim: int
    decay: List[float]
    act: str = "none"        # activation on q, k and v after their projections: none | silu
    rot_dims: int = 0        # leading dimensions of q and k that are rotated (half-split pairs)
    rot_base: float = 10000.0
    key_scale: float = 1.0   # factor on k after rotation
    norm: str = "head"       # head: weightless RMS norm of each head | concat: one over all heads, with a weight
    gate: str = "silu"       # output gate: silu | sigmoid of its own projection
    out_scale: float = 1.0


@dataclass
class TimeMixSpec:
    """A linear recurrence whose decay is a function of the token, per head and key channel: o = (S + diag(u) k v^T)^T r,
    then S <- diag(w) S + k v^T. Its five inputs read the token's own vector moved towards the previous token's, each by a
    learned amount per coordinate; w = exp(-exp(.)) comes out of a low-rank map."""
    heads: int
    dim: int
    width: int               # of the model: the state also holds the previous token's vector
    out_scale: float = 1.0


@dataclass
class ExpertsSpec:
    """A mixture of gated experts: the ``top`` largest router logits choose, and the softmax over the chosen logits weights
    them (which is the softmax over all experts, divided by the chosen ones' sum). With ``groups`` > 1, equal groups of
    neighbouring experts are ranked by their largest logit first, and only experts of the best ``keep`` groups count.

    An expert is silu(gate) * up; with ``limit`` > 0, g * sigmoid(``alpha`` g) * (u + 1) with g = min(gate, limit) and
    u = up clamped to +-limit."""
    experts: int
    top: int
    ff: int
    router_bias: bool = False  # a bias on the router logits, before the choice
    groups: int = 1
    keep: int = 1
    limit: float = 0.0
    alpha: float = 1.0
    plain: bool = False      # an expert is down(relu(up)^2): no gate
    # sigmoid: the weights are the chosen logits' sigmoids times ``scale``, not normalised
    scoring: str = "softmax"
    scale: float = 1.0
    shared_ff: int = 0       # a shared expert beside the routed ones, times the sigmoid of one number per token (0: none)


@dataclass
class LayerSpec:
    """One layer of a model whose layers differ: its mixers (side by side when there are both) and its feed-forward,
    which is dense (``ff``), routed (``moe``) or absent."""
    attn: Optional[AttentionSpec] = None
    linear: Optional[LinearAttentionSpec] = None
    timemix: Optional[TimeMixSpec] = None
    latent: Optional[LatentAttentionSpec] = None
    recurrence: Optional[RecurrenceSpec] = None
    ff: int = 0              # dense feed-forward width (0: none)
    moe: Optional[ExpertsSpec] = None
    gated: bool = True       # dense feed-forward: act(gate) * up, else act(up)
    parallel: bool = False   # mixers and feed-forward read the same norm: x + (mixers(h) + ff(h))
    ff_bias: bool = False    # biases of the dense feed-forward's projections
    ff_act: str = ""         # its activation ("": the model's)
    layer_scale: bool = False  # each sublayer's result times a learned vector
    # mixers and feed-forward run side by side over norms of their own of the same stream, and each one's result is
    # multiplied, number by number, by the sigmoid of a map of what it read
    gated_residual: bool = False

    @property
    def state_shape(self):
        if self.timemix is not None:  # every head's state [key][value], then the previous token's vector
            t = self.timemix
            return (1, 1, t.heads * t.dim * t.dim + t.width)
        if self.recurrence is not None:  # the recurrent state, then the convolution's last inputs, oldest first
            return (1, self.recurrence.taps, self.recurrence.width)
        return (self.linear.heads, self.linear.dim, self.linear.vdim) if self.linear else None

    @property
    def has_ff(self) -> bool:
        return self.ff > 0 or self.moe is not None

    @property
    def kv_width(self) -> int:
        """Cache elements per token."""
        a = self.attn
        if self.latent is not None:
            return self.latent.width
        if a is None or a.kv_from is not None:
            return 0
        return a.kv_heads * (a.dim + (0 if a.shared_kv else a.vdim))


@dataclass
class LoopSpec:
    """Layers start .. stop - 1 run ``times`` times in a row with the same weights. A learned vector per pass is added to
    the stream ahead of the pass, and ahead of every pass but the first also the embedding output."""
    start: int
    stop: int
    times: int


@dataclass
class ModelConfig:
    model_type: str = "llama"
    architectures: List[str] = field(default_factory=list)
    vocab_size: int = 32000
    hidden_size: int = 4096
    num_layers: int = 32
    num_heads: int = 32
    num_kv_heads: int = 32
    head_dim: int = 128
    intermediate_size: int = 11008
    max_position_embeddings: int = 4096
    rms_norm_eps: float = 1e-6
    rope_theta: float = 10000.0
    rope_scaling: RopeScaling = field(default_factory=RopeScaling)
    rope_interleaved: bool = False  # GPT-J style pairs instead of neox halves
    rotary_dim: int = 0  # 0 = full head_dim
    position_encoding: str = "rope"  # rope | alibi | learned | none
    tie_word_embeddings: bool = False
    hidden_act: str = "silu"
    norm_type: str = "rmsnorm"  # rmsnorm | layernorm
    post_norm: bool = False  # GPT-style
    qkv_bias: bool = False
    o_bias: bool = False
    mlp_bias: bool = False
    gated_mlp: bool = True
    qk_norm: bool = False  # per-head RMSNorm on q and k before RoPE (Qwen3)
    cla_share_factor: int = 0  # cross-layer attention: K/V projections shared by groups of this many layers (Hunyuan)
    qk_norm_after_rope: bool = False  # ... applied after RoPE instead (Hunyuan)
    sliding_window: int = 0  # attention window in tokens (0: full causal); per layer via sliding_layers
    sliding_layers: List[int] = field(default_factory=list)  # 1 = windowed layer; empty with a window: every layer
    qk_l2_norm: bool = False  # weightless RMS normalisation of q and k after RoPE on the RoPE layers (Llama 4)
    rope_layers: List[int] = field(default_factory=list)  # per layer: 1 = RoPE, 0 = no position encoding (Llama 4)
    moe_layers: List[int] = field(default_factory=list)   # explicit MoE layer indices (Llama 4); empty: by frequency
    moe_router: str = "standard"  # standard | llama4 (top-k on logits, sigmoid score scales the expert INPUT)
    attn_temperature_tuning: bool = False  # Llama 4: query scaling on the no-RoPE layers
    attention_chunk_size: int = 0  # Llama 4: RoPE layers attend inside blocks of this many positions (0 = off)
    attn_floor_scale: float = 8192.0
    attn_scale_coef: float = 0.1
    bos_token_id: Optional[int] = None
    eos_token_ids: List[int] = field(default_factory=list)
    pad_token_id: Optional[int] = None
    torch_dtype: str = "bfloat16"
    emb_scale: float = 1.0
    logit_scale: float = 1.0
    residual_scale: float = 1.0
    # MoE
    num_experts: int = 0
    num_experts_per_tok: int = 0
    moe_intermediate_size: int = 0
    num_shared_experts: int = 0
    shared_expert_intermediate_size: int = 0
    shared_expert_gate: bool = False
    first_k_dense_replace: int = 0
    moe_layer_freq: int = 1
    norm_topk_prob: bool = False
    scoring_func: str = "softmax"  # softmax | sigmoid
    n_group: int = 1
    topk_group: int = 1
    routed_scaling_factor: float = 1.0
    topk_method: str = "greedy"  # greedy | group_limited_greedy | noaux_tc
    # MLA
    use_mla: bool = False
    q_lora_rank: int = 0
    kv_lora_rank: int = 0
    qk_nope_head_dim: int = 0
    qk_rope_head_dim: int = 0
    v_head_dim: int = 0
    # MTP
    # sparse attention indexer (DeepSeek-V3.2, GLM DSA): every query keeps the index_topk best-scoring keys
    mla_norm_eps: float = 0.0  # epsilon of the low-rank q / kv norms when it differs from rms_norm_eps (0: same)
    index_topk: int = 0
    index_n_heads: int = 0
    index_head_dim: int = 0
    num_nextn_predict_layers: int = 0
    reranker_start_layer: int = 0  # layer-wise reranker: depth of the first scoring head lm_head.0.linear_head
    num_register_token: int = 0  # parallel token prediction: register tokens appended per step (0 = off)
    reg_token_id: int = 0
    # models described layer by layer (empty: every layer follows the fields above)
    layers: List[LayerSpec] = field(default_factory=list)
    logit_softcap: float = 0.0    # logits <- cap * tanh(logits / cap); 0 = off
    residual_fp32: bool = False   # the residual stream is kept in 32-bit floats
    loop: Optional[LoopSpec] = None
    # hyper-connections: the residual is this many streams; each sublayer reads a weighted sum of them, and every stream
    # becomes a weighted sum of all old ones and the sublayer's result (0: one plain residual)
    streams: int = 0
    # quantisation
    quant: QuantConfig = field(default_factory=QuantConfig)
    raw: Dict[str, Any] = field(default_factory=dict)

    @property
    def is_moe(self) -> bool:
        return self.num_experts > 0

    def is_moe_layer(self, layer_idx: int) -> bool:
        if self.layers:
            return self.layers[layer_idx].moe is not None
        if not self.is_moe:
            return False
        if self.moe_layers:
            return layer_idx in self.moe_layers
        return layer_idx >= self.first_k_dense_replace and (layer_idx % max(self.moe_layer_freq, 1) == 0)

    @property
    def has_state(self) -> bool:
        """Some layer carries a recurrent state from token to token."""
        return any(l.state_shape is not None for l in self.layers)

    def layer_runs(self) -> List[Tuple[int, Optional[int]]]:
        """The layers in the order they run, each with the number of the pass that starts with it (None: no pass does).
        Every run has a cache of its own."""
        order = list(range(self.num_layers))
        if self.loop is None:
            return [(i, None) for i in order]
        lo, hi = self.loop.start, self.loop.stop
        passes = [(i, t if i == lo else None) for t in range(self.loop.times) for i in order[lo:hi]]
        return [(i, None) for i in order[:lo]] + passes + [(i, None) for i in order[hi:]]

    @property
    def q_head_dim(self) -> int:
        return self.qk_nope_head_dim + self.qk_rope_head_dim if self.use_mla else self.head_dim


def _rope_scaling(d: Optional[Dict[str, Any]], cfg: Dict[str, Any]) -> RopeScaling:
    rs = RopeScaling()
    if not d:
        return rs
    t = d.get("rope_type", d.get("type", "default")) or "default"
    rs.type = {"ntk": "dynamic", "dynamic_ntk": "dynamic", "deepseek_yarn": "yarn", "mrope": "default"}.get(t, t)
    rs.factor = float(d.get("factor", 1.0) or 1.0)
    rs.original_max_position_embeddings = int(
        d.get("original_max_position_embeddings", cfg.get("max_position_embeddings", 0)) or 0)
    rs.low_freq_factor = float(d.get("low_freq_factor", 1.0))
    rs.high_freq_factor = float(d.get("high_freq_factor", 4.0))
    rs.beta_fast = float(d.get("beta_fast", 32.0))
    rs.beta_slow = float(d.get("beta_slow", 1.0))
    rs.mscale = float(d.get("mscale", 1.0))
    rs.mscale_all_dim = float(d.get("mscale_all_dim", 0.0))
    rs.mrope_section = list(d.get("mrope_section", []) or [])
    rs.alpha = float(d.get("alpha", 0.0) or 0.0)
    return rs


def _quant(d: Optional[Dict[str, Any]]) -> QuantConfig:
    q = QuantConfig()
    if not d:
        return q
    method = str(d.get("quant_method", d.get("quant_algo", "none"))).lower()
    if method == "fp8":
        wbs = d.get("weight_block_size")
        if wbs:
            q.method, q.weight_block_size, q.bits = "fp8_block", [int(x) for x in wbs], 8
        else:
            q.method, q.bits = "fp8", 8
    elif method in ("gptq", "awq"):
        q.method = method
        q.bits = int(d.get("bits", d.get("w_bit", 4)))
        q.group_size = int(d.get("group_size", d.get("q_group_size", 128)))
        q.desc_act = bool(d.get("desc_act", False))
        q.zero_point = bool(d.get("zero_point", method == "awq"))
    elif method in ("w4a8_awq", "mixed", "modelopt", "rtn"):
        q.method = method
        q.bits = int(d.get("bits", 4))
        q.group_size = int(d.get("group_size", 128))
    else:
        q.method = method
    q.modules_to_not_convert = list(d.get("modules_to_not_convert", []) or [])
    return q


def _molopel_mixers(kind: str, c: Dict[str, Any]) -> LayerSpec:
    if kind == "lightning":
        return LayerSpec(linear=LinearAttentionSpec(
            int(c["heads"]), int(c["dim"]), int(c["vdim"]), [float(x) for x in c["decay"]], act="silu",
            norm="concat", gate="sigmoid"))
    if kind == "parallel":
        a, r = c["left"], c["right"]
        return LayerSpec(
            attn=AttentionSpec(int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"]), float(a["scale"]),
                               window=int(a["mask"]["size"]), bias_max=float(a["bias_max"]), qkv_bias=True,
                               qk_norm=True, out_scale=float(c["left_scale"])),
            linear=LinearAttentionSpec(int(r["heads"]), int(r["dim"]), int(r["vdim"]), [float(x) for x in r["decay"]],
                                       rot_dims=int(r["rot"]["dims"]), rot_base=float(r["rot"]["base"]),
                                       key_scale=float(r["dim"]) ** -0.5, norm="head", gate="silu",
                                       out_scale=float(c["right_scale"])))
    raise ValueError(f"unknown Molopel layer type {kind!r}")


def _layered_config(c: Dict[str, Any], model_type: str) -> ModelConfig:
    """What the designs whose ``config.json`` lists their layers one by one have in common; reads ``m.layers``' sizes into
    the fields other parts of the engine look at."""
    m = ModelConfig(model_type=model_type, architectures=[str(c["architecture"])], raw=c)
    m.vocab_size, m.hidden_size = int(c["vocab"]), int(c["width"])
    m.rms_norm_eps = float(c["norm"]["eps"])
    m.emb_scale = float((c.get("embedding") or {}).get("scale", 1.0))
    m.residual_fp32 = True
    m.hidden_act = "gelu_tanh"
    m.torch_dtype = str(c.get("torch_dtype", "bfloat16"))
    eos = c.get("eos_token_id")
    m.eos_token_ids = [int(e) for e in eos] if isinstance(eos, (list, tuple)) else ([int(eos)] if eos is not None else [])
    m.bos_token_id, m.pad_token_id = c.get("bos_token_id"), c.get("pad_token_id")
    return m


def _set_layers(m: ModelConfig, layers: List[LayerSpec]) -> None:
    m.layers, m.num_layers = layers, len(layers)
    attn = next((l.attn for l in layers if l.attn is not None), None)
    latent = next((l.latent for l in layers if l.latent is not None), None)
    if attn is not None:
        m.num_heads, m.num_kv_heads, m.head_dim = attn.heads, attn.kv_heads, attn.dim
    elif latent is not None:
        m.num_heads, m.num_kv_heads, m.head_dim = latent.heads, 1, latent.dim + latent.rot_dim
    m.intermediate_size = max((l.ff for l in layers), default=0)
    m.num_experts = max((l.moe.experts for l in layers if l.moe), default=0)
    m.num_experts_per_tok = max((l.moe.top for l in layers if l.moe), default=0)
    m.moe_intermediate_size = max((l.moe.ff for l in layers if l.moe), default=0)


def _givirax_layer(entry: Dict[str, Any]) -> LayerSpec:
    if str(entry["type"]) != "attention":
        raise ValueError(f"unknown Givirax layer type {entry['type']!r}")
    a, mlp = entry["mixer"], entry.get("mlp")
    spec = LayerSpec(parallel=True, gated=False, attn=AttentionSpec(
        int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"]), float(a["scale"]),
        window=int(a["mask"]["size"]), keep_first=int(a["mask"]["keep_first"]), shared_kv=True))
    if spec.attn.vdim != spec.attn.dim or spec.attn.heads % spec.attn.kv_heads:
        raise ValueError("values that are the keys have the keys' size, and heads are a multiple of kv_heads")
    if spec.attn.window < 1:
        raise ValueError("a position sees at least itself: mask.size >= 1")
    if mlp is not None:
        kind = str(mlp.get("kind", "dense"))
        if kind == "dense":
            spec.ff = int(mlp["ff"])
        elif kind == "moe":
            r = mlp["router"]
            spec.moe = ExpertsSpec(int(r["experts"]), int(r["top"]), int(mlp["expert"]["ff"]), router_bias=True)
            if not 1 <= spec.moe.top <= spec.moe.experts:
                raise ValueError("router.top must lie between 1 and router.experts")
        else:
            raise ValueError(f"unknown Givirax feed-forward {kind!r}")
    return spec


def _givirax_config(c: Dict[str, Any]) -> ModelConfig:
    """Givirax: layers whose attention (a sliding window plus the first tokens, no rotation, values = keys) and
    feed-forward (plain GELU or routed SiLU experts) read one norm side by side; learned positions, a range of layers that
    runs several times, untied head."""
    m = _layered_config(c, "givirax")
    _set_layers(m, [_givirax_layer(e) for e in c["layers"]])
    m.position_encoding, m.gated_mlp = "learned", False
    m.max_position_embeddings = int(c["max_positions"])
    loop = c.get("loop")
    if loop:
        m.loop = LoopSpec(int(loop["start"]), int(loop["stop"]), int(loop["times"]))
        if not (0 <= m.loop.start < m.loop.stop <= m.num_layers and m.loop.times >= 1):
            raise ValueError(f"loop {loop} does not fit {m.num_layers} layers")
    return m


def _molopel_config(c: Dict[str, Any]) -> ModelConfig:
    """Molopel: layers of linear attention alone ("lightning") or of windowed attention beside retention
    ("parallel"), each with sizes of its own; LayerNorm without bias, tied embeddings, soft-capped logits."""
    m = _layered_config(c, "molopel")
    layers = []
    for entry in c["layers"]:
        spec = _molopel_mixers(str(entry["type"]), entry["mixer"])
        mlp = entry.get("mlp")
        if mlp is not None:
            if str(mlp.get("kind", "dense")) != "dense":
                raise ValueError(f"unknown Molopel feed-forward {mlp.get('kind')!r}")
            spec.ff = int(mlp["ff"])
        if spec.linear is not None and len(spec.linear.decay) != spec.linear.heads:
            raise ValueError("one decay per head is needed")
        layers.append(spec)
    _set_layers(m, layers)
    m.norm_type, m.position_encoding = "layernorm", "none"
    m.tie_word_embeddings = True
    m.logit_softcap = float(c.get("logit_softcap") or 0.0)
    m.max_position_embeddings = int(c.get("max_position_embeddings", 1 << 20))
    return m


def _ladusun_rotary(r: Dict[str, Any], kind: str) -> RotarySpec:
    s = r.get("scaling")
    if not s:
        return RotarySpec(int(r["dims"]), float(r["base"]))
    rs = RopeScaling(type=kind, factor=float(s["factor"]), original_max_position_embeddings=int(s["original"]))
    if kind == "yarn":
        rs.beta_fast, rs.beta_slow = float(s["fast"]), float(s["slow"])
        rs.attention_factor = 0.1 * math.log(rs.factor) + 1.0
    else:
        rs.low_freq_factor, rs.high_freq_factor = float(s["low"]), float(s["high"])
    spec = RotarySpec(int(r["dims"]), float(r["base"]), rs)
    if spec.dims % 2:
        raise ValueError("rot.dims counts pairs of dimensions")
    return spec


def _ladusun_layer(entry: Dict[str, Any]) -> LayerSpec:
    kind, c, mlp = str(entry["type"]), entry["mixer"], entry.get("mlp")
    spec = LayerSpec(gated=False, layer_scale=True)
    if kind == "rglru":
        spec.recurrence = RecurrenceSpec(int(c["width"]), int(c["blocks"]), int(c["conv"]))
        if spec.recurrence.width % spec.recurrence.blocks or spec.recurrence.taps < 1:
            raise ValueError("the recurrence's width is a multiple of its blocks, and the convolution has at least one tap")
    elif kind == "attention":
        kv_from = c.get("kv_from")
        spec.attn = AttentionSpec(
            int(c["heads"]), int(c["kv_heads"]), int(c["dim"]), int(c["vdim"]), float(c["scale"]), qkv_bias=True,
            rot=_ladusun_rotary(c["rot"], "llama3"), softcap=float(c.get("softcap") or 0.0), sink=True, head_gate=True, o_bias=True,
            kv_from=None if kv_from is None else int(kv_from))
        if spec.attn.heads % spec.attn.kv_heads or spec.attn.rot.dims > spec.attn.dim:
            raise ValueError("heads are a multiple of kv_heads, and at most a whole head is rotated")
    elif kind == "latent_attention":
        spec.latent = LatentAttentionSpec(
            int(c["heads"]), int(c["dim"]), int(c["rot_dim"]), int(c["vdim"]), int(c["kv_rank"]), float(c["scale"]),
            rot=_ladusun_rotary(c["rot"], "yarn"), head_gate=True)
        if spec.latent.rot.dims != spec.latent.rot_dim:
            raise ValueError("the rotated part is rotated as a whole: rot.dims = rot_dim")
    else:
        raise ValueError(f"unknown Ladusun layer type {kind!r}")
    if mlp is None:
        return spec
    ff = str(mlp.get("kind", "dense"))
    if ff == "dense":
        spec.ff, spec.ff_bias, spec.ff_act = int(mlp["ff"]), True, "relu2"
    elif ff == "moe":
        r, e = mlp["router"], mlp["expert"]
        g = r.get("groups") or dict(count=1, keep=1)
        spec.moe = ExpertsSpec(int(r["experts"]), int(r["top"]), int(e["ff"]), groups=int(g["count"]), keep=int(g["keep"]),
                               limit=float(e["limit"]), alpha=1.702)
        m = spec.moe
        if m.groups < 1 or m.experts % m.groups or not 1 <= m.keep <= m.groups or \
                not 1 <= m.top <= m.experts // m.groups * m.keep or m.limit <= 0:
            raise ValueError(f"router {r} does not fit, or the experts' limit is not positive")
    else:
        raise ValueError(f"unknown Ladusun feed-forward {ff!r}")
    return spec


def _ladusun_config(c: Dict[str, Any]) -> ModelConfig:
    """Ladusun: layers of latent attention, capped attention with a sink (some read another layer's keys and values), or
    a gated linear recurrence; squared-ReLU or routed clamped experts; several residual streams joined by
    hyper-connections; tied embeddings."""
    m = _layered_config(c, "ladusun")
    layers = [_ladusun_layer(e) for e in c["layers"]]
    for i, l in enumerate(layers):
        if l.attn is None or l.attn.kv_from is None:
            continue
        j = l.attn.kv_from
        src = layers[j].attn if 0 <= j < i else None
        if src is None or src.kv_from is not None or (src.kv_heads, src.dim, src.vdim, src.rot) != \
                (l.attn.kv_heads, l.attn.dim, l.attn.vdim, l.attn.rot):
            raise ValueError(f"layer {i} cannot read the keys and values of layer {j}")
    _set_layers(m, layers)
    m.streams = int(c["streams"])
    if m.streams < 1:
        raise ValueError("streams counts residual streams, at least one")
    m.position_encoding, m.gated_mlp, m.tie_word_embeddings = "none", False, True
    m.max_position_embeddings = int(c.get("max_position_embeddings", 1 << 20))
    return m


def _vibunex_layer(entry: Dict[str, Any], width: int) -> LayerSpec:
    if str(entry["type"]) != "parallel":
        raise ValueError(f"unknown Vibunex layer type {entry['type']!r}")
    c, mlp = entry["mixer"], entry.get("mlp")
    a, r = c["left"], c["right"]
    rot = _ladusun_rotary(a["rot"], "yarn")
    rot.halves = True
    spec = LayerSpec(
        parallel=True, gated=False, gated_residual=True,
        attn=AttentionSpec(int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"]), float(a["scale"]), rot=rot,
                           out_scale=float(c["left_scale"]), qk_norm_all=True, talk=True, out_gate=True),
        timemix=TimeMixSpec(int(r["heads"]), int(r["dim"]), width, float(c["right_scale"])))
    if spec.attn.heads % spec.attn.kv_heads or rot.dims > spec.attn.dim or rot.dims % 2:
        raise ValueError("heads are a multiple of kv_heads, and pairs of at most a whole head are rotated")
    if mlp is not None:
        if str(mlp.get("kind", "moe")) != "moe":
            raise ValueError(f"unknown Vibunex feed-forward {mlp.get('kind')!r}")
        q = mlp["router"]
        spec.moe = ExpertsSpec(int(q["experts"]), int(q["top"]), int(mlp["expert"]["ff"]), plain=True, scoring="sigmoid",
                               scale=float(q["scale"]), shared_ff=int(mlp["shared"]["ff"]))
        if not 1 <= spec.moe.top <= spec.moe.experts:
            raise ValueError("router.top must lie between 1 and router.experts")
    return spec


def _vibunex_config(c: Dict[str, Any]) -> ModelConfig:
    """Vibunex: attention whose heads' weights are mixed, beside time mixing with token-dependent decays, beside routed
    squared-ReLU experts and a shared one; sublayers gated into one scaled residual; norms with one number; untied head."""
    m = _layered_config(c, "vibunex")
    _set_layers(m, [_vibunex_layer(e, m.hidden_size) for e in c["layers"]])
    m.residual_scale = float(c["residual_mult"])
    m.position_encoding, m.gated_mlp = "none", False
    m.max_position_embeddings = int(c.get("max_position_embeddings", 1 << 20))
    return m


def model_config_from_dict(c: Dict[str, Any]) -> ModelConfig:
    design = {"molopel": _molopel_config, "givirax": _givirax_config, "ladusun": _ladusun_config,
              "vibunex": _vibunex_config}.get(str(c.get("architecture", "")).lower())
    if design is not None:
        return design(c)
    if isinstance(c.get("text_config"), dict) and str(c.get("model_type", "")).lower() in ("llama4",):
        # multimodal wrapper configs keep the language model under "text_config"
        inner = dict(c["text_config"])
        inner.setdefault("model_type", "llama4_text")
        for k in ("torch_dtype", "dtype", "quantization_config"):
            if k in c and k not in inner:
                inner[k] = c[k]
        c = inner
    if isinstance(c.get("text_config"), dict) and str(c.get("model_type", "")).lower() in ("qwen2_vl", "qwen2_5_vl",
                                                                                              "internvl"):
        inner = dict(c["text_config"])
        if str(c["model_type"]).lower() != "internvl":  # InternVL's tower keeps its own type (qwen2, llama, ...)
            inner["model_type"] = str(c["model_type"]).lower()
        for k in ("torch_dtype", "dtype", "quantization_config", "tie_word_embeddings", "architectures"):
            if k in c and k not in inner:
                inner[k] = c[k]
        c = inner
    mt = str(c.get("model_type", "llama")).lower()
    m = ModelConfig(model_type=mt, architectures=list(c.get("architectures", []) or []), raw=c)
    g = c.get
    m.vocab_size = int(g("vocab_size", g("padded_vocab_size", 32000)))
    m.hidden_size = int(g("hidden_size", g("n_embd", g("d_model", 4096))))
    m.num_layers = int(g("num_hidden_layers", g("n_layer", g("num_layers", 32))))
    m.num_heads = int(g("num_attention_heads", g("n_head", 32)))
    kv = g("num_key_value_heads", None)
    if kv is None:
        if g("multi_query_attention", False):
            kv = g("multi_query_group_num", 1)
        else:
            kv = g("num_kv_heads", m.num_heads)
    m.num_kv_heads = int(kv)
    m.head_dim = int(g("head_dim", None) or g("kv_channels", None) or (m.hidden_size // m.num_heads))
    m.intermediate_size = int(g("intermediate_size", g("ffn_hidden_size", g("n_inner", None) or 4 * m.hidden_size)))
    m.max_position_embeddings = int(g("max_position_embeddings", g("n_positions", g("seq_length", 4096))))
    m.rms_norm_eps = float(g("rms_norm_eps", g("layer_norm_epsilon", g("layernorm_epsilon", g("layer_norm_eps", 1e-6)))))
    # transformers >= 5 folds rope_theta and the scaling block into one "rope_parameters" dict
    rp = g("rope_parameters", None) or {}
    m.rope_theta = float(g("rope_theta", None) or rp.get("rope_theta", None) or g("rotary_emb_base", 10000.0))
    rs_dict = g("rope_scaling", None)
    if rs_dict is None and rp and (str(rp.get("rope_type", rp.get("type", "default"))) != "default" or
                                   rp.get("mrope_section")):
        rs_dict = rp
    m.rope_scaling = _rope_scaling(rs_dict, c)
    xd = g("xdrope_section", None)
    if xd and g("position_embedding_xdrope", True):
        # XD-RoPE (Arc-Hunyuan-Video): four position axes, sections given as fractions of half the head size; the
        # table itself is the alpha-scaled NTK one (reference: arc_hunyuan_video_config_parser.cpp:72-93,
        # rotary_embedding.cu:361-372)
        half = (m.head_dim or m.hidden_size // m.num_heads) // 2
        m.rope_scaling.mrope_section = [int(float(f) * half) for f in xd]
        if m.rope_scaling.type in ("default", "xdrope"):
            m.rope_scaling.type = "dynamic"
            m.rope_scaling.alpha = float((rs_dict or {}).get("alpha", 1000.0))
    m.tie_word_embeddings = bool(g("tie_word_embeddings", False))
    m.hidden_act = str(g("hidden_act", g("activation_function", "silu")))
    m.torch_dtype = str(g("torch_dtype", g("dtype", "bfloat16")))
    m.bos_token_id = g("bos_token_id", None)
    eos = g("eos_token_id", None)
    m.eos_token_ids = [int(e) for e in eos] if isinstance(eos, (list, tuple)) else ([int(eos)] if eos is not None else [])
    m.pad_token_id = g("pad_token_id", None)
    m.qkv_bias = bool(g("attention_bias", g("qkv_bias", g("add_qkv_bias", False))))
    m.mlp_bias = bool(g("mlp_bias", False))
    sw = g("sliding_window", None)
    if sw and g("use_sliding_window", True):
        m.sliding_window = int(sw)
        lt = g("layer_types", None)
        if lt:
            m.sliding_layers = [1 if str(t) == "sliding_attention" else 0 for t in lt]

    if mt in ("qwen2", "qwen2_moe", "qwen", "qwen2_vl", "qwen2_5_vl"):
        m.qkv_bias = True if g("attention_bias", None) is None else bool(g("attention_bias"))
    if mt in ("qwen3", "qwen3_moe"):
        m.qk_norm = True
        m.qkv_bias = bool(g("attention_bias", False))
    if mt.startswith("hunyuan"):
        m.qk_norm = bool(g("use_qk_norm", True))
        m.qk_norm_after_rope = m.qk_norm
        if g("use_cla", False):
            m.cla_share_factor = int(g("cla_share_factor", 0) or 0)
    if mt.startswith("llama4"):
        m.rope_interleaved = True
        m.qk_l2_norm = bool(g("use_qk_norm", True))
        m.rope_layers = [int(x) for x in (g("no_rope_layers", None) or [])]
        m.attn_temperature_tuning = bool(g("attn_temperature_tuning", False))
        m.attn_floor_scale = float(g("floor_scale", 8192))
        m.attention_chunk_size = int(g("attention_chunk_size", 0) or 0)
        m.attn_scale_coef = float(g("attn_scale", 0.1))
    if mt in ("gpt2", "fairseq_transformer", "gpt"):
        m.norm_type, m.post_norm, m.gated_mlp, m.position_encoding = "layernorm", False, False, "learned"
        m.qkv_bias = m.o_bias = m.mlp_bias = True
        m.hidden_act = str(g("activation_function", "gelu_new"))
        m.tie_word_embeddings = bool(g("tie_word_embeddings", True))
    if mt == "baichuan":
        # Baichuan-13B (hidden 5120) uses ALiBi, 7B uses RoPE
        if m.hidden_size >= 5120:
            m.position_encoding = "alibi"
    if mt == "chatglm":
        m.rope_interleaved = True
        m.rotary_dim = m.head_dim // 2
        m.qkv_bias = bool(g("add_qkv_bias", True))
        m.rope_theta = 10000.0 * float(g("rope_ratio", 1.0))
    if mt in ("glm", "glm4"):
        # the HF port of GLM-4: interleaved rotary pairs on a fraction of the head, fused gate_up_proj
        m.rope_interleaved = True
        prf = float(g("partial_rotary_factor", None) or rp.get("partial_rotary_factor", 0.5) or 0.5)
        m.rotary_dim = int(m.head_dim * prf)
        m.qkv_bias = bool(g("attention_bias", True))
    if mt in ("internlm2", "internvl_chat", "internlmxcomposer2"):
        m.qkv_bias = bool(g("bias", False))
    if mt in ("minicpm", "minicpm3"):
        m.emb_scale = float(g("scale_emb", 1.0))
        depth = float(g("scale_depth", 1.0))
        m.residual_scale = depth / (m.num_layers ** 0.5) if depth != 1.0 else 1.0
        dmb = float(g("dim_model_base", m.hidden_size))
        m.logit_scale = dmb / m.hidden_size

    # ---- MoE ------------------------------------------------------------------------------
    ne = g("num_experts", None) or g("num_local_experts", None) or g("n_routed_experts", None) or 0
    if isinstance(ne, (list, tuple)):
        ne = ne[0] if ne else 0
    m.num_experts = int(ne or 0)
    if m.num_experts:
        m.num_experts_per_tok = int(g("num_experts_per_tok", g("moe_topk", 2)))
        mis = g("moe_intermediate_size", m.intermediate_size)
        m.moe_intermediate_size = int(mis[0] if isinstance(mis, (list, tuple)) else mis)
        m.norm_topk_prob = bool(g("norm_topk_prob", mt == "mixtral"))
        m.num_shared_experts = int(g("n_shared_experts", 0) or 0)
        sei = g("shared_expert_intermediate_size", 0) or 0
        if sei:
            m.num_shared_experts = max(m.num_shared_experts, 1)
            m.shared_expert_intermediate_size = int(sei)
            m.shared_expert_gate = mt == "qwen2_moe"
        elif m.num_shared_experts:
            m.shared_expert_intermediate_size = m.moe_intermediate_size * m.num_shared_experts
        m.first_k_dense_replace = int(g("first_k_dense_replace", 0) or 0)
        m.moe_layer_freq = int(g("moe_layer_freq", g("decoder_sparse_step", 1)) or 1)
        v3_like = mt in ("deepseek_v3", "deepseek_v32", "kimi_k2", "glm_moe_dsa")  # sigmoid routing even when the field is absent
        m.scoring_func = str(g("scoring_func", "sigmoid" if v3_like else "softmax"))
        m.n_group = int(g("n_group", 1) or 1)
        m.topk_group = int(g("topk_group", 1) or 1)
        m.routed_scaling_factor = float(g("routed_scaling_factor", 1.0) or 1.0)
        m.topk_method = str(g("topk_method", "noaux_tc" if v3_like else "greedy"))
        if mt.startswith("llama4"):
            # experts use intermediate_size, the dense layers and nothing else intermediate_size_mlp
            m.moe_intermediate_size = int(g("intermediate_size", m.moe_intermediate_size))
            m.intermediate_size = int(g("intermediate_size_mlp", m.intermediate_size))
            m.num_shared_experts, m.shared_expert_intermediate_size = 1, m.moe_intermediate_size
            m.moe_router = "llama4"
            ml = g("moe_layers", None)
            step = int(g("interleave_moe_layer_step", 1) or 1)
            m.moe_layers = [int(x) for x in ml] if ml is not None else list(range(step - 1, m.num_layers, step))
        mlt = g("mlp_layer_types", None)
        if mlt:  # explicit per-layer list of "dense" / "sparse" (GLM MoE)
            m.moe_layers = [i for i, t in enumerate(mlt) if str(t) == "sparse"]
            m.first_k_dense_replace = 0
        if mt.startswith("hunyuan"):
            tk = g("moe_topk", m.num_experts_per_tok)
            m.num_experts_per_tok = int(tk[0] if isinstance(tk, (list, tuple)) else tk)
            ne_ = g("num_experts", m.num_experts)
            m.num_experts = int(ne_[0] if isinstance(ne_, (list, tuple)) else ne_)
            m.moe_intermediate_size = m.intermediate_size  # the experts are full-width MLPs
            nse = g("num_shared_expert", 1)
            m.num_shared_experts = int(nse[0] if isinstance(nse, (list, tuple)) else nse) or 1
            m.shared_expert_intermediate_size = m.intermediate_size * m.num_shared_experts
            m.norm_topk_prob = True

    # ---- MLA ------------------------------------------------------------------------------
    if g("kv_lora_rank", None):
        m.use_mla = True
        m.q_lora_rank = int(g("q_lora_rank", 0) or 0)
        m.kv_lora_rank = int(g("kv_lora_rank"))
        m.qk_nope_head_dim = int(g("qk_nope_head_dim", 128))
        m.qk_rope_head_dim = int(g("qk_rope_head_dim", 64))
        m.v_head_dim = int(g("v_head_dim", 128))
        m.num_kv_heads = 1
        m.rope_interleaved = bool(g("rope_interleave", mt != "glm_moe_dsa"))
        if mt == "glm_moe_dsa":
            m.mla_norm_eps = 1e-6  # the transformers implementation keeps the default there
        if g("index_topk", None) and (mt in ("deepseek_v32", "glm_moe_dsa") or g("index_n_heads", None)):
            m.index_topk = int(g("index_topk"))
            m.index_n_heads = int(g("index_n_heads", 64))
            m.index_head_dim = int(g("index_head_dim", 128))
    m.num_nextn_predict_layers = int(g("num_nextn_predict_layers", 0) or 0)
    if g("start_layer", None) is not None:  # reference: models/bge_reranker_minicpm/bge_reranker_minicpm_config.h:19
        m.reranker_start_layer = int(g("start_layer"))
    m.num_register_token = int(g("num_register_token", 0) or 0)  # reference: models/common/common_config.h:36-37
    m.reg_token_id = int(g("reg_token_id", 0) or 0)
    m.quant = _quant(g("quantization_config", None))
    return m


def load_model_config(model_dir: str) -> ModelConfig:
    path = os.path.join(model_dir, "config.json")
    with open(path, "r", encoding="utf-8") as f:
        raw = json.load(f)
    # ModelOpt / TensorRT-LLM exports describe their quantisation in hf_quant_config.json:
    # {"quantization": {"quant_algo": "W4A8_AWQ", "group_size": 128, ...}}
    # (reference: utils/config/quant_config_parser.cpp:52-60)
    hq = os.path.join(model_dir, "hf_quant_config.json")
    if "quantization_config" not in raw and os.path.isfile(hq):
        with open(hq, "r", encoding="utf-8") as f:
            qd = json.load(f).get("quantization") or {}
        if qd.get("quant_algo"):
            raw["quantization_config"] = dict(qd, modules_to_not_convert=qd.get("exclude_modules") or [])
    cfg = model_config_from_dict(raw)
    # generation_config.json may name further end-of-sequence ids (Llama 3: <|eot_id|> next to <|end_of_text|>);
    # the reference adds them to every request's stop ids (python/ksana_llm/processor_op_base.py:74-90)
    gen = os.path.join(model_dir, "generation_config.json")
    if os.path.isfile(gen):
        try:
            with open(gen, "r", encoding="utf-8") as f:
                eos = json.load(f).get("eos_token_id")
        except (OSError, ValueError):
            eos = None
        extra = eos if isinstance(eos, (list, tuple)) else ([eos] if eos is not None else [])
        for t in extra:
            if int(t) not in cfg.eos_token_ids:
                cfg.eos_token_ids.append(int(t))
    return cfg


# ---- named synthetic configurations used by benchmarks and tests ---------------------------------

def tiny_llama_config() -> ModelConfig:
    return model_config_from_dict(dict(
        model_type="llama", hidden_size=256, num_hidden_layers=2, num_attention_heads=4, num_key_value_heads=4,
        intermediate_size=688, rms_norm_eps=1e-6, rope_theta=10000.0, vocab_size=32000,
        max_position_embeddings=2048, torch_dtype="float32", eos_token_id=2, bos_token_id=1))


def llama2_7b_config() -> ModelConfig:
    return model_config_from_dict(dict(
        model_type="llama", hidden_size=4096, num_hidden_layers=32, num_attention_heads=32, num_key_value_heads=32,
        intermediate_size=11008, rms_norm_eps=1e-5, rope_theta=10000.0, vocab_size=32000,
        max_position_embeddings=4096, torch_dtype="bfloat16", eos_token_id=2, bos_token_id=1))


def llama3_70b_config() -> ModelConfig:
    return model_config_from_dict(dict(
        model_type="llama", hidden_size=8192, num_hidden_layers=80, num_attention_heads=64, num_key_value_heads=8,
        intermediate_size=28672, rms_norm_eps=1e-5, rope_theta=500000.0, vocab_size=128256,
        max_position_embeddings=8192, torch_dtype="bfloat16", eos_token_id=128001, bos_token_id=128000))


def qwen3_32b_config(fp8_block: bool = True) -> ModelConfig:
    d = dict(model_type="qwen3", hidden_size=5120, num_hidden_layers=64, num_attention_heads=64,
             num_key_value_heads=8, head_dim=128, intermediate_size=25600, rms_norm_eps=1e-6, rope_theta=1000000.0,
             vocab_size=151936, max_position_embeddings=40960, torch_dtype="bfloat16", eos_token_id=151645)
    if fp8_block:
        d["quantization_config"] = dict(quant_method="fp8", weight_block_size=[128, 128], activation_scheme="dynamic")
    return model_config_from_dict(d)


def deepseek_v3_config(num_layers: int = 61, fp8_block: bool = True) -> ModelConfig:
    d = dict(model_type="deepseek_v3", hidden_size=7168, num_hidden_layers=num_layers, num_attention_heads=128,
             num_key_value_heads=128, intermediate_size=18432, moe_intermediate_size=2048, n_routed_experts=256,
             n_shared_experts=1, num_experts_per_tok=8, first_k_dense_replace=3, n_group=8, topk_group=4,
             scoring_func="sigmoid", topk_method="noaux_tc", norm_topk_prob=True, routed_scaling_factor=2.5,
             q_lora_rank=1536, kv_lora_rank=512, qk_nope_head_dim=128, qk_rope_head_dim=64, v_head_dim=128,
             rms_norm_eps=1e-6, rope_theta=10000.0, vocab_size=129280, max_position_embeddings=163840,
             num_nextn_predict_layers=1, torch_dtype="bfloat16", eos_token_id=1,
             rope_scaling=dict(type="yarn", factor=40, original_max_position_embeddings=4096, beta_fast=32,
                               beta_slow=1, mscale=1.0, mscale_all_dim=1.0))
    if fp8_block:
        d["quantization_config"] = dict(quant_method="fp8", weight_block_size=[128, 128], activation_scheme="dynamic")
    return model_config_from_dict(d)


def tiny_moe_config() -> ModelConfig:
    return model_config_from_dict(dict(
        model_type="mixtral", hidden_size=64, num_hidden_layers=2, num_attention_heads=4, num_key_value_heads=2,
        intermediate_size=96, num_local_experts=4, num_experts_per_tok=2, vocab_size=32000, rms_norm_eps=1e-6,
        max_position_embeddings=2048, torch_dtype="float32", eos_token_id=2, bos_token_id=1))


def tiny_moe_128_config() -> ModelConfig:
    """A small MoE whose shapes the CUDA kernels take (head_dim 128, hidden and expert widths multiples of 128)."""
    return model_config_from_dict(dict(
        model_type="mixtral", hidden_size=256, num_hidden_layers=2, num_attention_heads=2, num_key_value_heads=2,
        head_dim=128, intermediate_size=128, num_local_experts=4, num_experts_per_tok=2, vocab_size=32000,
        rms_norm_eps=1e-6, max_position_embeddings=2048, torch_dtype="bfloat16", eos_token_id=2, bos_token_id=1))


def molopel_config(width: int = 4096, layers: int = 32, ff: int = 12288, heads: int = 32, kv_heads: int = 8,
                   dim: int = 128, window: int = 1024, vocab: int = 32000) -> ModelConfig:
    """Molopel at the sizes of an ordinary decoder of that width: three windowed-attention + retention layers, then one
    of linear attention alone. The retention half has half as many heads with values twice as wide."""
    def decays(n):
        return [1.0 - 2.0 ** (-5.0 - 4.0 * i / max(n - 1, 1)) for i in range(n)]
    half = max(heads // 2, 1)
    parallel = dict(type="parallel", mlp=dict(kind="dense", ff=ff), mixer=dict(
        left=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=dim ** -0.5, bias_max=max(window // 2, 17),
                  mask=dict(size=window)),
        right=dict(heads=half, dim=dim, vdim=2 * dim, decay=decays(half), rot=dict(dims=dim, base=10000.0)),
        left_scale=0.5, right_scale=0.5))
    lightning = dict(type="lightning", mlp=None, mixer=dict(heads=heads, dim=dim, vdim=dim, decay=decays(heads)))
    return model_config_from_dict(dict(
        architecture="Molopel", embedding=dict(scale=1.0), norm=dict(eps=1e-6), vocab=vocab, width=width,
        logit_softcap=30.0, layers=[lightning if i % 4 == 3 else parallel for i in range(layers)], eos_token_id=2))


def tiny_molopel_config() -> ModelConfig:
    cfg = molopel_config(width=128, layers=4, ff=192, heads=4, kv_heads=2, dim=32, window=24)
    cfg.torch_dtype = "float32"
    return cfg


def givirax_config(width: int = 4096, layers: int = 16, ff: int = 12288, experts: int = 16, top: int = 2,
                   expert_ff: int = 3072, heads: int = 32, kv_heads: int = 8, dim: int = 128, window: int = 1024,
                   keep_first: int = 4, loop: Optional[Dict[str, int]] = None, vocab: int = 32000,
                   max_positions: int = 8192) -> ModelConfig:
    """Givirax at the sizes of an ordinary decoder of that width: dense and routed feed-forwards in turn."""
    mixer = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=dim ** -0.5,
                 mask=dict(size=window, keep_first=keep_first))
    dense = dict(kind="dense", ff=ff)
    moe = dict(kind="moe", expert=dict(ff=expert_ff), router=dict(experts=experts, top=top))
    return model_config_from_dict(dict(
        architecture="Givirax", embedding=dict(scale=1.0), norm=dict(eps=1e-6), vocab=vocab, width=width,
        max_positions=max_positions, loop=loop, eos_token_id=2,
        layers=[dict(type="attention", mixer=mixer, mlp=moe if i % 2 else dense) for i in range(layers)]))


def tiny_givirax_config() -> ModelConfig:
    cfg = givirax_config(width=128, layers=3, ff=192, experts=6, expert_ff=48, heads=4, kv_heads=2, dim=32, window=24,
                         keep_first=2, loop=dict(start=0, stop=2, times=3), max_positions=512)
    cfg.torch_dtype = "float32"
    return cfg


def ladusun_config(width: int = 4096, layers: int = 8, ff: int = 12288, experts: int = 16, top: int = 2,
                   expert_ff: int = 3072, heads: int = 32, kv_heads: int = 8, dim: int = 128, rank: int = 512,
                   rot_dim: int = 64, streams: int = 4, vocab: int = 32000, groups: int = 4, keep: int = 2) -> ModelConfig:
    """Ladusun at the sizes of an ordinary decoder of that width: latent attention, the recurrence, attention, and every
    second attention layer reading the one before it; dense and routed feed-forwards in turn."""
    latent = dict(type="latent_attention", mixer=dict(
        heads=heads, dim=dim, rot_dim=rot_dim, vdim=dim, kv_rank=rank, scale=(dim + rot_dim) ** -0.5,
        rot=dict(dims=rot_dim, base=1e5, scaling=dict(factor=4.0, original=4096, fast=32.0, slow=1.0))))
    rec = dict(type="rglru", mixer=dict(width=width, blocks=max(width // 128, 1), conv=4))
    attn = dict(type="attention", mixer=dict(
        heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=dim ** -0.5, softcap=50.0,
        rot=dict(dims=dim, base=5e5, scaling=dict(factor=8.0, low=1.0, high=4.0, original=8192))))
    out, owner = [], None
    for i in range(layers):
        entry = json.loads(json.dumps((latent, rec, attn, rec)[i % 4]))
        if entry["type"] == "attention":
            if owner is None:
                owner = i
            else:
                entry["mixer"]["kv_from"], owner = owner, None
        entry["mlp"] = dict(kind="dense", ff=ff) if i % 2 == 0 else dict(
            kind="moe", expert=dict(ff=expert_ff, limit=7.0),
            router=dict(experts=experts, top=top, groups=dict(count=groups, keep=keep)))
        out.append(entry)
    return model_config_from_dict(dict(
        architecture="Ladusun", embedding=dict(scale=1.0), norm=dict(eps=1e-6), vocab=vocab, width=width, streams=streams,
        layers=out, eos_token_id=2))


def tiny_ladusun_config() -> ModelConfig:
    cfg = ladusun_config(width=128, layers=7, ff=192, experts=6, expert_ff=48, heads=4, kv_heads=2, dim=32, rank=48,
                         rot_dim=16, streams=3, groups=3)
    cfg.torch_dtype = "float32"
    return cfg


def vibunex_config(width: int = 4096, layers: int = 8, experts: int = 16, top: int = 2, expert_ff: int = 4096,
                   shared_ff: int = 4096, heads: int = 32, kv_heads: int = 8, dim: int = 128, mix_heads: int = 64,
                   mix_dim: int = 64, vocab: int = 32000) -> ModelConfig:
    """Vibunex at the sizes of an ordinary decoder of that width."""
    layer = dict(type="parallel", mixer=dict(
        left=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=dim ** -0.5, rot=dict(
            dims=dim // 2, base=5e5, scaling=dict(factor=4.0, original=8192, fast=32.0, slow=1.0))),
        right=dict(heads=mix_heads, dim=mix_dim), left_scale=0.7, right_scale=0.7),
        mlp=dict(kind="moe", expert=dict(ff=expert_ff), router=dict(experts=experts, top=top, scale=1.5),
                 shared=dict(ff=shared_ff)))
    return model_config_from_dict(dict(
        architecture="Vibunex", norm=dict(eps=1e-6), vocab=vocab, width=width, residual_mult=0.5,
        layers=[json.loads(json.dumps(layer)) for _ in range(layers)], eos_token_id=2))


def tiny_vibunex_config() -> ModelConfig:
    cfg = vibunex_config(width=128, layers=3, experts=6, expert_ff=48, shared_ff=80, heads=4, kv_heads=2, dim=32,
                         mix_heads=3, mix_dim=24)
    cfg.torch_dtype = "float32"
    return cfg


NAMED_CONFIGS = {
    "tiny-vibunex": tiny_vibunex_config,
    "vibunex": vibunex_config,
    "tiny-ladusun": tiny_ladusun_config,
    "ladusun": ladusun_config,
    "tiny-givirax": tiny_givirax_config,
    "givirax": givirax_config,
    "tiny-molopel": tiny_molopel_config,
    "molopel": molopel_config,
    "tiny-llama": tiny_llama_config,
    "tiny-moe": tiny_moe_config,
    "tiny-moe-128": tiny_moe_128_config,
    "llama-2-7b": llama2_7b_config,
    "llama-3-70b": llama3_70b_config,
    "qwen3-32b-fp8": qwen3_32b_config,
    "deepseek-v3-fp8": deepseek_v3_config,
}
