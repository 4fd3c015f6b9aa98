"""Prefill and decode throughput of the designs described layer by layer, at layer sizes of real models, each beside the
closest other model of the same width, heads and depth. Random weights, bf16, one GPU; every number comes from
``LLMEngine.step()``.

    python bench.py --throughput molopel
    python bench.py --throughput givirax
    python bench.py --throughput ladusun
    python bench.py --throughput vibunex

Molopel: beside the dense model (Qwen3 blocks: QK norm, grouped-query attention, SwiGLU) whose feed-forward is as wide as
makes the parameter counts equal. Givirax (half of its layers run twice): beside Qwen3-MoE blocks, dense and routed in
turn, as many layers as Givirax has runs, with the same experts and a gated feed-forward of the same number of weights.
Ladusun (four residual streams): beside DeepSeek blocks (latent attention, routed experts) of the same width, depth, heads
and latent size, dense and routed in turn, with the same experts and a gated feed-forward of the same number of weights.
Vibunex: beside two models, each closest in one respect: Qwen2-MoE blocks (grouped-query attention, routed and shared
experts) with the same experts and the same number of feed-forward weights, and Molopel blocks (attention to all keys beside
retention with as many channels) with a dense feed-forward of as many weights as a Vibunex token meets.

prefill: prompts of 4096 tokens, 8192 tokens a step. decode: 128 sequences behind prompts of 1024 tokens, one token each
per step. Weights and caches are larger than L2, so each step starts cold. CUDA events around the timed steps; the host
clock around the same steps is given beside it.
"""
from __future__ import annotations

import json
import time

import torch

from ksanallm_b200.config.model_config import (givirax_config, ladusun_config, model_config_from_dict, molopel_config,
                                               vibunex_config)
from ksanallm_b200.config.schema import parse_serving_config
from ksanallm_b200.engine.llm_engine import LLMEngine
from ksanallm_b200.engine.sampling_params import SamplingParams
from ksanallm_b200.models.loader import load_model_weights
from ksanallm_b200.models.transformer import TransformerModel
from ksanallm_b200.ops import cuda

# width, depth, feed-forward, heads, key / value heads, window
SIZES = [(2048, 8, 6144, 16, 4, 1024), (4096, 8, 12288, 32, 8, 1024), (8192, 4, 24576, 64, 8, 2048)]
# width, depth, feed-forward, experts, experts per token, expert width, heads, key / value heads, window
GIVIRAX_SIZES = [(2048, 8, 8192, 16, 2, 2048, 16, 4, 1024), (4096, 8, 16384, 16, 2, 4096, 32, 8, 1024),
                 (8192, 4, 32768, 8, 2, 8192, 64, 8, 2048)]
# width, depth, feed-forward, experts, experts per token, expert width, heads, key / value heads, latent size
LADUSUN_SIZES = [(2048, 8, 8192, 16, 2, 2048, 16, 4, 512), (4096, 8, 16384, 16, 2, 4096, 32, 8, 512),
                 (8192, 4, 32768, 8, 2, 8192, 64, 8, 512)]
# width, depth, experts, experts per token, expert width, shared expert's width, heads, key / value heads, time-mixing heads of 64
VIBUNEX_SIZES = [(2048, 8, 16, 2, 2048, 2048, 16, 4, 32), (4096, 8, 16, 2, 4096, 4096, 32, 8, 64),
                 (8192, 4, 8, 2, 8192, 8192, 64, 8, 128)]
PROMPT, STEP_TOKENS = 4096, 8192
BATCH, CONTEXT, DECODE_STEPS = 128, 1024, 40


def parameters(weights) -> int:
    return sum(w.numel() for k, w in weights.items() if k.startswith("model.layers."))


def dense_config(width, depth, ff, heads, kv_heads):
    return model_config_from_dict(dict(
        model_type="qwen3", hidden_size=width, num_hidden_layers=depth, num_attention_heads=heads,
        num_key_value_heads=kv_heads, head_dim=128, intermediate_size=ff, rms_norm_eps=1e-6, vocab_size=32000,
        max_position_embeddings=8192, torch_dtype="bfloat16", eos_token_id=2, tie_word_embeddings=True))


def moe_config(width, depth, ff, experts, top, expert_ff, heads, kv_heads):
    return model_config_from_dict(dict(
        model_type="qwen3_moe", hidden_size=width, num_hidden_layers=depth, num_attention_heads=heads,
        num_key_value_heads=kv_heads, head_dim=128, intermediate_size=ff, moe_intermediate_size=expert_ff,
        num_experts=experts, num_experts_per_tok=top, norm_topk_prob=True, rms_norm_eps=1e-6, vocab_size=32000,
        mlp_layer_types=["sparse" if i % 2 else "dense" for i in range(depth)],
        max_position_embeddings=8192, torch_dtype="bfloat16", eos_token_id=2))


def shared_moe_config(width, depth, experts, top, expert_ff, shared_ff, heads, kv_heads):
    return model_config_from_dict(dict(
        model_type="qwen2_moe", hidden_size=width, num_hidden_layers=depth, num_attention_heads=heads,
        num_key_value_heads=kv_heads, head_dim=128, intermediate_size=shared_ff, moe_intermediate_size=expert_ff,
        shared_expert_intermediate_size=shared_ff, num_experts=experts, num_experts_per_tok=top, norm_topk_prob=False,
        rms_norm_eps=1e-6, vocab_size=32000, decoder_sparse_step=1, max_position_embeddings=8192, torch_dtype="bfloat16",
        eos_token_id=2))


def retention_config(width, depth, ff, heads, kv_heads, channels):
    """Molopel whose layers all have attention to every key beside retention over ``channels``."""
    cfg = molopel_config(width, 1, ff, heads, kv_heads, 128, 8192)
    raw = json.loads(json.dumps(cfg.raw))
    layer = raw["layers"][0]
    layer["mixer"]["right"].update(heads=channels // 64, dim=64, vdim=64, decay=[0.99] * (channels // 64), rot=dict(dims=64, base=10000.0))
    raw["layers"] = [layer] * depth
    return model_config_from_dict(raw)


def mla_config(width, depth, ff, experts, top, expert_ff, heads, rank):
    return model_config_from_dict(dict(
        model_type="deepseek_v2", hidden_size=width, num_hidden_layers=depth, num_attention_heads=heads,
        num_key_value_heads=heads, intermediate_size=ff, moe_intermediate_size=expert_ff, n_routed_experts=experts,
        num_experts_per_tok=top, n_group=4, topk_group=2, topk_method="group_limited_greedy", scoring_func="softmax",
        norm_topk_prob=True, kv_lora_rank=rank, qk_nope_head_dim=128, qk_rope_head_dim=64, v_head_dim=128,
        mlp_layer_types=["sparse" if i % 2 else "dense" for i in range(depth)], rms_norm_eps=1e-6, vocab_size=32000,
        max_position_embeddings=8192, torch_dtype="bfloat16", eos_token_id=2, tie_word_embeddings=True))


def build(cfg):
    weights = load_model_weights(cfg, synthetic_seed=0, device="cuda:0", dtype=torch.bfloat16)
    n = parameters(weights)
    return TransformerModel(cfg, weights, max_positions=8192), n


def engine_of(model):
    serving = parse_serving_config({"setting": {"batch_scheduler": {
        "max_batch_size": BATCH, "max_step_tokens": STEP_TOKENS, "max_token_len": 8192, "enable_auto_prefix_cache": False}}})
    blocks = BATCH * (CONTEXT + DECODE_STEPS + 64) // 16 + 2048
    return LLMEngine(model, serving, num_blocks=blocks, num_host_blocks=0)


def timed(fn) -> tuple:
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    t0 = time.perf_counter()
    e0.record()
    fn()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / 1e3, time.perf_counter() - t0


def drain(eng) -> int:
    steps = 0
    while eng.has_unfinished():
        eng.step()
        steps += 1
    return steps


def measure(model) -> dict:
    gen = torch.Generator().manual_seed(1)
    vocab = model.cfg.vocab_size

    def prompt(n):
        return torch.randint(3, vocab, (n,), generator=gen).tolist()

    eng = engine_of(model)
    one = SamplingParams(topk=1, max_new_tokens=1, ignore_eos=True)
    out = {}
    for wave in range(2):  # the first warms up
        for _ in range(8):
            eng.add_request(prompt(PROMPT), one)
        dev, host = timed(lambda: drain(eng))
    out["prefill_tok_s"] = round(8 * PROMPT / dev)
    out["prefill_tok_s_host_clock"] = round(8 * PROMPT / host)
    many = SamplingParams(topk=1, max_new_tokens=DECODE_STEPS + 8, ignore_eos=True)
    for _ in range(BATCH):
        eng.add_request(prompt(CONTEXT), many)
    while eng.sched.num_waiting or any(not s.output_tokens for r in eng.requests.values() for s in r.seqs):
        eng.step()
    for _ in range(3):
        eng.step()
    before = cuda.launch_count
    done = [0]

    def run():
        for _ in range(DECODE_STEPS - 20):
            done[0] += eng.step()
    dev, host = timed(run)
    out["decode_tok_s"] = round(done[0] / dev)
    out["decode_tok_s_host_clock"] = round(done[0] / host)
    out["decode_ms_per_step"] = round(dev / (DECODE_STEPS - 20) * 1e3, 3)
    out["decode_batch"] = round(done[0] / (DECODE_STEPS - 20))
    out["launches_per_step"] = round((cuda.launch_count - before) / (DECODE_STEPS - 20))
    drain(eng)
    if cuda.read_error():
        out["kernel_error_word"] = True
    return out


def run_givirax() -> None:
    for width, depth, ff, experts, top, expert_ff, heads, kv, window in GIVIRAX_SIZES:
        loop = dict(start=depth // 4, stop=depth // 4 + depth // 2, times=2)
        runs = depth + depth // 2
        rows = {}
        # the other model's layers are its own: the kinds of feed-forward follow the order of Givirax' runs
        for name, cfg in (("givirax", givirax_config(width, depth, ff, experts, top, expert_ff, heads, kv, 128, window, 4, loop)),
                          ("moe", moe_config(width, runs, ff * 2 // 3 // 128 * 128, experts, top, expert_ff, heads, kv))):
            model, n = build(cfg)
            rows[name] = dict(parameters_m=round(n / 1e6), **measure(model))
            del model
            torch.cuda.empty_cache()
        print(json.dumps(dict(metric="throughput", design="givirax", width=width, layers=depth, layer_runs=runs, ff=ff,
                              experts=experts, top=top, expert_ff=expert_ff, heads=heads, kv_heads=kv, window=window,
                              keep_first=4, dtype="bf16", data="synthetic", **rows)), flush=True)


def run_ladusun() -> None:
    for width, depth, ff, experts, top, expert_ff, heads, kv, rank in LADUSUN_SIZES:
        rows = {}
        for name, cfg in (("ladusun", ladusun_config(width, depth, ff, experts, top, expert_ff, heads, kv, 128, rank)),
                          ("latent_moe", mla_config(width, depth, ff * 2 // 3 // 128 * 128, experts, top, expert_ff, heads, rank))):
            model, n = build(cfg)
            rows[name] = dict(parameters_m=round(n / 1e6), **measure(model))
            del model
            torch.cuda.empty_cache()
        print(json.dumps(dict(metric="throughput", design="ladusun", width=width, layers=depth, ff=ff, experts=experts, top=top,
                              expert_ff=expert_ff, heads=heads, kv_heads=kv, rank=rank, streams=4, dtype="bf16",
                              data="synthetic", **rows)), flush=True)


def run_vibunex() -> None:
    for width, depth, experts, top, expert_ff, shared_ff, heads, kv, mix in VIBUNEX_SIZES:
        rows = {}
        third = lambda n: n * 2 // 3 // 128 * 128  # noqa: E731  (a gated feed-forward has three matrices)
        for name, cfg in (
                ("vibunex", vibunex_config(width, depth, experts, top, expert_ff, shared_ff, heads, kv, 128, mix, 64)),
                ("shared_moe", shared_moe_config(width, depth, experts, top, third(expert_ff), third(shared_ff), heads, kv)),
                ("molopel", retention_config(width, depth, third(top * expert_ff + shared_ff), heads, kv, mix * 64))):
            model, n = build(cfg)
            rows[name] = dict(parameters_m=round(n / 1e6), **measure(model))
            del model
            torch.cuda.empty_cache()
        print(json.dumps(dict(metric="throughput", design="vibunex", width=width, layers=depth, experts=experts, top=top,
                              expert_ff=expert_ff, shared_ff=shared_ff, heads=heads, kv_heads=kv, mix_heads=mix, dtype="bf16",
                              data="synthetic", **rows)), flush=True)


def run(design: str) -> None:
    if design == "vibunex":
        return run_vibunex()
    if design == "givirax":
        return run_givirax()
    if design == "ladusun":
        return run_ladusun()
    assert design == "molopel"
    for width, depth, ff, heads, kv, window in SIZES:
        rows = {}
        model, n = build(molopel_config(width, depth, ff, heads, kv, 128, window))
        rows["molopel"] = dict(parameters_m=round(n / 1e6), **measure(model))
        del model
        torch.cuda.empty_cache()
        attn = depth * width * 128 * 2 * (heads + kv)
        dense_ff = max((n - attn) // (3 * depth * width) // 128 * 128, 128)
        model, n = build(dense_config(width, depth, dense_ff, heads, kv))
        rows["dense"] = dict(parameters_m=round(n / 1e6), **measure(model))
        del model
        torch.cuda.empty_cache()
        print(json.dumps(dict(metric="throughput", design=design, width=width, layers=depth, ff=ff, dense_ff=dense_ff,
                              heads=heads, kv_heads=kv, window=window, dtype="bf16", data="synthetic", **rows)), flush=True)


if __name__ == "__main__":
    run("molopel")
