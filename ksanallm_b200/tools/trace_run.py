"""Replays recorded token ids through a model and writes logits: ``bin/trace_run --model DIR --dtype bfloat16|float32
--out DIR --max-tokens N``.

Steps come from standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

Every entry brings the next tokens of one request and the places among them whose logits are wanted; "end" names the
requests that are over after the step. A step with wanted logits writes OUT/<step>.f32 (fp32, [wanted, vocab], in the
order of the entries); after each step a line "done <step>" is printed. All the entries of a step run as one batch
through :meth:`LLMEngine.replay`, i.e. the scheduler, cache, state slots and kernels that generation uses.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, Optional, Sequence

import torch

LIVE_REQUESTS = 4  # requests that may be live at the same time


def build_engine(model_dir: str, dtype: torch.dtype, max_tokens: int, device: str = "cuda"):
    from ..config.model_config import load_model_config
    from ..config.schema import parse_serving_config
    from ..engine.llm_engine import LLMEngine
    from ..models.loader import load_model_weights
    from ..models.registry import resolve_family
    from ..models.transformer import TransformerModel

    cfg = load_model_config(model_dir)
    if device.startswith("cuda"):
        from ..ops import cuda
        cuda.lib(resolve_family(cfg.model_type, model_dir) or "")
    weights = load_model_weights(cfg, model_dir, device=device, dtype=dtype)
    # requests hold whole blocks; max_tokens counts each request rounded up to a multiple of 64
    serving = parse_serving_config({"setting": {"batch_scheduler": {
        "max_batch_size": LIVE_REQUESTS, "max_step_tokens": max_tokens, "max_token_len": max_tokens + 1,
        "enable_auto_prefix_cache": False}}})
    model = TransformerModel(cfg, weights, max_positions=max_tokens)
    block = serving.setting.block_manager.block_token_num
    if cfg.use_mla and block == 16:
        block = 64
    return LLMEngine(model, serving, num_blocks=(max_tokens + block - 1) // block, num_host_blocks=0,
                     num_state_slots=LIVE_REQUESTS)


def run(engine, out_dir: str, lines, emit) -> None:
    ids: Dict[str, int] = {}
    fresh = 0
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            if e["id"] not in ids:
                fresh += 1
                ids[e["id"]] = fresh
            entries.append((ids[e["id"]], e["tokens"], e.get("want", [])))
        logits = engine.replay(entries, [ids.pop(x) for x in step.get("end", []) if x in ids])
        if logits.shape[0]:
            path = os.path.join(out_dir, f"{step['step']}.f32")
            with open(path, "wb") as f:
                f.write(logits.contiguous().numpy().astype("<f4").tobytes())
        emit(f"done {step['step']}")


def main(argv: Optional[Sequence[str]] = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay given token ids and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and the weights")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits files")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens live requests hold at any time")
    ap.add_argument("--device", default="cuda")
    a = ap.parse_args(argv)
    torch.backends.cuda.matmul.allow_tf32 = False
    torch.backends.cudnn.allow_tf32 = False
    engine = build_engine(a.model, getattr(torch, a.dtype), a.max_tokens, a.device)

    def emit(text: str) -> None:
        sys.stdout.write(text + "\n")
        sys.stdout.flush()

    run(engine, a.out, sys.stdin, emit)
    return 0


if __name__ == "__main__":
    sys.exit(main())
