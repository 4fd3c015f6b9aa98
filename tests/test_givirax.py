"""Givirax on the CPU path: mechanisms alone, whole models through the engine's own step function against the plain
oracle, generation through the scheduler, and the command-line replay."""
import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import givirax_cases as C
import givirax_oracle as O
import replay_cases as R
from givirax_cases_attention import check
from ksanallm_b200.config.model_config import load_model_config, model_config_from_dict
from ksanallm_b200.config.schema import parse_serving_config
from ksanallm_b200.engine.llm_engine import LLMEngine
from ksanallm_b200.engine.sampling_params import SamplingParams
from ksanallm_b200.models.loader import load_model_weights
from ksanallm_b200.models.registry import resolve_family
from ksanallm_b200.models.transformer import TransformerModel
from ksanallm_b200.ops import reference as ref

REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    return {n: C.Case(tmp_path_factory.mktemp(n), n) for n in C.CASES}


# ---- mechanisms -----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("window,keep", [(1, 0), (1, 1), (16, 0), (17, 5), (40, 16), (33, 130), (300, 3)])
def test_window_and_first_token_edges(window, keep):
    check(torch.float32, "cpu", window, keep)


def test_grouped_heads_read_their_own_key_head():
    check(torch.float32, "cpu", 23, 4, h=6, hk=3, d=20)


@pytest.mark.parametrize("experts,top,cols", [(5, 2, 8), (1, 1, 8), (9, 9, 16), (40, 3, 40)])
def test_router(experts, top, cols):
    g = torch.Generator().manual_seed(experts)
    z = torch.randn(30, cols, generator=g)
    z[:, experts:] = 100.0  # padding columns are no experts, however large
    b = torch.randn(experts, generator=g)
    ids, w = ref.moe_topk(z, experts, top, b)
    for t in range(30):
        want, ww = O.route((z[t, :experts] + b).double(), top)
        assert ids[t].tolist() == want
        assert (w[t].double() - ww).abs().max() < 1e-6


def test_router_weights_ignore_experts_that_are_not_chosen():
    z = torch.tensor([[5.0, 4.0, 4.999, -3.0]])
    ids, w = ref.moe_topk(z, 4, 2)
    assert ids.tolist() == [[0, 2]] and float(w.sum()) == pytest.approx(1.0)
    assert float(w[0, 0] / w[0, 1]) == pytest.approx(2.718281828 ** 0.001, rel=1e-5)


def test_stream_norm_takes_every_term():
    g = torch.Generator().manual_seed(3)
    T, H, k = 4, 24, 2
    x, start, rows = (torch.randn(T, H, generator=g) for _ in range(3))
    vec, w, y = torch.randn(H, generator=g), torch.randn(H, generator=g), torch.randn(T * k, H, generator=g)
    pos, wts = torch.randperm(T * k, generator=g).int(), torch.rand(T, k, generator=g)
    pos[3] = -1
    out = torch.empty_like(start)
    got = ref.stream_norm(x, w, 1e-5, False, start, out, None, rows, vec, (y, pos, wts))
    v = start + x + rows + vec
    for t in range(T):
        for j in range(k):
            p = int(pos[t * k + j])
            if p >= 0:
                v[t] += wts[t, j] * y[p]
    assert (out - v).abs().max() < 1e-5
    assert (got - O.rms_norm(v, w, 1e-5)).abs().max() < 1e-5


def test_layer_runs():
    runs = lambda n, loop: model_config_from_dict(C.model(8, 9, [C.layer(1, 1, 8, 4, 0, 1.0)] * n, loop=loop)).layer_runs()  # noqa: E731
    for n, loop in ((4, None), (4, dict(start=1, stop=3, times=3)), (3, dict(start=0, stop=3, times=2)),
                    (3, dict(start=2, stop=3, times=4)), (2, dict(start=0, stop=1, times=1))):
        assert runs(n, loop) == list(O.layer_runs(n, loop))


# ---- configuration and loading ------------------------------------------------------------------------------------
def test_configuration(cases):
    cfg = load_model_config(cases["odd"].dir)
    assert resolve_family(cfg.model_type) == "givirax" and not cfg.has_state
    assert [(l.attn.window, l.attn.keep_first) for l in cfg.layers] == [(7, 3), (20, 17), (33, 1), (50, 0)]
    assert [l.ff for l in cfg.layers] == [76, 0, 0, 0]
    assert [(l.moe.experts, l.moe.top, l.moe.ff) if l.moe else None for l in cfg.layers] == [None, (5, 3, 22), None, (11, 1, 13)]
    assert [l.kv_width for l in cfg.layers] == [20, 56, 72, 24]
    for change in (lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mixer"].update(vdim=24),
                   lambda c: c["layers"][0]["mixer"].update(kv_heads=2), lambda c: c["loop"].update(stop=5),
                   lambda c: c["layers"][1]["mlp"]["router"].update(top=6), lambda c: c["layers"][1]["mlp"].update(kind="x")):
        bad = copy.deepcopy(C.ODD)
        change(bad)
        with pytest.raises(ValueError):
            model_config_from_dict(bad)


@pytest.mark.parametrize("name", ["l0.mix.k", "l0.mlp.down", "l1.mlp.e4.up", "l1.mlp.router.b", "loop.step", "pos", "head"])
def test_missing_tensor_is_named(cases, tmp_path, name):
    w = dict(cases["odd"].w)
    del w[name]
    O.write_model(tmp_path, C.ODD, w)
    canonical = {"l0.mix.k": "k", "l0.mlp.down": "ff.down", "l1.mlp.e4.up": "experts.4.up_proj", "loop.step": "loop.step",
                 "l1.mlp.router.b": "gate.bias", "pos": "embed_positions", "head": "lm_head"}[name]
    with pytest.raises(KeyError, match=canonical):
        cfg = load_model_config(str(tmp_path))
        TransformerModel(cfg, load_model_weights(cfg, str(tmp_path), dtype=torch.float32))


def test_one_cache_per_run_of_keys_alone(cases):
    cfg = load_model_config(cases["odd"].dir)
    model = TransformerModel(cfg, load_model_weights(cfg, cases["odd"].dir, dtype=torch.float32))
    caches = model.allocate_kv_cache(3, 16)
    assert [tuple(c.shape) for c in caches] == [(3, 16 * w) for w in [20, 56, 72, 56, 72, 56, 72, 24]]
    assert model.kv_block_bytes(16) == 4 * 16 * sum([20, 56, 72, 56, 72, 56, 72, 24])
    assert model.layers[1].in_proj.weight.data_ptr() == model.layers[3].in_proj.weight.data_ptr()


def test_what_it_does_not_combine_with(cases):
    from ksanallm_b200.parallel.comm import TPGroup
    cfg = load_model_config(cases["odd"].dir)
    w = load_model_weights(cfg, cases["odd"].dir, dtype=torch.float32)
    with pytest.raises(NotImplementedError):
        TransformerModel(cfg, w, TPGroup(0, 2, None, torch.device("cpu"), use_fused=False))
    serving = parse_serving_config({"setting": {"global": {"pipeline_para_size": 2}}})
    with pytest.raises(NotImplementedError):
        LLMEngine(TransformerModel(cfg, w), serving, num_blocks=8, num_host_blocks=0)


# ---- whole models ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", list(C.CASES))
def test_residual_stream_after_each_run(cases, name):
    """Run by run: the stream is the oracle's, up to what comes ahead of the next pass."""
    case = cases[name]
    toks = case.tokens(40, 2)
    want = []
    O.forward(case.cfg, case.w64, toks, want)
    model, seen = case.engine(torch.float32, 64, "cpu").model, []
    eng = case.engine(torch.float32, 64, "cpu")
    for layer in eng.model.layers:
        def hook(h, residual, meta, cache, nw, nb=None, start=None, inner=layer.forward):
            y = inner(h, residual, meta, cache, nw, nb, start)
            r = residual.clone()
            if start is not None:
                r = r - start.step - (meta.start if start.add_start else 0)
            seen.append(r)
            return y
        layer.forward = hook
    eng.replay([(1, toks, [])])
    assert len(seen) == len(want) == len(model.layers)
    for got, w in zip(seen, want):
        assert (got.double() - w).abs().max() < 2e-5 * w.abs().max()


@pytest.mark.parametrize("name", list(C.CASES))
def test_portions(cases, name):
    R.run_portions(cases[name], cases[name].engine(torch.float32, 192, "cpu"), 2e-5)


@pytest.mark.parametrize("name", list(C.CASES))
def test_batches_and_reuse(cases, name):
    R.run_batches(cases[name], cases[name].engine(torch.float32, 64 * 7, "cpu"), 2e-5)


def test_long_decode(cases):
    R.run_long_decode(cases["odd"], cases["odd"].engine(torch.float32, 320, "cpu"), 2e-5)


def test_bf16_storage(cases):
    R.run_portions(cases["even"], cases["even"].engine(torch.bfloat16, 192, "cpu"), 6e-2)


@pytest.mark.parametrize("mistake", ["window", "first tokens", "one first token more", "position", "step", "start", "router",
                                     "top", "scale", "shared values"])
def test_the_comparison_would_show(cases, mistake, monkeypatch):
    """Small mistakes in the oracle move its logits by far more than the tolerance of these tests."""
    case = cases["odd"]
    cfg, w = copy.deepcopy(case.cfg), dict(case.w64)
    mask = cfg["layers"][1]["mixer"]["mask"]
    if mistake == "window":
        mask["size"] += 1
    elif mistake == "first tokens":
        mask["keep_first"] -= 1
    elif mistake == "one first token more":
        mask["keep_first"] += 1
    elif mistake == "position":
        w["pos"] = torch.roll(w["pos"], 1, 0)
    elif mistake == "step":
        w["loop.step"] = torch.roll(w["loop.step"], 1, 0)
    elif mistake == "start":
        monkeypatch.setattr(O, "layer_runs", lambda n, loop: [(i, 0 if i == 1 else None) for i in (0, 1, 2, 1, 2, 1, 2, 3)])
    elif mistake == "router":
        w["l1.mlp.router.b"] = torch.zeros_like(w["l1.mlp.router.b"])
    elif mistake == "top":
        cfg["layers"][1]["mlp"]["router"]["top"] = 2
    elif mistake == "scale":
        cfg["layers"][2]["mixer"]["scale"] *= 1.01
    elif mistake == "shared values":
        inner = O.shared_kv_attention
        monkeypatch.setattr(O, "shared_kv_attention", lambda q, k, *a: inner(q, k, *a) * 1.001)
    toks = case.tokens(90, 4)
    good = case.logits(toks)
    bad = O.forward(cfg, w, toks)
    rms = ((good - bad) ** 2).mean(1).sqrt() / good.std()
    assert float(rms[45:].max()) > 20 * 2e-5


# ---- generation through the scheduler -----------------------------------------------------------------------------------
def serve(case, n_blocks=64, host_blocks=0, device="cpu", dtype=torch.float32, **bs):
    cfg = load_model_config(case.dir)
    setting = dict(max_batch_size=4, max_step_tokens=256, max_token_len=512)
    setting.update(bs)
    serving = parse_serving_config({"setting": {"batch_scheduler": setting}})
    model = TransformerModel(cfg, load_model_weights(cfg, case.dir, device=device, dtype=dtype))
    return LLMEngine(model, serving, num_blocks=n_blocks, num_host_blocks=host_blocks)


def greedy_check(case, eng, lens, new, seed=50, **params):
    prompts = [case.tokens(n, seed + n) for n in lens]
    reqs = eng.generate(prompts, SamplingParams(topk=1, max_new_tokens=new, ignore_eos=True, **params))
    for p, r in zip(prompts, reqs):
        assert r.output_token_ids[0] == O.greedy(case.cfg, case.w64, p, new), len(p)
    return eng


@pytest.mark.parametrize("bs", [dict(), dict(split_fuse_token_num=9), dict(enable_async=True), dict(max_step_tokens=24)])
def test_greedy_generation(cases, bs):
    greedy_check(cases["odd"], serve(cases["odd"], **bs), [1, 2, 30, 17, 41, 8], 8)


def test_shared_prefixes_are_reused(cases):
    """Cached blocks hold keys of positions counted from the sequence's start: equal prefixes may share them."""
    case = cases["odd"]
    eng = serve(case, enable_auto_prefix_cache=True)
    greedy_check(case, eng, [50], 4)
    assert eng.cache.stats.prefix_hit_tokens == 0
    greedy_check(case, eng, [50], 4)
    prompt = case.tokens(50, 100)[:40] + case.tokens(15, 9)
    r = eng.generate([prompt], SamplingParams(topk=1, max_new_tokens=4, ignore_eos=True))[0]
    assert r.output_token_ids[0] == O.greedy(case.cfg, case.w64, prompt, 4)
    assert eng.cache.stats.prefix_hit_tokens >= 48 + 32


def test_speculative_drafts(cases):
    """Verified drafts: steps of several tokens per sequence behind cached keys."""
    case = cases["flat"]
    eng = serve(case, enable_speculative_decoding=True)
    prompt = case.tokens(6, 3) * 5
    for _ in range(2):
        r = eng.generate([prompt], SamplingParams(topk=1, max_new_tokens=12, ignore_eos=True))[0]
        assert r.output_token_ids[0] == O.greedy(case.cfg, case.w64, prompt, 12)


@pytest.mark.parametrize("mode", ["swap", "recompute"])
def test_preemption(cases, mode):
    case = cases["odd"]
    eng = serve(case, n_blocks=7, host_blocks=16 if mode == "swap" else 0, preempt_mode=0 if mode == "swap" else 1,
                launch_block_threshold=0.0, swapin_block_threshold=0.0)
    greedy_check(case, eng, [14, 15, 13], 20)
    st = eng.sched.stats
    assert (st.preempt_swap if mode == "swap" else st.preempt_recompute) > 0


def test_beam_search(cases):
    case = cases["flat"]
    eng = serve(case, max_batch_size=8)
    prompt, n = case.tokens(11, 7), 5
    r = eng.generate([prompt], SamplingParams(topk=1, num_beams=3, max_new_tokens=n, ignore_eos=True, length_penalty=1.0))[0]
    lp = [torch.log_softmax(case.logits(prompt + list(o))[len(prompt) - 1:-1], -1) for o in r.output_token_ids]
    best = max(float(sum(l[i, t] for i, t in enumerate(o))) for l, o in zip(lp, r.output_token_ids))
    beams = [([], 0.0)]
    for _ in range(n):
        cand = []
        for toks, s in beams:
            l = torch.log_softmax(O.forward(case.cfg, case.w64, prompt + toks)[-1], -1)
            cand += [(toks + [int(t)], s + float(l[t])) for t in l.topk(6).indices]
        beams = sorted(cand, key=lambda x: -x[1])[:3]
    assert best == pytest.approx(beams[0][1], abs=1e-3)


@pytest.mark.parametrize("bs", [dict(), dict(enable_async=True)])
def test_generation_ends_with_the_position_table(tmp_path, bs):
    """The last row of the table of learned positions is used, and nothing beyond it is asked for."""
    cfg = dict(C.FLAT, max_positions=29)
    case = R.ModelCase(tmp_path, O, cfg, O.random_weights(cfg, 5))
    eng = serve(case, **bs)
    prompt = case.tokens(20, 1)
    r = eng.generate([prompt], SamplingParams(topk=1, max_new_tokens=30, ignore_eos=True))[0]
    assert r.output_token_ids[0] == O.greedy(cfg, case.w64, prompt, 10)
    full = case.tokens(29, 2)
    assert len(eng.generate([full], SamplingParams(topk=1, max_new_tokens=5, ignore_eos=True))[0].output_token_ids[0]) == 1
    from ksanallm_b200.engine.llm_engine import EngineError
    with pytest.raises(EngineError):
        eng.generate([case.tokens(30, 3)], SamplingParams(topk=1, max_new_tokens=2))
    with pytest.raises(RuntimeError, match="longer than"):
        case.engine(torch.float32, 64, "cpu").replay([(1, case.tokens(30, 3), [])])


def test_sampling_parameters_apply(cases):
    eng = serve(cases["one"])
    r = eng.generate([[1, 2, 3]], SamplingParams(topk=5, temperature=0.8, max_new_tokens=5, seed=3, ignore_eos=True, logprobs=2))[0]
    assert len(r.output_token_ids[0]) == 5 and len(r.seqs[0].logprobs) == 5


def test_synthetic_named_model():
    from ksanallm_b200.config.model_config import NAMED_CONFIGS
    cfg = NAMED_CONFIGS["tiny-givirax"]()
    model = TransformerModel(cfg, load_model_weights(cfg, synthetic_seed=1, dtype=torch.float32))
    eng = LLMEngine(model, parse_serving_config({}), num_blocks=32, num_host_blocks=0)
    assert len(eng.generate([[5, 6, 7]], SamplingParams(topk=1, max_new_tokens=3, ignore_eos=True))[0].output_token_ids[0]) == 3


def test_public_engine_serves_the_model_folder(cases, tmp_path):
    """The serving entry point on a folder with config.json and weights, token ids in, token ids out."""
    import asyncio
    from ksanallm_b200.serving.ksana_engine import EngineArgs, KsanaLLMEngine
    case = cases["flat"]
    O.write_model(tmp_path, dict(case.cfg, torch_dtype="float32"), case.w)
    args = EngineArgs(model_dir=str(tmp_path), device="cpu", serving=parse_serving_config(
        {"setting": {"batch_scheduler": {"max_batch_size": 2, "max_token_len": 128, "max_step_tokens": 128}}}))
    eng = KsanaLLMEngine.from_engine_args(args)
    eng.initialize()
    try:
        prompt = case.tokens(9, 3)
        out = eng.generate({"input_tokens": prompt, "sampling_config": {"topk": 1, "max_new_tokens": 4, "ignore_eos": True}})
        if asyncio.iscoroutine(out):
            out = asyncio.run(out)
        status, result = out
        assert status.OK()
        assert list(result.output_tokens[0]) == O.greedy(case.cfg, case.w64, prompt, 4)
    finally:
        eng.shutdown()


# ---- command-line replay --------------------------------------------------------------------------------------------------
def test_replay_command(cases, tmp_path):
    case = cases["odd"]
    a, b = case.tokens(30, 1), case.tokens(5, 2)
    steps = [dict(step=0, entries=[dict(id="p", tokens=a[:28], want=[0, 27]), dict(id="q", tokens=b[:1], want=[])], end=[]),
             dict(step=1, entries=[dict(id="q", tokens=b[1:], want=[3]), dict(id="p", tokens=a[28:29], want=[0])], end=["q"]),
             dict(step=2, entries=[dict(id="p", tokens=a[29:], want=[])], end=["p"])]
    r = subprocess.run([sys.executable, os.path.join(REPO, "bin", "trace_run"), "--model", case.dir, "--dtype", "float32",
                        "--out", str(tmp_path), "--max-tokens", "128", "--device", "cpu"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=120)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]

    def read(i):
        return torch.frombuffer(bytearray((tmp_path / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, case.cfg["vocab"])
    la, lb = case.logits(a), case.logits(b)
    assert (read(0).double() - la[[0, 27]]).abs().max() < 1e-3
    assert (read(1).double() - torch.stack((lb[4], la[28]))).abs().max() < 1e-3
    assert not (tmp_path / "2.f32").exists()
