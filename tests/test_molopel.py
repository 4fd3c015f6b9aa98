"""Molopel on the CPU path: mechanisms alone, the state slots of the cache manager and scheduler, whole models through
the engine's own step function against the plain oracle, generation, and the command-line replay."""
import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import molopel_cases as C
import molopel_oracle as M
from ksanallm_b200 import host
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
@pytest.mark.parametrize("rows,bias_max", [(16, 30), (12, 100), (24, 130), (2, 5), (8, 64)])
def test_distance_bias_buckets(rows, bias_max):
    rel = torch.arange(rows, dtype=torch.float32).unsqueeze(1)
    got = ref.distance_bias(rel, bias_max, 300)[0]
    assert got.tolist() == [float(M.distance_bucket(n, rows, bias_max)) for n in range(300)]


def test_distance_bias_exact_boundaries():
    """Distances that lie exactly on a boundary belong to the upper bucket whatever the logarithms round to."""
    got = ref.distance_bias(torch.arange(16.0).unsqueeze(1), 128, 129)[0]  # boundaries at 8 * 2^(k / 2)
    assert [int(got[8 * 2 ** k]) for k in range(5)] == [8, 10, 12, 14, 15]


def test_rotary_table_partial():
    x = torch.randn(5, 2, 24, dtype=torch.float64)
    table = ref.rotary_table(16, 700.0, 50)
    cs = table[40:45].double()
    got = ref.apply_rope(x, cs[:, :8], cs[:, 8:], False, 16).double()
    assert (got - M.rotate_half(x, 40, 16, 700.0)).abs().max() < 1e-5


@pytest.mark.parametrize("window", [1, 16, 17, 40])
def test_window_edges_in_prompts_and_decoding(window):
    from molopel_cases_attention import check_window
    check_window(torch.float32, "cpu", window)


# ---- state slots ------------------------------------------------------------------------------------------------
def test_cache_manager_state_slots():
    c = host.KVCacheManager(16, 4, 16, True)
    c.configure_states(2, 1)
    assert c.stateful
    c.create_seq(1, list(range(20)))
    c.create_seq(2, list(range(20)))
    assert {c.state_slot(1), c.state_slot(2)} == {0, 1} and c.num_free_state_slots == 0
    with pytest.raises(RuntimeError):
        c.create_seq(3, [1])
    c.free_seq(1)
    c.create_seq(3, [1])
    assert c.state_slot(3) == 0
    c.free_seq(2)
    c.free_seq(3)
    assert c.num_free_state_slots == 2


def test_scheduler_admits_no_more_sequences_than_slots():
    c = host.KVCacheManager(64, 0, 16, False)
    c.configure_states(2, 0)
    sc = host.SchedulerConfig()
    sc.max_batch_size, sc.max_token_len, sc.preempt_mode = 8, 256, 1
    s = host.Scheduler(sc, c)
    for i in range(5):
        assert s.enqueue(i, [1, 2, 3], 2, True) == host.RET_SUCCESS
    seen = []
    for _ in range(40):
        plan = s.schedule(0)
        if plan.empty():
            break
        assert len(plan.entries) <= 2
        slots = [c.state_slot(e.seq_id) for e in plan.entries]
        assert len(set(slots)) == len(slots)
        seen += [r.seq_id for r in s.update(plan, [7] * plan.total_logits) if r.finish_reason != host.FINISH_NONE]
    assert sorted(seen) == list(range(5)) and c.num_free_state_slots == 2


# ---- configuration and loading ------------------------------------------------------------------------------------
def test_configuration(cases):
    cfg = load_model_config(cases["odd"].dir)
    assert resolve_family(cfg.model_type) == "molopel" and cfg.has_state
    assert [l.attn.window if l.attn else 0 for l in cfg.layers] == [0, 20, 7, 0]
    assert [l.ff for l in cfg.layers] == [76, 100, 0, 0]
    assert cfg.layers[1].linear.rot_dims == 24 and cfg.layers[1].linear.key_scale == pytest.approx(44 ** -0.5)
    assert cfg.layers[0].linear.norm == "concat" and cfg.layers[0].linear.gate == "sigmoid"
    bad = copy.deepcopy(C.ODD)
    bad["layers"][0]["type"] = "other"
    with pytest.raises(ValueError):
        model_config_from_dict(bad)
    bad = copy.deepcopy(C.ODD)
    bad["layers"][0]["mixer"]["decay"] = [0.5]
    with pytest.raises(ValueError):
        model_config_from_dict(bad)


def test_missing_tensor_is_named(cases, tmp_path):
    w = dict(cases["odd"].w)
    del w["l1.mix.right.g"]
    M.write_model(tmp_path, C.ODD, w)
    with pytest.raises(KeyError, match="right.g"):
        load_model_weights(load_model_config(str(tmp_path)), str(tmp_path), dtype=torch.float32)


def test_what_recurrent_models_do_not_combine_with(cases):
    from ksanallm_b200.parallel.comm import TPGroup
    cfg = load_model_config(cases["odd"].dir)
    w = load_model_weights(cfg, cases["odd"].dir, dtype=torch.float32)
    with pytest.raises(NotImplementedError):
        TransformerModel(cfg, w, TPGroup(0, 2, None, torch.device("cpu"), use_fused=False))
    serving = parse_serving_config({"setting": {"connector": {"group_role": "prefill"}}})
    with pytest.raises(NotImplementedError):
        LLMEngine(TransformerModel(cfg, w), serving, num_blocks=8, num_host_blocks=0)


# ---- whole models ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", list(C.CASES))
def test_residual_stream_after_each_layer(cases, name):
    """Layer by layer: the stream that enters layer i + 1 is the oracle's."""
    case = cases[name]
    toks = case.tokens(40, 2)
    want = []
    M.forward(case.cfg, case.w64, toks, want)
    eng = case.engine(torch.float32, 64, "cpu")
    model, seen = eng.model, []
    for layer in model.layers:
        def hook(h, residual, meta, cache, nw, nb=None, inner=layer.forward):
            y = inner(h, residual, meta, cache, nw, nb)
            seen.append(residual.clone())
            return y
        layer.forward = hook
    eng.replay([(1, toks, [])])
    assert len(seen) == len(want)
    for got, w in zip(seen, want):
        assert (got.double() - w).abs().max() < 2e-5 * w.abs().max()


@pytest.mark.parametrize("name", list(C.CASES))
def test_portions(cases, name):
    C.run_portions(cases[name], cases[name].engine(torch.float32, 192, "cpu"), 2e-5)


@pytest.mark.parametrize("name", list(C.CASES))
def test_batches_and_reuse(cases, name):
    C.run_batches(cases[name], cases[name].engine(torch.float32, 64 * 7, "cpu"), 2e-5)


def test_long_decode(cases):
    C.run_long_decode(cases["odd"], cases["odd"].engine(torch.float32, 320, "cpu"), 2e-5)


def test_bf16_storage(cases):
    C.run_portions(cases["even"], cases["even"].engine(torch.bfloat16, 192, "cpu"), 6e-2)


@pytest.mark.parametrize("mistake", ["window", "decay", "bias", "rotation", "first tokens"])
def test_the_comparison_would_show(cases, mistake):
    """Small mistakes in the oracle move its logits by far more than the tolerance of these tests."""
    case = cases["even"]
    cfg, w = copy.deepcopy(case.cfg), dict(case.w64)
    left, right = cfg["layers"][0]["mixer"]["left"], cfg["layers"][0]["mixer"]["right"]
    if mistake == "window":
        left["mask"]["size"] += 1
    elif mistake == "decay":
        right["decay"][0] *= 1.001
    elif mistake == "bias":
        left["bias_max"] += 5
    elif mistake == "rotation":
        right["rot"]["base"] *= 1.01
    toks = case.tokens(120, 4)
    good = case.logits(toks)
    bad = M.forward(cfg, w, toks) if mistake != "first tokens" else \
        torch.cat((torch.zeros(1, cfg["vocab"], dtype=torch.float64), M.forward(cfg, w, toks[1:])))
    rms = ((good - bad) ** 2).mean(1).sqrt() / good.std()
    assert float(rms[60:].max()) > 20 * 2e-5


# ---- generation through the scheduler -----------------------------------------------------------------------------------
def serve(case, n_blocks=64, host_blocks=0, slots=None, device="cpu", dtype=torch.float32, **bs):
    cfg = load_model_config(case.dir)
    setting = dict(max_batch_size=4, max_step_tokens=256, max_token_len=512)
    setting.update(bs)
    serving = parse_serving_config({"setting": {"batch_scheduler": setting}})
    model = TransformerModel(cfg, load_model_weights(cfg, case.dir, device=device, dtype=dtype))
    return LLMEngine(model, serving, num_blocks=n_blocks, num_host_blocks=host_blocks, num_state_slots=slots)


def greedy_check(case, eng, lens, new, **params):
    prompts = [case.tokens(n, 50 + n) for n in lens]
    reqs = eng.generate(prompts, SamplingParams(topk=1, max_new_tokens=new, ignore_eos=True, **params))
    for p, r in zip(prompts, reqs):
        assert r.output_token_ids[0] == M.greedy(case.cfg, case.w64, p, new), len(p)
    assert eng.cache.num_free_state_slots == eng.cache.num_state_slots
    return eng


@pytest.mark.parametrize("bs", [dict(), dict(split_fuse_token_num=9), dict(enable_async=True), dict(max_step_tokens=24)])
def test_greedy_generation(cases, bs):
    greedy_check(cases["odd"], serve(cases["odd"], **bs), [1, 2, 30, 17, 41, 8], 8)


def test_greedy_generation_with_prefix_cache_asked_for(cases):
    """Equal prefixes are computed again: the state behind a cached prefix is not kept."""
    case = cases["odd"]
    eng = serve(case, enable_auto_prefix_cache=True)
    for _ in range(2):
        greedy_check(case, eng, [40, 40], 4)


def test_speculative_drafts_are_off(cases):
    eng = greedy_check(cases["one"], serve(cases["one"], enable_speculative_decoding=True), [12, 20], 10)
    assert eng.sched.stats.draft_proposed == 0


@pytest.mark.parametrize("mode", ["swap", "recompute"])
def test_preemption_keeps_the_state(cases, mode):
    case = cases["odd"]
    eng = serve(case, n_blocks=7, host_blocks=16 if mode == "swap" else 0, preempt_mode=0 if mode == "swap" else 1,
                launch_block_threshold=0.0, swapin_block_threshold=0.0)
    greedy_check(case, eng, [14, 15, 13], 20)
    st = eng.sched.stats
    assert (st.preempt_swap if mode == "swap" else st.preempt_recompute) > 0


def test_fewer_slots_than_requests(cases):
    greedy_check(cases["one"], serve(cases["one"], slots=2), [5, 9, 14, 3, 7], 6)


def test_beam_search_forks_the_state(cases):
    """The best beam's score is the sum of its tokens' log-probabilities under the oracle."""
    case = cases["one"]
    eng = serve(case, max_batch_size=8)
    prompt, n = case.tokens(11, 7), 6
    r = eng.generate([prompt], SamplingParams(topk=1, num_beams=3, max_new_tokens=n, ignore_eos=True, length_penalty=1.0))[0]
    lp = [torch.log_softmax(case.logits(prompt + list(o))[len(prompt) - 1:-1], -1) for o in r.output_token_ids]
    best = max(float(sum(l[i, t] for i, t in enumerate(o))) for l, o in zip(lp, r.output_token_ids))
    # exhaustive beam search in the oracle
    beams = [([], 0.0)]
    for _ in range(n):
        cand = []
        for toks, s in beams:
            l = torch.log_softmax(M.forward(case.cfg, case.w64, prompt + toks)[-1], -1)
            cand += [(toks + [int(t)], s + float(l[t])) for t in l.topk(6).indices]
        beams = sorted(cand, key=lambda x: -x[1])[:3]
    assert best == pytest.approx(beams[0][1], abs=1e-3)


def test_sampling_parameters_apply(cases):
    eng = serve(cases["one"])
    r = eng.generate([[1, 2, 3]], SamplingParams(topk=5, temperature=0.8, max_new_tokens=5, seed=3, ignore_eos=True, logprobs=2))[0]
    assert len(r.output_token_ids[0]) == 5 and len(r.seqs[0].logprobs) == 5


def test_synthetic_named_model():
    from ksanallm_b200.config.model_config import NAMED_CONFIGS
    cfg = NAMED_CONFIGS["tiny-molopel"]()
    model = TransformerModel(cfg, load_model_weights(cfg, synthetic_seed=1, dtype=torch.float32))
    eng = LLMEngine(model, parse_serving_config({}), num_blocks=32, num_host_blocks=0)
    assert len(eng.generate([[5, 6, 7]], SamplingParams(topk=1, max_new_tokens=3, ignore_eos=True))[0].output_token_ids[0]) == 3


def test_public_engine_serves_the_model_folder(cases, tmp_path):
    """The serving entry point on a folder with config.json and weights, token ids in, token ids out."""
    import asyncio
    from ksanallm_b200.serving.ksana_engine import EngineArgs, KsanaLLMEngine
    case = cases["one"]
    raw = dict(case.cfg, torch_dtype="float32")
    M.write_model(tmp_path, raw, case.w)
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
        assert list(result.output_tokens[0]) == M.greedy(case.cfg, case.w64, prompt, 4)
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
    V = case.cfg["vocab"]

    def read(i):
        return torch.frombuffer(bytearray((tmp_path / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, V)
    la, lb = case.logits(a), case.logits(b)
    assert (read(0).double() - la[[0, 27]]).abs().max() < 1e-3
    assert (read(1).double() - torch.stack((lb[4], la[28]))).abs().max() < 1e-3
    assert not (tmp_path / "2.f32").exists()


def test_replay_refuses_what_the_pool_cannot_hold(cases):
    eng = cases["one"].engine(torch.float32, 64, "cpu")
    with pytest.raises(RuntimeError, match="too small"):
        eng.replay([(1, cases["one"].tokens(80, 1), [])])
