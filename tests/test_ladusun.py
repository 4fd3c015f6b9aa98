"""Ladusun on the CPU path: mechanisms alone, whole models through the engine's own step function against the plain
oracle, generation through the scheduler, and the command-line replay."""
import copy
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import ladusun_cases as C
import ladusun_mechanisms as M
import ladusun_oracle as O
import replay_cases as R
from ksanallm_b200.config.model_config import _ladusun_rotary, load_model_config, model_config_from_dict
from ksanallm_b200.config.schema import parse_serving_config
from ksanallm_b200.engine.llm_engine import LLMEngine
from ksanallm_b200.engine.sampling_params import SamplingParams
from ksanallm_b200.models.loader import load_model_weights
from ksanallm_b200.models.registry import resolve_family
from ksanallm_b200.models.transformer import TransformerModel
from ksanallm_b200.ops import reference as ref

REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32 = torch.float32


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    return {n: C.Case(tmp_path_factory.mktemp(n), n) for n in C.CASES}


@pytest.fixture(scope="module")
def cases16(tmp_path_factory):
    return {n: C.Case(tmp_path_factory.mktemp(n), n, every_expert=True) for n in C.CASES}


# ---- mechanisms -----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("kind", ["random", "far", "faint"])
def test_capped_attention(kind):
    M.attention_case(F32, "cpu", 3, 1, 20, 36, 2.0, 12, n=150, kind=kind)


@pytest.mark.parametrize("kind", ["random", "far"])
def test_latent_attention(kind):
    M.latent_case(F32, "cpu", 3, 20, 12, 28, 36, n=150, kind=kind)


@pytest.mark.parametrize("C,B,K", [(24, 3, 4), (16, 1, 1), (20, 2, 6)])
def test_gated_recurrence(C, B, K):
    M.recurrence_case(F32, "cpu", C, B, K, n=150)


def test_slow_decays_keep_their_precision():
    M.recurrence_case(F32, "cpu", 16, 2, 2, n=600, lam_mean=-14.0, tol=2e-6)


def test_recurrence_batch():
    M.recurrence_batch(F32, "cpu", 24, 2, 3)


@pytest.mark.parametrize("S,H", [(1, 20), (3, 36), (6, 8)])
def test_streams(S, H):
    M.hyper_case(F32, "cpu", S, H)


@pytest.mark.parametrize("experts,top,groups,keep", [(8, 3, 4, 3), (16, 4, 4, 2), (9, 2, 3, 1), (6, 1, 6, 1), (5, 5, 1, 1), (12, 6, 2, 2)])
def test_router(experts, top, groups, keep):
    M.router_case("cpu", experts, top, groups, keep)


def test_activations():
    M.activation_case(F32, "cpu", 9, 13)


@pytest.mark.parametrize("dims,base,s", [
    (32, 1e4, dict(factor=8.0, low=1.0, high=4.0, original=64)), (2, 10.0, dict(factor=3.0, low=1.0, high=2.0, original=8192)),
    (64, 5e5, dict(factor=32.0, low=0.5, high=16.0, original=512))])
def test_frequencies_in_bands(dims, base, s):
    r = _ladusun_rotary(dict(dims=dims, base=base, scaling=s), "llama3")
    t = ref.rotary_table(r.dims, r.base, 700, "cpu", r.scaling)
    a = torch.outer(torch.arange(700, dtype=torch.float64), torch.tensor(O.banded_frequencies(dims, base, s), dtype=torch.float64))
    assert (t.double() - torch.cat((a.cos(), a.sin()), 1)).abs().max() < 1e-6


@pytest.mark.parametrize("dims,base,s", [
    (32, 1e4, dict(factor=4.0, fast=32.0, slow=1.0, original=2048)), (16, 100.0, dict(factor=2.5, fast=4.0, slow=0.5, original=64)),
    (8, 50.0, dict(factor=2.0, fast=3.0, slow=3.0, original=100)),     # no room for a ramp
    (8, 2.0, dict(factor=3.0, fast=1e-4, slow=1e-5, original=4096)),   # every pair turns faster than that
    (64, 1e5, dict(factor=16.0, fast=4000.0, slow=900.0, original=64)),  # every pair turns slower than that
    (12, 300.0, dict(factor=1.0, fast=32.0, slow=1.0, original=64))])
def test_frequencies_on_a_ramp(dims, base, s):
    r = _ladusun_rotary(dict(dims=dims, base=base, scaling=s), "yarn")
    t = ref.rotary_table(r.dims, r.base, 300, "cpu", r.scaling)
    f, mag = O.ramped_frequencies(dims, base, s)
    a = torch.outer(torch.arange(300, dtype=torch.float64), torch.tensor(f, dtype=torch.float64))
    assert mag == pytest.approx(0.1 * math.log(s["factor"]) + 1)
    assert (t.double() - mag * torch.cat((a.cos(), a.sin()), 1)).abs().max() < 1e-6


def test_rotary_tables_are_kept_apart_and_grow():
    from ksanallm_b200.models.mixers import RotaryTables
    tables = RotaryTables("cpu")
    a = _ladusun_rotary(C.banded(8, 100.0), "llama3")
    b = _ladusun_rotary(C.banded(8, 100.0, factor=2.0), "llama3")
    tables.reserve(10)
    ta, tb = tables.get(a), tables.get(b)
    assert ta.shape == (10, 8) and not torch.equal(ta, tb) and tables.get(copy.deepcopy(a)) is ta
    tables.reserve(30)
    assert tables.get(a).shape == (30, 8) and torch.equal(tables.get(a)[:10], ta)


# ---- configuration and loading ------------------------------------------------------------------------------------
def test_configuration(cases):
    cfg = load_model_config(cases["odd"].dir)
    assert resolve_family(cfg.model_type) == "ladusun" and cfg.has_state and cfg.streams == 3
    assert [l.attn.kv_from if l.attn else None for l in cfg.layers] == [None, None, None, 1, None, None, 1, None]
    assert [l.kv_width for l in cfg.layers] == [0, 96, 48, 0, 0, 56, 0, 48]
    assert [l.state_shape for l in cfg.layers] == [(1, 3, 60)] + [None] * 3 + [(1, 5, 36)] + [None] * 3
    assert [(l.moe.experts, l.moe.top, l.moe.groups, l.moe.keep, l.moe.limit) if l.moe else l.ff for l in cfg.layers] == [
        76, (9, 3, 3, 2, 1.5), 0, 50, 0, (6, 1, 6, 1, 0.8), 0, (8, 4, 2, 2, 2.0)]
    assert not load_model_config(cases["stateless"].dir).has_state
    L = lambda c, i: c["layers"][i]  # noqa: E731
    for change in (lambda c: L(c, 0).update(type="other"), lambda c: L(c, 0)["mixer"].update(blocks=7),
                   lambda c: L(c, 1)["mixer"].update(kv_heads=3), lambda c: L(c, 3)["mixer"].update(kv_from=2),
                   lambda c: L(c, 3)["mixer"].update(kv_from=5), lambda c: L(c, 6)["mixer"].update(kv_from=3),
                   lambda c: L(c, 3)["mixer"]["rot"].update(base=1.0), lambda c: L(c, 2)["mixer"].update(rot_dim=16),
                   lambda c: L(c, 1)["mlp"]["router"].update(top=7), lambda c: L(c, 1)["mlp"]["router"]["groups"].update(count=2),
                   lambda c: L(c, 1)["mlp"]["router"]["groups"].update(keep=4), lambda c: L(c, 0)["mlp"].update(kind="x"),
                   lambda c: c.update(streams=0)):
        bad = copy.deepcopy(C.ODD)
        change(bad)
        with pytest.raises(ValueError):
            model_config_from_dict(bad)


@pytest.mark.parametrize("name,canonical", [
    ("embed", "embed_tokens"), ("final.norm", "model.norm"), ("l0.norm1", "input_layernorm"), ("l0.norm2", "post_attention"),
    ("l0.ls1", "ls1"), ("l1.ls2", "ls2"), ("l2.hc1.in", "hc1.in"), ("l3.hc2.mix", "hc2.mix"), ("l0.hc1.out", "hc1.out"),
    ("l0.mix.ra.b", "ra.b"), ("l0.mix.lam", "lam"), ("l0.mix.conv", "conv"), ("l1.mix.k.b", "k.b"), ("l1.mix.o.b", "o.b"),
    ("l1.mix.g", "g"), ("l2.mix.uk", "uk"), ("l2.mix.dkv.norm", "dkv.norm"), ("l6.mix.q", "q"),
    ("l0.mlp.up.b", "up_proj.bias"), ("l0.mlp.down", "down_proj"), ("l1.mlp.e4.up", "experts.4.up_proj"),
    ("l1.mlp.router", "gate.weight")])
def test_missing_tensor_is_named(cases, tmp_path, name, canonical):
    w = dict(cases["odd"].w)
    del w[name]
    O.write_model(tmp_path, C.ODD, w)
    with pytest.raises(KeyError, match=canonical):
        cfg = load_model_config(str(tmp_path))
        TransformerModel(cfg, load_model_weights(cfg, str(tmp_path), dtype=F32))


def test_caches_and_slots(cases):
    cfg = load_model_config(cases["odd"].dir)
    model = TransformerModel(cfg, load_model_weights(cfg, cases["odd"].dir, dtype=F32))
    assert [tuple(c.shape) for c in model.allocate_kv_cache(3, 16)] == [(3, 16 * w) for w in [0, 96, 48, 0, 0, 56, 0, 48]]
    assert model.kv_block_bytes(16) == 4 * 16 * (96 + 48 + 56 + 48)
    assert model.state_slot_bytes() == 4 * (3 * 60 + 5 * 36)
    assert [s.numel() for s in model.allocate_state(2)] == [360, 0, 0, 0, 360, 0, 0, 0]


def test_what_it_does_not_combine_with(cases):
    from ksanallm_b200.parallel.comm import TPGroup
    cfg = load_model_config(cases["odd"].dir)
    w = load_model_weights(cfg, cases["odd"].dir, dtype=F32)
    with pytest.raises(NotImplementedError):
        TransformerModel(cfg, w, TPGroup(0, 2, None, torch.device("cpu"), use_fused=False))
    serving = parse_serving_config({"setting": {"global": {"pipeline_para_size": 2}}})
    with pytest.raises(NotImplementedError):
        LLMEngine(TransformerModel(cfg, w), serving, num_blocks=8, num_host_blocks=0)


# ---- whole models ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", list(C.CASES))
def test_streams_after_each_layer(cases, name):
    case = cases[name]
    toks = case.tokens(40, 2)
    want, seen = [], []
    O.forward(case.cfg, case.w64, toks, want)
    eng = case.engine(F32, 64, "cpu")
    for layer in eng.model.layers:
        def hook(h, residual, *args, inner=layer.forward):
            y = inner(h, residual, *args)
            seen.append(residual.sum(1))
            return y
        layer.forward = hook
    eng.replay([(1, toks, [])])
    assert len(seen) == len(want)
    for got, w in zip(seen, want):
        assert (got.double() - w).abs().max() < 2e-5 * w.abs().max()


@pytest.mark.parametrize("name", list(C.CASES))
def test_portions(cases, name):
    R.run_portions(cases[name], cases[name].engine(F32, 192, "cpu"), 3e-5)


@pytest.mark.parametrize("name", list(C.CASES))
def test_batches_and_reuse(cases, name):
    R.run_batches(cases[name], cases[name].engine(F32, 64 * 7, "cpu"), 3e-5)


def test_long_decode(cases):
    R.run_long_decode(cases["odd"], cases["odd"].engine(F32, 320, "cpu"), 3e-5)


def test_bf16_storage(cases16):
    R.run_portions(cases16["even"], cases16["even"].engine(torch.bfloat16, 192, "cpu"), 6e-2)


MISTAKES = ["cap", "sink", "gate", "scale", "rotation", "pairs", "bands", "magnitude", "whose keys", "latent norm", "shared key",
            "convolution", "state", "decay", "input gate", "limit", "expert", "groups", "top", "expert weights", "mix order",
            "layer scale", "squared", "bias"]


@pytest.mark.parametrize("mistake", MISTAKES)
def test_the_comparison_would_show(cases, mistake, monkeypatch):
    """Small mistakes in the oracle move its logits by far more than the tolerance of these tests."""
    case = cases["odd"]
    cfg, w = copy.deepcopy(case.cfg), dict(case.w64)
    L = [x["mixer"] for x in cfg["layers"]]
    patch = lambda name, f: monkeypatch.setattr(O, name, f(getattr(O, name)))  # noqa: E731
    toks = case.tokens(90, 4)
    good = case.logits(toks)
    if mistake == "cap":
        L[1]["softcap"] *= 1.01
    elif mistake == "sink":
        patch("softmax_rows", lambda f: lambda s, sink: f(s, False))
    elif mistake == "gate":
        patch("head_gate", lambda f: lambda o, h, g: f(o, h, g.roll(1, 0)))
    elif mistake == "scale":
        L[2]["scale"] *= 1.01
    elif mistake == "rotation":
        patch("rotate_pairs", lambda f: lambda x, pos, *a: f(x, [p + 1 if p > 50 else p for p in pos], *a))
    elif mistake == "pairs":
        patch("rotate_pairs", lambda f: lambda x, pos, fr, m=1.0: f(x, pos, fr[:-1], m))
    elif mistake == "bands":
        patch("banded_frequencies", lambda f: lambda dims, base, s: O.plain_frequencies(dims, base))
    elif mistake == "magnitude":
        patch("ramped_frequencies", lambda f: lambda *a: (f(*a)[0], 1.0))
    elif mistake == "whose keys":
        w["l1.mix.k"] = w["l1.mix.k"].clone()
        w["l1.mix.k"][5] *= 1.02
    elif mistake == "latent norm":
        w["l2.mix.dkv.norm"] = torch.ones_like(w["l2.mix.dkv.norm"])
    elif mistake == "shared key":
        patch("latent_attention", lambda f: lambda q, c, r, *a: f(q, c, r * 0.9, *a))
    elif mistake == "convolution":
        w["l0.mix.conv"] = w["l0.mix.conv"].roll(1, 1)
    elif mistake == "state":  # lost in the middle
        patch("gated_recurrence", lambda f: lambda u, r, i, lam: (torch.cat((f(u[:64], r[:64], i[:64], lam)[0],
                                                                            f(u[64:], r[64:], i[64:], lam)[0])), None))
    elif mistake == "decay":
        w["l0.mix.lam"] = w["l0.mix.lam"] + 0.02
    elif mistake == "input gate":
        patch("gated_recurrence", lambda f: lambda u, r, i, lam: f(u, r, torch.ones_like(i), lam))
    elif mistake == "limit":
        cfg["layers"][1]["mlp"]["expert"]["limit"] *= 1.1
    elif mistake == "expert":
        patch("expert", lambda f: lambda h, limit, w_, p: f(h, limit, w_, p) * 0.99)
    elif mistake == "groups":
        cfg["layers"][1]["mlp"]["router"]["groups"]["keep"] = 3
    elif mistake == "top":
        cfg["layers"][1]["mlp"]["router"]["top"] = 2
    elif mistake == "expert weights":
        patch("route", lambda f: lambda *a: (f(*a)[0], f(*a)[1] * 0.99))
    elif mistake == "mix order":
        w["l0.hc1.mix"] = w["l0.hc1.mix"].T
    elif mistake == "layer scale":
        w["l3.ls2"] = torch.ones_like(w["l3.ls2"])
    elif mistake == "squared":
        patch("squared_relu", lambda f: lambda z: torch.clamp(z, min=0))
    elif mistake == "bias":
        w["l1.mix.o.b"] = torch.zeros_like(w["l1.mix.o.b"])
    bad = O.forward(cfg, w, toks)
    rms = ((good - bad) ** 2).mean(1).sqrt() / good.std()
    assert float(rms[45:].max()) > 20 * 3e-5


# ---- generation through the scheduler -----------------------------------------------------------------------------------
def serve(case, n_blocks=64, host_blocks=0, device="cpu", dtype=F32, **bs):
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
        out = r.output_token_ids[0]
        # every token is the largest logit behind the ones before it
        assert len(out) == new and out == case.logits(p + out)[len(p) - 1:-1].argmax(1).tolist(), len(p)
    return eng


@pytest.mark.parametrize("bs", [dict(), dict(split_fuse_token_num=9), dict(enable_async=True), dict(max_step_tokens=24)])
def test_greedy_generation(cases, bs):
    greedy_check(cases["odd"], serve(cases["odd"], **bs), [1, 2, 30, 17, 41, 8], 8)


def test_greedy_oracle_agrees(cases):
    case = cases["one"]
    r = serve(case).generate([case.tokens(9, 3)], SamplingParams(topk=1, max_new_tokens=6, ignore_eos=True))[0]
    assert r.output_token_ids[0] == O.greedy(case.cfg, case.w64, case.tokens(9, 3), 6)


def test_states_are_not_shared_by_prefix(cases):
    """A recurrent state is not kept per block: equal prompts are computed in full."""
    eng = serve(cases["odd"], enable_auto_prefix_cache=True)
    for _ in range(2):
        greedy_check(cases["odd"], eng, [50], 4)
    assert eng.cache.stats.prefix_hit_tokens == 0


def test_shared_prefixes_are_reused_without_states(cases):
    case = cases["stateless"]
    eng = serve(case, enable_auto_prefix_cache=True)
    greedy_check(case, eng, [50], 4)
    greedy_check(case, eng, [50], 4)
    assert eng.cache.stats.prefix_hit_tokens >= 48


def test_speculative_drafts(cases):
    """Verified drafts: steps of several tokens per sequence behind cached keys and latents."""
    case = cases["stateless"]
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
    case = cases["one"]
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


def test_sampling_parameters_apply(cases):
    eng = serve(cases["one"])
    r = eng.generate([[1, 2, 3]], SamplingParams(topk=5, temperature=0.8, max_new_tokens=5, seed=3, ignore_eos=True, logprobs=2))[0]
    assert len(r.output_token_ids[0]) == 5 and len(r.seqs[0].logprobs) == 5


def test_synthetic_named_model():
    from ksanallm_b200.config.model_config import NAMED_CONFIGS
    cfg = NAMED_CONFIGS["tiny-ladusun"]()
    model = TransformerModel(cfg, load_model_weights(cfg, synthetic_seed=1, dtype=F32))
    eng = LLMEngine(model, parse_serving_config({}), num_blocks=32, num_host_blocks=0)
    assert len(eng.generate([[5, 6, 7]], SamplingParams(topk=1, max_new_tokens=3, ignore_eos=True))[0].output_token_ids[0]) == 3


def test_public_engine_serves_the_model_folder(cases, tmp_path):
    """The serving entry point on a folder with config.json and weights, token ids in, token ids out."""
    import asyncio
    from ksanallm_b200.serving.ksana_engine import EngineArgs, KsanaLLMEngine
    case = cases["one"]
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
        return torch.frombuffer(bytearray((tmp_path / f"{i}.f32").read_bytes()), dtype=F32).view(-1, case.cfg["vocab"])
    la, lb = case.logits(a), case.logits(b)
    assert (read(0).double() - la[[0, 27]]).abs().max() < 1e-3
    assert (read(1).double() - torch.stack((lb[4], la[28]))).abs().max() < 1e-3
    assert not (tmp_path / "2.f32").exists()
