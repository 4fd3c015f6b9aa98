"""Vibunex on the CPU path: mechanisms alone, whole models through the engine's own step function against the plain oracle,
generation through the scheduler, and the command-line replay."""
import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import replay_cases as R
import vibunex_cases as C
import vibunex_mechanisms as M
import vibunex_oracle as O
from ksanallm_b200.config.model_config import NAMED_CONFIGS, load_model_config, model_config_from_dict
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
@pytest.mark.parametrize("kind", ["random", "far", "sink", "swap"])
def test_attention_with_mixed_weights(kind):
    M.attention_case(F32, "cpu", 6, 2, 20, 36, 12, n=150, kind=kind)


@pytest.mark.parametrize("W", [24, 13])
def test_token_mix(W):
    M.token_mix_case(F32, "cpu", W)


@pytest.mark.parametrize("h,d", [(2, 12), (3, 7), (1, 1)])
@pytest.mark.parametrize("z", [-4.0, 1.0])
def test_time_mixing(h, d, z):
    M.recurrence_case(F32, "cpu", h, d, n=150, z_mean=z)


def test_an_early_token_is_read_through_all_decays():
    M.recurrence_case(F32, "cpu", 2, 12, n=150, z_mean=-6.0, probe=True)


def test_slow_decays_keep_their_precision():
    M.recurrence_case(F32, "cpu", 1, 6, n=600, z_mean=-14.0, tol=3e-6)


def test_time_mixing_batch():
    M.recurrence_batch(F32, "cpu", 2, 8)


def test_tanh_parts():
    M.tanh_case("cpu", 16)


@pytest.mark.parametrize("h,d", [(3, 20), (1, 7)])
def test_head_norm(h, d):
    M.head_norm_case(F32, "cpu", h, d)


@pytest.mark.parametrize("H", [36, 13])
def test_gated_residual(H):
    M.residual_case(F32, "cpu", H)


@pytest.mark.parametrize("experts,top", [(8, 3), (1, 1), (5, 5), (40, 2)])
def test_router(experts, top):
    M.router_case("cpu", experts, top)


def test_plain_experts():
    M.expert_case(F32, "cpu", 30, 5, 2, 28, 22)


def test_squared_relu():
    M.relu2_case(F32, "cpu", 13)


def test_rotation_by_halves_differs_from_neighbours():
    x = torch.randn(5, 2, 12, generator=torch.Generator().manual_seed(0)).double()
    freqs, mag = O.ramped_frequencies(8, 30.0, dict(factor=2.0, fast=4.0, slow=1.0, original=32))
    table = ref.rotary_table(8, 30.0, 5, "cpu", _scaling(8, 30.0, dict(factor=2.0, fast=4.0, slow=1.0, original=32)))
    pos = torch.arange(5)
    want = O.rotate_halves(x, range(5), freqs, mag)
    assert (ref.rotate_pairs(x.float(), pos, table, False).double() - want).abs().max() < 1e-5
    assert (ref.rotate_pairs(x.float(), pos, table, True).double() - want).abs().max() > 0.1
    assert torch.equal(want[:, :, 8:], x[:, :, 8:])


def _scaling(dims, base, s):
    from ksanallm_b200.config.model_config import _ladusun_rotary
    return _ladusun_rotary(dict(dims=dims, base=base, scaling=s), "yarn").scaling


# ---- configuration and loading ------------------------------------------------------------------------------------
def test_configuration(cases):
    cfg = load_model_config(cases["odd"].dir)
    assert resolve_family(cfg.model_type) == "vibunex" and cfg.has_state and cfg.residual_scale == 0.6
    assert [l.kv_width for l in cfg.layers] == [96, 56, 120, 96]
    assert [l.state_shape for l in cfg.layers] == [(1, 1, n + 84) for n in (3 * 400, 2 * 144, 5 * 49, 33 * 33)]
    assert [(l.moe.experts, l.moe.top, l.moe.ff, l.moe.shared_ff, l.moe.scale) if l.moe else None for l in cfg.layers] == [
        (9, 3, 22, 30, 1.7), None, (5, 5, 13, 9, 0.8), (7, 1, 20, 44, 2.5)]
    assert cfg.layers[0].attn.rot.halves and cfg.layers[0].attn.rot.scaling.type == "yarn"
    assert cfg.layers[2].attn.rot.scaling.type == "default"
    assert [(l.attn.out_scale, l.timemix.out_scale) for l in cfg.layers] == [(0.9, 1.2), (1.1, 0.4), (0.5, 1.0), (1.3, 0.7)]
    L = lambda c, i: c["layers"][i]  # noqa: E731
    for change in (lambda c: L(c, 0).update(type="other"), lambda c: L(c, 0)["mixer"]["left"].update(kv_heads=3),
                   lambda c: L(c, 0)["mixer"]["left"]["rot"].update(dims=30), lambda c: L(c, 0)["mixer"]["left"]["rot"].update(dims=5),
                   lambda c: L(c, 0)["mlp"]["router"].update(top=10), lambda c: L(c, 0)["mlp"].update(kind="x")):
        bad = copy.deepcopy(C.ODD)
        change(bad)
        with pytest.raises(ValueError):
            model_config_from_dict(bad)


@pytest.mark.parametrize("name,canonical", [
    ("embed", "embed_tokens"), ("head", "lm_head"), ("final.norm", "model.norm"), ("l0.norm1", "input_layernorm"),
    ("l0.norm2", "post_attention"), ("l1.rg1", "rg"), ("l1.rg1.b", "rg.b"), ("l0.rg2", "rg.weight"), ("l2.rg2.b", "rg.bias"),
    ("l0.mix.left.q", "left.q"), ("l0.mix.left.k.norm", "left.k.norm"), ("l3.mix.left.talk", "talk"), ("l1.mix.left.sink", "sink"),
    ("l0.mix.left.g", "left.g"), ("l0.mix.right.mu.w", "mu.w"), ("l2.mix.right.w2", "w2"), ("l0.mix.right.u", "right.u"),
    ("l0.mix.right.norm", "right.norm"), ("l3.mix.right.o", "right.o"), ("l0.mlp.e4.up", "experts.4.up_proj"),
    ("l0.mlp.router", "gate.weight"), ("l0.mlp.shared.down", "shared_expert.down"), ("l2.mlp.shared.sg", "shared_expert_gate")])
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
    assert [tuple(c.shape) for c in model.allocate_kv_cache(3, 16)] == [(3, 16 * w) for w in [96, 56, 120, 96]]
    assert model.state_slot_bytes() == 4 * (3 * 400 + 2 * 144 + 5 * 49 + 33 * 33 + 4 * 84)


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
def test_stream_after_each_layer(cases, name):
    case = cases[name]
    toks = case.tokens(40, 2)
    want, seen = [], []
    O.forward(case.cfg, case.w64, toks, want)
    eng = case.engine(F32, 64, "cpu")
    for layer in eng.model.layers:
        def hook(h, residual, *args, inner=layer.forward):
            y = inner(h, residual, *args)
            seen.append(residual.clone())
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
    R.run_long_decode(cases["one"], cases["one"].engine(F32, 320, "cpu"), 3e-5)


def test_bf16_storage(cases16):
    R.run_portions(cases16["even"], cases16["even"].engine(torch.bfloat16, 192, "cpu"), 6e-2)


MISTAKES = ["sink", "mixed weights", "mix transposed", "whose values", "scale", "rotation", "pairs", "magnitude", "norm per head",
            "output gate", "left scale", "right scale", "bonus", "state", "decay", "decay input", "previous token", "head norm",
            "time gate", "residual gate", "second norm", "multiplier", "top", "expert weights", "shared gate", "squared"]


@pytest.mark.parametrize("mistake", MISTAKES)
def test_the_comparison_would_show(cases, mistake, monkeypatch):
    """Small mistakes in the oracle move its logits by far more than the tolerance of these tests."""
    case = cases["odd"]
    cfg, w = copy.deepcopy(case.cfg), dict(case.w64)
    L = [x["mixer"] for x in cfg["layers"]]
    patch = lambda name, f: monkeypatch.setattr(O, name, f(getattr(O, name)))  # noqa: E731
    toks = case.tokens(90, 4)
    good = case.logits(toks)
    if mistake == "sink":
        patch("sink_weights", lambda f: lambda s, sink: f(s, sink * 0))
    elif mistake == "mixed weights":
        w["l0.mix.left.talk"] = torch.eye(4).double()
    elif mistake == "mix transposed":
        w["l0.mix.left.talk"] = w["l0.mix.left.talk"].T
    elif mistake == "whose values":  # of the head that the weights come from
        patch("talking_attention", lambda f: lambda q, k, v, scale, sink, talk, first=0: f(q, k, v.flip(1), scale, sink, talk, first))
    elif mistake == "scale":
        L[0]["left"]["scale"] *= 1.03
    elif mistake == "rotation":
        patch("rotate_halves", lambda f: lambda x, pos, *a: f(x, [p + 1 if p > 50 else p for p in pos], *a))
    elif mistake == "pairs":
        patch("rotate_halves", lambda f: lambda x, pos, fr, m=1.0: f(x, pos, fr[:-1], m))
    elif mistake == "magnitude":
        patch("ramped_frequencies", lambda f: lambda *a: (f(*a)[0], 1.0))
    elif mistake == "norm per head":
        def per_head(f):
            def g(x, wt, eps):
                if isinstance(wt, torch.Tensor) and wt.shape == (4 * 28,):
                    return f(x.view(-1, 4, 28), wt.view(4, 28), eps).flatten(1)
                return f(x, wt, eps)
            return g
        patch("rms_norm", per_head)
    elif mistake == "output gate":
        w["l0.mix.left.g"] = w["l0.mix.left.g"].roll(1, 0)
    elif mistake == "left scale":
        L[1]["left_scale"] *= 1.03
    elif mistake == "right scale":
        L[0]["right_scale"] *= 1.01
    elif mistake == "bonus":
        w["l0.mix.right.u"] = torch.ones_like(w["l0.mix.right.u"])
    elif mistake == "state":  # lost in the middle
        patch("bonus_recurrence", lambda f: lambda r, k, v, d, u: (torch.cat((f(r[:64], k[:64], v[:64], d[:64], u)[0],
                                                                              f(r[64:], k[64:], v[64:], d[64:], u)[0])), None))
    elif mistake == "decay":
        w["l0.mix.right.w0"] = w["l0.mix.right.w0"] + 0.02
    elif mistake == "decay input":
        w["l0.mix.right.mu.w"] = w["l0.mix.right.mu.k"]
    elif mistake == "previous token":  # forgotten once
        patch("shifted", lambda f: lambda h, mu: torch.cat((f(h[:64], mu), f(h[64:], mu))))
    elif mistake == "head norm":
        w["l0.mix.right.norm"] = w["l0.mix.right.norm"].roll(1)
    elif mistake == "time gate":
        patch("silu", lambda f: lambda z: O.sigmoid(z))
    elif mistake == "residual gate":
        w["l0.rg2.b"] = w["l0.rg2.b"] * 0
    elif mistake == "second norm":
        w["l0.norm2"] = w["l0.norm1"]
    elif mistake == "multiplier":
        cfg["residual_mult"] *= 1.01
    elif mistake == "top":
        cfg["layers"][0]["mlp"]["router"]["top"] = 2
    elif mistake == "expert weights":
        cfg["layers"][0]["mlp"]["router"]["scale"] *= 1.01
    elif mistake == "shared gate":
        w["l0.mlp.shared.sg"] = w["l0.mlp.shared.sg"] * 0.9
    elif mistake == "squared":
        patch("squared_relu", lambda f: lambda z: torch.clamp(z, min=0))
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


@pytest.mark.parametrize("mode", ["swap", "recompute"])
def test_preemption(cases, mode):
    case = cases["odd"]
    eng = serve(case, n_blocks=7, host_blocks=16 if mode == "swap" else 0, preempt_mode=0 if mode == "swap" else 1,
                launch_block_threshold=0.0, swapin_block_threshold=0.0)
    greedy_check(case, eng, [14, 15, 13], 20)
    st = eng.sched.stats
    assert (st.preempt_swap if mode == "swap" else st.preempt_recompute) > 0


def test_beam_search(cases):
    """Beams fork states and caches: the best one is the oracle's."""
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
    cfg = NAMED_CONFIGS["tiny-vibunex"]()
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
