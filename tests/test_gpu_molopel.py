"""Molopel on the GPU: whole models through the engine's own step function against the plain oracle, in both number
formats, and generation through the scheduler."""
import pytest
import torch

import molopel_cases as C
import molopel_oracle as M
from molopel_cases_attention import check_window
from test_molopel import greedy_check, serve

pytestmark = pytest.mark.gpu
FORMATS = [(torch.float32, 1e-4), (torch.bfloat16, 6e-2)]


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    return {n: C.Case(tmp_path_factory.mktemp(n), n) for n in C.CASES}


@pytest.mark.parametrize("dtype,tol", FORMATS)
@pytest.mark.parametrize("name", list(C.CASES))
def test_portions(cases, name, dtype, tol):
    C.run_portions(cases[name], cases[name].engine(dtype, 192, "cuda"), tol)


@pytest.mark.parametrize("dtype,tol", FORMATS)
@pytest.mark.parametrize("name", list(C.CASES))
def test_batches_and_reuse(cases, name, dtype, tol):
    C.run_batches(cases[name], cases[name].engine(dtype, 64 * 7, "cuda"), tol)


@pytest.mark.parametrize("dtype,tol", FORMATS)
def test_long_decode(cases, dtype, tol):
    for name in ("odd", "even"):
        C.run_long_decode(cases[name], cases[name].engine(dtype, 320, "cuda"), tol)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("window", [1, 16, 17, 40, 128])
def test_window_edges_in_prompts_and_decoding(dtype, window):
    check_window(dtype, "cuda", window)


def test_layer_path_and_native_executor_agree(cases, monkeypatch):
    """One call per step and one call per kernel launch the same kernels."""
    case = cases["even"]
    toks = [case.tokens(n, n) for n in (140, 20, 33)]

    def run():
        eng = case.engine(torch.bfloat16, 512, "cuda")
        a = eng.replay([(i, t[:-1], [len(t) - 2]) for i, t in enumerate(toks)])
        b = eng.replay([(i, t[-1:], [0]) for i, t in enumerate(toks)])
        return torch.cat((a, b)), eng.model
    native, m1 = run()
    assert type(m1._native).__name__ == "MixerExecutor"
    monkeypatch.setenv("KSANA_DISABLE_NATIVE_EXECUTOR", "1")
    layers, m2 = run()
    assert m2._native is None
    assert torch.equal(native, layers)


def test_activation_as_gemm_epilogue(cases, monkeypatch):
    """KSANA_FUSED_SWIGLU=1: prompt-sized steps run GELU(gate) * up inside the GEMM."""
    monkeypatch.setenv("KSANA_FUSED_SWIGLU", "1")
    case = cases["even"]
    eng = case.engine(torch.bfloat16, 512, "cuda")
    toks = [case.tokens(130, i) for i in range(3)]
    got = eng.replay([(i, t, list(range(130))) for i, t in enumerate(toks)])
    assert eng.model._native._wgu_il
    want = torch.cat([case.logits(t) for t in toks])
    assert (((got.double() - want) ** 2).mean(1).sqrt() / want.std()).max() < 6e-2


@pytest.mark.parametrize("bs", [dict(), dict(split_fuse_token_num=9), dict(enable_async=True)])
def test_greedy_generation(cases, bs):
    greedy_check(cases["odd"], serve(cases["odd"], device="cuda", **bs), [1, 2, 30, 17, 41, 8], 8)


@pytest.mark.parametrize("mode", ["swap", "recompute"])
def test_preemption_keeps_the_state(cases, mode):
    eng = serve(cases["odd"], n_blocks=7, host_blocks=16 if mode == "swap" else 0, device="cuda",
                preempt_mode=0 if mode == "swap" else 1, launch_block_threshold=0.0, swapin_block_threshold=0.0)
    greedy_check(cases["odd"], eng, [14, 15, 13], 20)
    st = eng.sched.stats
    assert (st.preempt_swap if mode == "swap" else st.preempt_recompute) > 0


def test_generation_in_16_bits_follows_its_own_logits(cases):
    """bf16 generation through the scheduler, in one batch, picks tokens the oracle ranks at (or within rounding of) the
    top."""
    case = cases["even"]
    eng = serve(case, device="cuda", dtype=torch.bfloat16, split_fuse_token_num=50)
    from ksanallm_b200.engine.sampling_params import SamplingParams
    prompts = [case.tokens(n, n) for n in (3, 70, 130, 41)]
    for p, r in zip(prompts, eng.generate(prompts, SamplingParams(topk=1, max_new_tokens=12, ignore_eos=True))):
        out = r.output_token_ids[0]
        lg = M.forward(case.cfg, case.w64, p + out)[len(p) - 1:-1]
        chosen = lg.gather(1, torch.tensor(out).unsqueeze(1))[:, 0]
        assert ((lg.max(1).values - chosen) < 0.25 * lg.std()).all()
