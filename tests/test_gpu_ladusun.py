"""Ladusun on the GPU: its kernels one by one, whole models through the engine's own step function against the plain
oracle in both number formats, and generation through the scheduler."""
import pytest
import torch

import ladusun_cases as C
import ladusun_mechanisms as M
import ladusun_oracle as O
import replay_cases as R
from ksanallm_b200 import ops
from ksanallm_b200.engine.sampling_params import SamplingParams
from ksanallm_b200.ops import reference as ref
from test_ladusun import greedy_check, serve

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
FORMATS = [F32, BF16]


def tolerance(dtype, name):
    """16 bits: twice what the CPU path, computing in 32 bits and storing in 16, is off by."""
    return 1e-4 if dtype == F32 else 0.2 if name == "odd" else 5e-2


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    """By number format: 16-bit models are compared without discrete choices (see Case)."""
    return {t: {n: C.Case(tmp_path_factory.mktemp(n), n, every_expert=t == BF16) for n in C.CASES} for t in (F32, BF16)}


# ---- mechanisms -----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("kind", ["random", "far", "faint"])
@pytest.mark.parametrize("H,G,d,dv,cap,dims", [(4, 2, 64, 64, 4.0, 16), (3, 1, 128, 64, 1.5, 32), (34, 2, 32, 128, 30.0, 8),
                                               (2, 2, 20, 36, 2.0, 12)])
def test_capped_attention(dtype, kind, H, G, d, dv, cap, dims):
    M.attention_case(dtype, "cuda", H, G, d, dv, cap, dims, kind=kind)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_caps_that_hardly_bend(dtype):
    M.attention_case(dtype, "cuda", cap=500.0)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("kind", ["random", "far"])
@pytest.mark.parametrize("H,dim,rot,vdim,rank", [(4, 64, 32, 64, 128), (9, 128, 64, 128, 512), (3, 40, 16, 72, 200), (2, 24, 8, 24, 32),
                                                 (17, 128, 8, 16, 320), (3, 20, 12, 28, 36), (1, 8, 2, 16, 16), (2, 136, 32, 64, 64)])
def test_latent_attention(dtype, kind, H, dim, rot, vdim, rank):
    M.latent_case(dtype, "cuda", H, dim, rot, vdim, rank, kind=kind)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("C,B,K", [(256, 2, 4), (192, 1, 6), (60, 3, 3), (128, 1, 1), (64, 4, 8), (512, 2, 2), (24, 1, 11), (144, 6, 4)])
def test_gated_recurrence(dtype, C, B, K):
    M.recurrence_case(dtype, "cuda", C, B, K)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("lam", [-9.0, 2.0])
def test_slow_and_fast_decays(dtype, lam):
    M.recurrence_case(dtype, "cuda", lam_mean=lam)


def test_slow_decays_keep_their_precision():
    """Decays within 1e-5 of 1: rounding them would add up over the tokens."""
    M.recurrence_case(F32, "cuda", 64, 2, 2, n=1500, lam_mean=-14.0, tol=2e-6)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("C,B,K", [(128, 2, 4), (60, 3, 3), (192, 1, 5)])
def test_recurrence_batch(dtype, C, B, K):
    M.recurrence_batch(dtype, "cuda", C, B, K)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("S,H", [(4, 128), (1, 92), (2, 4096), (3, 1028), (4, 2048), (4, 8192), (5, 30), (16, 64), (2, 9000)])
def test_streams(dtype, S, H):
    M.hyper_case(dtype, "cuda", S, H)


@pytest.mark.parametrize("experts,top,groups,keep", [(8, 3, 4, 3), (16, 4, 4, 2), (9, 2, 3, 1), (6, 1, 6, 1), (5, 5, 1, 1), (512, 8, 64, 33), (12, 6, 2, 2)])
def test_router(experts, top, groups, keep):
    M.router_case("cuda", experts, top, groups, keep)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("cols", [104, 13, 2048])
def test_activations(dtype, cols):
    M.activation_case(dtype, "cuda", 9, cols)


@pytest.mark.parametrize("dtype,T,E,top,H,I", [(BF16, 300, 6, 3, 264, 104), (BF16, 40, 3, 2, 92, 22), (F32, 70, 5, 2, 92, 24)])
def test_clamped_experts(dtype, T, E, top, H, I):
    g = torch.Generator().manual_seed(T + E)
    x = torch.randn(T, H, generator=g).to(dtype).cuda()
    w1 = (2 * torch.randn(E, 2 * I, H, generator=g) / H ** 0.5).to(dtype).cuda()
    w2 = (torch.randn(E, H, I, generator=g) / I ** 0.5).to(dtype).cuda()
    ids = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)]).int().cuda()
    y, pos = ops.moe_expert_rows(x, ids, w1, w2, 1.3, 1.702)
    want, _ = ref.moe_expert_rows(x.double().cpu(), ids.cpu(), w1.double().cpu(), w2.double().cpu(), 1.3, 1.702)
    err = (y[pos.long()].double().cpu() - want).abs().max() / want.abs().max()
    assert err < (2e-6 if dtype == F32 else 2e-2)


# ---- whole models ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", FORMATS)
@pytest.mark.parametrize("name", list(C.CASES))
def test_portions(cases, name, dtype):
    R.run_portions(cases[dtype][name], cases[dtype][name].engine(dtype, 192, "cuda"), tolerance(dtype, name))


@pytest.mark.parametrize("dtype", FORMATS)
@pytest.mark.parametrize("name", list(C.CASES))
def test_batches_and_reuse(cases, name, dtype):
    R.run_batches(cases[dtype][name], cases[dtype][name].engine(dtype, 64 * 7, "cuda"), tolerance(dtype, name))


def test_prompts_written_out_in_several_rounds(cases, monkeypatch):
    """Contexts whose keys and values are written out a few sequences at a time, of very different lengths."""
    from ksanallm_b200.ops import cuda_latent
    m = C.EVEN["layers"][0]["mixer"]
    monkeypatch.setenv("KSANA_DISABLE_NATIVE_EXECUTOR", "1")
    monkeypatch.setattr(cuda_latent, "EXPAND_BYTES", 100 * 2 * m["heads"] * (m["dim"] + m["vdim"]))
    R.run_batches(cases[BF16]["even"], cases[BF16]["even"].engine(BF16, 64 * 7, "cuda"), 5e-2)


@pytest.mark.parametrize("dtype", FORMATS)
def test_long_decode(cases, dtype):
    for name in ("odd", "even"):
        R.run_long_decode(cases[dtype][name], cases[dtype][name].engine(dtype, 320, "cuda"), tolerance(dtype, name))


@pytest.mark.parametrize("name", ["even", "wide"])
def test_layer_path_and_native_executor_agree(cases, name, monkeypatch):
    """One call per step and one call per kernel launch the same kernels."""
    case = cases[BF16][name]
    toks = [case.tokens(n, n) for n in (140, 20, 33, 1)]

    def run():
        eng = case.engine(BF16, 512, "cuda")
        a = eng.replay([(i, t[:-1] or t, [0]) for i, t in enumerate(toks)], [2, 3])
        b = eng.replay([(i, t[-1:], [0]) for i, t in enumerate(toks[:2])] + [(9, toks[2], [32])])
        return torch.cat((a, b)), eng.model
    native, m1 = run()
    assert type(m1._native).__name__ == "MixerExecutor"
    monkeypatch.setenv("KSANA_DISABLE_NATIVE_EXECUTOR", "1")
    layers, m2 = run()
    assert m2._native is None
    assert torch.equal(native, layers)


@pytest.mark.parametrize("bs", [dict(), dict(split_fuse_token_num=9), dict(enable_async=True)])
def test_greedy_generation(cases, bs):
    greedy_check(cases[F32]["odd"], serve(cases[F32]["odd"], device="cuda", **bs), [1, 2, 30, 17, 41, 8], 6)


@pytest.mark.parametrize("mode", ["swap", "recompute"])
def test_preemption(cases, mode):
    eng = serve(cases[F32]["odd"], n_blocks=7, host_blocks=16 if mode == "swap" else 0, device="cuda",
                preempt_mode=0 if mode == "swap" else 1, launch_block_threshold=0.0, swapin_block_threshold=0.0)
    greedy_check(cases[F32]["odd"], eng, [14, 15, 13], 20)
    st = eng.sched.stats
    assert (st.preempt_swap if mode == "swap" else st.preempt_recompute) > 0


def test_shared_prefixes_and_drafts(cases):
    case = cases[F32]["stateless"]
    eng = serve(case, device="cuda", enable_auto_prefix_cache=True, enable_speculative_decoding=True)
    for _ in range(2):
        greedy_check(case, eng, [50, 33], 6)
    assert eng.cache.stats.prefix_hit_tokens >= 48


def test_generation_in_16_bits_follows_its_own_logits(cases):
    """bf16 generation through the scheduler, in one batch, picks tokens the oracle ranks at (or within rounding of) the
    top."""
    case = cases[BF16]["even"]
    eng = serve(case, device="cuda", dtype=BF16, split_fuse_token_num=50)
    prompts = [case.tokens(n, n) for n in (3, 70, 130, 41)]
    for p, r in zip(prompts, eng.generate(prompts, SamplingParams(topk=1, max_new_tokens=12, ignore_eos=True))):
        out = r.output_token_ids[0]
        lg = O.forward(case.cfg, case.w64, p + out)[len(p) - 1:-1]
        chosen = lg.gather(1, torch.tensor(out).unsqueeze(1))[:, 0]
        assert ((lg.max(1).values - chosen) < 0.25 * lg.std()).all()


@pytest.mark.parametrize("name", ["odd", "even", "wide"])
def test_routing_in_16_bits(cases, name):
    """With choices that rounding may turn, most positions still follow the oracle closely."""
    case = cases[F32][name]
    toks = case.tokens(150, 1)
    want = case.logits(toks)
    eng = case.engine(BF16, 192, "cuda")
    got = torch.cat([eng.replay([(1, toks[:120], list(range(120)))]), eng.replay([(1, toks[120:], list(range(30)))], [1])])
    err = ((got.double() - want) ** 2).mean(1).sqrt() / want.std()
    assert float(err.median()) < 4e-2 and float((err > 0.2).float().mean()) < 0.3
