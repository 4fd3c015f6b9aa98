"""Vibunex on the GPU: its kernels one by one, whole models through the engine's own step function against the plain oracle
in both number formats, and generation through the scheduler."""
import pytest
import torch

import replay_cases as R
import vibunex_cases as C
import vibunex_mechanisms as M
import vibunex_oracle as O
from ksanallm_b200.engine.sampling_params import SamplingParams
from test_vibunex import greedy_check, serve

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
FORMATS = [F32, BF16]


def tolerance(dtype):
    """16 bits: about twice what the CPU path, computing in 32 bits and storing in 16, is off by."""
    return 1e-4 if dtype == F32 else 8e-2


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    """By number format: 16-bit models are compared without discrete choices (see Case)."""
    return {t: {n: C.Case(tmp_path_factory.mktemp(n), n, every_expert=t == BF16) for n in C.CASES} for t in (F32, BF16)}


# ---- mechanisms -----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", FORMATS)
@pytest.mark.parametrize("kind", ["random", "far", "sink", "swap"])
@pytest.mark.parametrize("H,G,d,dv,dims", [(4, 2, 64, 64, 16), (32, 8, 128, 128, 64), (6, 2, 20, 36, 12), (34, 2, 32, 128, 8),
                                           (16, 16, 64, 40, 64)])
def test_attention_with_mixed_weights(dtype, kind, H, G, d, dv, dims):
    M.attention_case(dtype, "cuda", H, G, d, dv, dims, kind=kind)


@pytest.mark.parametrize("H,G,d,dv", [(1, 1, 8, 8), (3, 1, 24, 128), (64, 4, 16, 16), (33, 11, 40, 72), (24, 8, 72, 64), (7, 7, 128, 64),
                                      (16, 8, 64, 64), (16, 4, 40, 128), (16, 2, 128, 24), (32, 16, 32, 64), (32, 4, 128, 72),
                                      (64, 16, 64, 16), (64, 8, 128, 128), (65, 13, 16, 24), (64, 64, 16, 16), (4, 1, 136, 32)])
def test_attention_sizes(H, G, d, dv):
    """Groups of 1 to 16 heads, heads of every size, both forms of the weights' kernel, and what only the general kernel takes."""
    M.attention_case(BF16, "cuda", H, G, d, dv, 8, kind="random")


@pytest.mark.parametrize("hk", [4, 8])
def test_weights_written_out_in_several_rounds(hk):
    """Prompts whose weights do not fit into one round's budget, blocks of several sequences in a round."""
    from ksanallm_b200.engine.step_input import make_step_input
    from ksanallm_b200.ops import cuda_talking, reference as ref
    g = torch.Generator(device="cuda").manual_seed(3)
    h, d, dv, lens, news = 64, 32, 16, [4100, 40, 2500], [4100, 40, 1200]
    cu = [0, 4100, 4140, 5340]
    table = torch.zeros(3, 260, dtype=torch.int32)
    for b, first in enumerate((1, 300, 310)):
        table[b, :(lens[b] + 15) // 16] = torch.arange(first, first + (lens[b] + 15) // 16)
    meta = make_step_input([0] * 5340, [p for n, m in zip(lens, news) for p in range(n - m, n)], [0] * 5340, cu, lens, table,
                           num_prefill=3, device="cuda")
    q = torch.randn(5340, h, d, generator=g, device="cuda").bfloat16()
    cache = torch.randn(480, 16 * hk * (d + dv), generator=g, device="cuda").bfloat16()
    sink, talk = torch.randn(h, generator=g, device="cuda"), torch.randn(h, h, generator=g, device="cuda").bfloat16().float()
    out = torch.empty(5340, h * dv, dtype=BF16, device="cuda")
    cuda_talking.talking_attention(q, cache, meta, 16, hk, dv, 0.3, sink, talk, 1.0, out)
    for b, i in ((0, 0), (0, 127), (0, 2000), (0, 4099), (1, 39), (2, 0), (2, 600), (2, 1199)):
        n = lens[b] - news[b] + i + 1
        one = ref.talking_attention(q[cu[b] + i:cu[b] + i + 1], cache, table[b:b + 1].cuda(), torch.tensor([0, 1]), torch.tensor([n]),
                                    16, hk, dv, 0.3, sink, talk)
        got = out[cu[b] + i].float()
        assert (got - one.flatten().float()).abs().max() < 1e-2 * one.float().abs().max(), (b, i)


@pytest.mark.parametrize("dtype", FORMATS)
@pytest.mark.parametrize("W", [128, 84, 13, 4096])
def test_token_mix(dtype, W):
    M.token_mix_case(dtype, "cuda", W)


@pytest.mark.parametrize("dtype", FORMATS)
@pytest.mark.parametrize("h,d", [(4, 64), (3, 32), (2, 128), (5, 24), (2, 72), (3, 20), (1, 8), (2, 136), (3, 7)])
def test_time_mixing(dtype, h, d):
    M.recurrence_case(dtype, "cuda", h, d)


@pytest.mark.parametrize("dtype", FORMATS)
@pytest.mark.parametrize("z", [-9.0, 0.5, 3.0])
@pytest.mark.parametrize("h,d", [(2, 64), (3, 16)])
def test_slow_and_fast_decays(dtype, z, h, d):
    M.recurrence_case(dtype, "cuda", h, d, z_mean=z)


@pytest.mark.parametrize("dtype", FORMATS)
@pytest.mark.parametrize("d", [64, 24])
def test_an_early_token_is_read_through_all_decays(dtype, d):
    M.recurrence_case(dtype, "cuda", 2, d, z_mean=-6.0, probe=True)


def test_slow_decays_keep_their_precision():
    M.recurrence_case(F32, "cuda", 2, 32, n=1500, z_mean=-14.0, tol=3e-6)


@pytest.mark.parametrize("dtype", FORMATS)
@pytest.mark.parametrize("h,d", [(4, 64), (2, 20), (3, 128)])
def test_time_mixing_batch(dtype, h, d):
    M.recurrence_batch(dtype, "cuda", h, d)


@pytest.mark.parametrize("n", [16, 24, 64])
def test_tanh_parts(n):
    M.tanh_case("cuda", n)


@pytest.mark.parametrize("dtype", FORMATS)
@pytest.mark.parametrize("h,d", [(64, 64), (3, 20), (2, 136), (1, 7), (9, 16), (2, 300)])
def test_head_norm(dtype, h, d):
    M.head_norm_case(dtype, "cuda", h, d)


@pytest.mark.parametrize("dtype", FORMATS)
@pytest.mark.parametrize("H", [128, 84, 1028, 2048, 4096, 8192, 13, 9000])
def test_gated_residual(dtype, H):
    M.residual_case(dtype, "cuda", H)


@pytest.mark.parametrize("experts,top", [(8, 3), (1, 1), (5, 5), (600, 20)])
def test_router(experts, top):
    M.router_case("cuda", experts, top)


@pytest.mark.parametrize("dtype,T,E,top,H,I", [(BF16, 300, 6, 3, 264, 104), (BF16, 40, 3, 2, 92, 22), (F32, 70, 5, 2, 92, 24),
                                               (BF16, 33, 4, 4, 128, 40), (BF16, 1, 9, 1, 64, 256)])
def test_plain_experts(dtype, T, E, top, H, I):
    M.expert_case(dtype, "cuda", T, E, top, H, I)


@pytest.mark.parametrize("dtype", FORMATS)
@pytest.mark.parametrize("cols", [104, 13, 2048])
def test_squared_relu(dtype, cols):
    M.relu2_case(dtype, "cuda", cols)


# ---- whole models ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", FORMATS)
@pytest.mark.parametrize("name", list(C.CASES))
def test_portions(cases, name, dtype):
    R.run_portions(cases[dtype][name], cases[dtype][name].engine(dtype, 192, "cuda"), tolerance(dtype))


@pytest.mark.parametrize("dtype", FORMATS)
@pytest.mark.parametrize("name", list(C.CASES))
def test_batches_and_reuse(cases, name, dtype):
    R.run_batches(cases[dtype][name], cases[dtype][name].engine(dtype, 64 * 7, "cuda"), tolerance(dtype))


@pytest.mark.parametrize("dtype", FORMATS)
def test_long_decode(cases, dtype):
    for name in ("odd", "even"):
        R.run_long_decode(cases[dtype][name], cases[dtype][name].engine(dtype, 320, "cuda"), tolerance(dtype))


@pytest.mark.parametrize("name", ["even", "wide", "one"])
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
