"""Givirax on the GPU: its kernels one by one, whole models through the engine's own step function against the plain
oracle in both number formats, and generation through the scheduler."""
import pytest
import torch

import givirax_cases as C
import givirax_oracle as O
import replay_cases as R
from givirax_cases_attention import check, feed
from ksanallm_b200 import ops
from ksanallm_b200.engine.sampling_params import SamplingParams
from ksanallm_b200.ops import reference as ref
from test_givirax import greedy_check, serve

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
FORMATS = [(F32, 1e-4), (BF16, 6e-2)]


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    return {n: C.Case(tmp_path_factory.mktemp(n), n) for n in C.CASES}


# ---- attention ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("window,keep", [(1, 0), (1, 1), (16, 0), (16, 16), (17, 5), (40, 18), (128, 3), (33, 130), (300, 3)])
def test_window_and_first_token_edges(dtype, window, keep):
    check(dtype, "cuda", window, keep)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("h,hk,d", [(6, 3, 128), (34, 2, 64), (17, 1, 128), (2, 2, 40), (5, 1, 96), (4, 4, 16), (2, 1, 20)])
def test_head_sizes(dtype, h, hk, d):
    check(dtype, "cuda", 37, 6, h=h, hk=hk, d=d)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("window,keep", [(100, 7), (200, 150), (513, 1), (5000, 0)])
def test_long_prompts_and_splits(dtype, window, keep):
    """Prompts over many tiles of keys, and single tokens whose pages are shared out over a cluster."""
    n, d = 1100, 64
    g = torch.Generator().manual_seed(window)
    q, k = torch.randn(n, 4, d, generator=g).to(dtype).float(), torch.randn(n, 2, d, generator=g).to(dtype).float()
    rows = [0, 1, 150, 151, 207, 208, 700, n - 22] + list(range(n - 20, n))
    got = feed(q, k, [n - 20] + [1] * 20, dtype, "cuda", 0.4, window, keep).view(n, 4, d)
    for i in rows:
        js = torch.tensor([j for j in range(i + 1) if O.sees(i, j, window, keep)])
        for h in range(4):
            keys = k[js, h // 2].double()
            p = torch.softmax(keys @ q[i, h].double() * 0.4, 0)
            assert (got[i, h] - p @ keys).abs().max() < (2e-5 if dtype == F32 else 2e-2), (i, h)


# ---- routed experts -------------------------------------------------------------------------------------------
@pytest.mark.parametrize("T,E,top", [(1, 5, 2), (37, 12, 3), (200, 1, 1), (9, 700, 9), (64, 40, 40)])
def test_router(T, E, top):
    g = torch.Generator().manual_seed(E)
    z, b = torch.randn(T, (E + 7) // 8 * 8, generator=g), torch.randn(E, generator=g)
    z[:, E:] = 50.0
    ids, w = ops.moe_topk(z.cuda(), E, top, b.cuda())
    want, ww = ref.moe_topk(z.double(), E, top, b)
    assert torch.equal(ids.cpu(), want) and (w.cpu() - ww).abs().max() < 1e-6


@pytest.mark.parametrize("n,E,offset,ids_of", [(1, 3, 0, 3), (2000, 12, 0, 12), (5000, 40, 8, 64), (33000, 16, 0, 16), (777, 1, 0, 1)])
def test_sort_by_expert(n, E, offset, ids_of):
    from ksanallm_b200.ops import cuda
    ids = torch.randint(0, ids_of, (n,), dtype=torch.int32, device="cuda")
    offs, pos, src = (torch.full((m,), -7, dtype=torch.int32, device="cuda") for m in (E + 1, n, n))
    assert cuda.lib().ksana_moe_sort(ids.data_ptr(), n, offset, E, offs.data_ptr(), pos.data_ptr(), src.data_ptr(),
                                     torch.cuda.current_stream().cuda_stream) == 0
    ids, offs, pos, src = ids.cpu().long() - offset, offs.cpu(), pos.cpu().long(), src.cpu().long()
    local = (ids >= 0) & (ids < E)
    assert offs.tolist() == [int((local & (ids < e)).sum()) for e in range(E + 1)]
    assert (pos[~local] == -1).all() and pos[local].sort().values.tolist() == list(range(int(local.sum())))
    assert torch.equal(src[pos[local]], local.nonzero()[:, 0])
    assert ((pos[local] >= offs[ids[local]]) & (pos[local] < offs[ids[local] + 1])).all()


@pytest.mark.parametrize("dtype,T,E,top,H,I", [
    (BF16, 1, 4, 2, 128, 64), (BF16, 300, 6, 3, 264, 104), (BF16, 129, 9, 2, 128, 48), (BF16, 40, 3, 2, 92, 22),
    (F32, 150, 5, 3, 92, 22), (F32, 1, 11, 2, 248, 72), (F32, 70, 2, 1, 128, 48)])
def test_expert_rows(dtype, T, E, top, H, I):
    g = torch.Generator().manual_seed(T + E)
    x = torch.randn(T, H, generator=g).to(dtype).cuda()
    w1 = (torch.randn(E, 2 * I, H, generator=g) / H ** 0.5).to(dtype).cuda()
    w2 = (torch.randn(E, H, I, generator=g) / I ** 0.5).to(dtype).cuda()
    ids = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)]).int().cuda()
    y, pos = ops.moe_expert_rows(x, ids, w1, w2)
    want, _ = ref.moe_expert_rows(x.double().cpu(), ids.cpu(), w1.double().cpu(), w2.double().cpu())
    err = (y[pos.long()].double().cpu() - want).abs().max() / want.abs().max()
    assert err < (2e-6 if dtype == F32 else 2e-2)


# ---- the stream -----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("H", [128, 92, 4096, 8192, 30])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("center", [False, True])
def test_stream_norm(H, dtype, center):
    g = torch.Generator().manual_seed(H)
    T, k = 5, 3
    x, y = torch.randn(T, H, generator=g).to(dtype), torch.randn(T * k, H, generator=g).to(dtype)
    stream, rows, vec = torch.randn(T, H, generator=g), torch.randn(T, H, generator=g), torch.randn(H, generator=g)
    w = torch.randn(H, generator=g).to(dtype)
    pos, wts = torch.randperm(T * k, generator=g).int(), torch.rand(T, k, generator=g)
    pos[4] = -1
    for use in range(8):
        more = dict(add_rows=rows if use & 1 else None, add_vec=vec if use & 2 else None,
                    routed=(y, pos, wts) if use & 4 else None)
        out = torch.empty_like(stream)
        want = ref.stream_norm(x, w, 1e-5, center, stream, out, F32, **more)
        dev = {n: (tuple(t.cuda() for t in v) if isinstance(v, tuple) else v.cuda()) if v is not None else None
               for n, v in more.items()}
        s = stream.cuda()
        got = ops.stream_norm(x.cuda(), w.cuda(), 1e-5, center, s, s, dtype, **dev)
        assert (s.cpu() - out).abs().max() < 1e-5
        assert (got.float().cpu() - want).abs().max() < (2e-5 if dtype == F32 else 4e-2)
    a = torch.empty_like(stream.cuda())
    got = ops.stream_norm(None, w.cuda(), 1e-5, center, stream.cuda(), a, dtype, add_vec=vec.cuda())
    assert torch.equal(a.cpu(), stream + vec)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("T,hk,d,I,gated", [(1, 2, 64, 160, 0), (70, 1, 20, 76, 0), (33, 3, 128, 0, 0), (40, 0, 8, 104, 1), (9, 2, 8, 30, 1)])
def test_cache_append_beside_the_activation(dtype, T, hk, d, I, gated):
    g = torch.Generator().manual_seed(T + d)
    cols = hk * d + (2 * I if gated else I)
    x = torch.randn(T, cols + 16, generator=g).to(dtype)
    slots = torch.randperm(T + 20, generator=g)[:T].int()
    slots[0] = -1 if T > 1 else slots[0]
    nb = (T + 20 + 15) // 16

    def run(dev):
        xx, cache = x.to(dev), torch.zeros(nb, max(hk, 1) * 16 * d, dtype=dtype, device=dev)
        out = torch.zeros(T, I + 8, dtype=dtype, device=dev)
        k = xx[:, 8:8 + hk * d].unflatten(1, (hk, d)) if hk else None
        u = xx[:, 8 + hk * d:8 + cols] if I else None
        if dev == "cpu":
            keep = slots >= 0
            ref.append_act(k[keep] if hk else None, None, slots[keep], cache, 16, None)
            ref.append_act(None, u, slots, cache, 16, out[:, 8:8 + I], bool(gated))
        else:
            ops.append_act(k, u, slots.to(dev), cache, 16, out[:, 8:8 + I] if I else None, bool(gated))
        return cache.cpu().double(), out.cpu().double()
    (c0, o0), (c1, o1) = run("cpu"), run("cuda")
    assert torch.equal(c0, c1) and (o0 - o1).abs().max() < (1e-6 if dtype == F32 else 3e-2)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_embedding_with_positions(dtype):
    ids, pos = torch.randint(0, 50, (9,), dtype=torch.int32), torch.tensor([0, 1, 2, 19, 18, 5, 5, 7, 0], dtype=torch.int32)
    table, ptab = torch.randn(50, 36).to(dtype), torch.randn(20, 36).to(dtype)
    got = ops.embedding(ids.cuda(), table.cuda(), 7.5, F32, pos.cuda(), ptab.cuda()).cpu()
    assert (got - (table.float()[ids.long()] * 7.5 + ptab.float()[pos.long()])).abs().max() < 1e-5


# ---- whole models ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype,tol", FORMATS)
@pytest.mark.parametrize("name", list(C.CASES))
def test_portions(cases, name, dtype, tol):
    R.run_portions(cases[name], cases[name].engine(dtype, 192, "cuda"), tol)


@pytest.mark.parametrize("dtype,tol", FORMATS)
@pytest.mark.parametrize("name", list(C.CASES))
def test_batches_and_reuse(cases, name, dtype, tol):
    R.run_batches(cases[name], cases[name].engine(dtype, 64 * 7, "cuda"), tol)


@pytest.mark.parametrize("dtype,tol", FORMATS)
def test_long_decode(cases, dtype, tol):
    for name in ("odd", "even"):
        R.run_long_decode(cases[name], cases[name].engine(dtype, 320, "cuda"), tol)


def test_layer_path_and_native_executor_agree(cases, monkeypatch):
    """One call per step and one call per kernel launch the same kernels."""
    case = cases["even"]
    toks = [case.tokens(n, n) for n in (140, 20, 33)]

    def run():
        eng = case.engine(BF16, 512, "cuda")
        a = eng.replay([(i, t[:-1], [len(t) - 2]) for i, t in enumerate(toks)])
        b = eng.replay([(i, t[-1:], [0]) for i, t in enumerate(toks)])
        return torch.cat((a, b)), eng.model
    native, m1 = run()
    assert type(m1._native).__name__ == "MixerExecutor"
    monkeypatch.setenv("KSANA_DISABLE_NATIVE_EXECUTOR", "1")
    layers, m2 = run()
    assert m2._native is None
    assert torch.equal(native, layers)


@pytest.mark.parametrize("bs", [dict(), dict(split_fuse_token_num=9), dict(enable_async=True)])
def test_greedy_generation(cases, bs):
    greedy_check(cases["odd"], serve(cases["odd"], device="cuda", **bs), [1, 2, 30, 17, 41, 8], 8)


@pytest.mark.parametrize("mode", ["swap", "recompute"])
def test_preemption(cases, mode):
    eng = serve(cases["odd"], n_blocks=7, host_blocks=16 if mode == "swap" else 0, device="cuda",
                preempt_mode=0 if mode == "swap" else 1, launch_block_threshold=0.0, swapin_block_threshold=0.0)
    greedy_check(cases["odd"], eng, [14, 15, 13], 20)
    st = eng.sched.stats
    assert (st.preempt_swap if mode == "swap" else st.preempt_recompute) > 0


def test_shared_prefixes_and_drafts(cases):
    case = cases["flat"]
    eng = serve(case, device="cuda", enable_auto_prefix_cache=True, enable_speculative_decoding=True)
    for _ in range(2):
        greedy_check(case, eng, [50, 33], 6)
    assert eng.cache.stats.prefix_hit_tokens >= 48


def test_generation_in_16_bits_follows_its_own_logits(cases):
    """bf16 generation through the scheduler, in one batch, picks tokens the oracle ranks at (or within rounding of) the
    top."""
    case = cases["even"]
    eng = serve(case, device="cuda", dtype=BF16, split_fuse_token_num=50)
    prompts = [case.tokens(n, n) for n in (3, 70, 130, 41)]
    for p, r in zip(prompts, eng.generate(prompts, SamplingParams(topk=1, max_new_tokens=12, ignore_eos=True))):
        out = r.output_token_ids[0]
        lg = O.forward(case.cfg, case.w64, p + out)[len(p) - 1:-1]
        chosen = lg.gather(1, torch.tensor(out).unsqueeze(1))[:, 0]
        assert ((lg.max(1).values - chosen) < 0.25 * lg.std()).all()
