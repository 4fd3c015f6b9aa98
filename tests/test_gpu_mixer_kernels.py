"""CUDA kernels of layers with mixers of their own sizes against plain 32-bit statements of the same operations."""
import pytest
import torch

from ksanallm_b200.engine.step_input import make_step_input

import molopel_oracle as M

pytestmark = pytest.mark.gpu
DEV = "cuda"
BS = 16


def steps(lens, q_lens, prefill, slots=None, seed=0):
    """Step metadata of sequences with ``lens`` tokens of which the last ``q_lens`` are new; pages are shuffled."""
    g = torch.Generator().manual_seed(seed)
    pages = [(n + BS - 1) // BS for n in lens]
    perm = torch.randperm(sum(pages) + 3, generator=g).tolist()
    tables, slot_map, pos, cu = [], [], [], [0]
    width = max(pages)
    for n, q in zip(lens, q_lens):
        t = [perm.pop() for _ in range((n + BS - 1) // BS)]
        tables.append(t + [0] * (width - len(t)))
        for p in range(n - q, n):
            slot_map.append(t[p // BS] * BS + p % BS)
            pos.append(p)
        cu.append(cu[-1] + q)
    meta = make_step_input([0] * cu[-1], pos, slot_map, cu, lens, tables, num_prefill=prefill, device=DEV,
                           state_slots=slots or list(range(len(lens))))
    return meta, tables, sum(pages) + 3


def fill_cache(tables, lens, ks, vs, blocks, hk, d, dv, dtype):
    cache = torch.zeros(blocks, hk * BS * (d + dv))
    K, V = cache[:, :hk * BS * d].view(blocks, hk, BS, d), cache[:, hk * BS * d:].view(blocks, hk, BS, dv)
    for t, n, k, v in zip(tables, lens, ks, vs):
        for p in range(n):
            K[t[p // BS], :, p % BS] = k[p]
            V[t[p // BS], :, p % BS] = v[p]
    return cache.to(dtype).to(DEV)


def attention_case(dtype, h, hk, d, dv, window, lens, q_lens, prefill, bias_max=50, rows=16, out_scale=0.7, seed=1):
    from ksanallm_b200.ops import cuda_mixer, reference as ref
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g).to(dtype).float()  # noqa: E731
    ks, vs = [rnd(n, hk, d) for n in lens], [rnd(n, hk, dv) for n in lens]
    qs = [rnd(q, h, d) for q in q_lens]
    rel = rnd(rows, h) * 2
    meta, tables, blocks = steps(lens, q_lens, prefill)
    cache = fill_cache(tables, lens, ks, vs, blocks, hk, d, dv, dtype)
    bias = ref.distance_bias(rel.to(DEV), bias_max, window or max(lens))
    out = torch.full((meta.total_tokens, h * dv + 8), 7.0, dtype=dtype, device=DEV)
    cuda_mixer.window_attention(torch.cat(qs).to(dtype).to(DEV), cache, meta, BS, hk, dv, d ** -0.5, window, bias,
                                out_scale, out[:, :h * dv])
    row = 0
    for n, ql, q, k, v in zip(lens, q_lens, qs, ks, vs):
        full = torch.zeros(n, h, d)
        full[n - ql:] = q
        want = M.windowed_attention(full.double(), k.double(), v.double(), d ** -0.5, window or n, rel.double(),
                                    bias_max)[n - ql:].flatten(1) * out_scale
        got = out[row:row + ql, :h * dv].double().cpu()
        tol = 2e-5 if dtype == torch.float32 else 1e-2
        assert (got - want).abs().max() < tol, (n, ql, (got - want).abs().max())
        row += ql
    assert (out[:, h * dv:] == 7).all()


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("h,hk,d,dv", [(4, 2, 64, 64), (6, 2, 128, 128), (3, 1, 96, 64), (2, 2, 48, 24), (4, 1, 64, 128),
                                       (2, 1, 20, 36)])
def test_window_attention_prompts(dtype, h, hk, d, dv):
    attention_case(dtype, h, hk, d, dv, 37, [150, 33, 20], [150, 17, 2], 3)


@pytest.mark.parametrize("window", [0, 1, 16, 128, 129, 300])
def test_window_attention_prompt_windows(window):
    attention_case(torch.bfloat16, 4, 2, 64, 64, window, [290, 140], [290, 9], 2)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("h,hk,d,dv", [(4, 2, 64, 64), (8, 1, 128, 128), (40, 2, 32, 64), (3, 3, 96, 128), (2, 1, 40, 72)])
def test_window_attention_single_tokens(dtype, h, hk, d, dv):
    attention_case(dtype, h, hk, d, dv, 60, [1 + 1, 17, 60, 61, 160, 161], [1] * 6, 0)


def test_window_attention_split_heads():
    """Long windows are cut into a cluster of CTAs whose parts are merged."""
    attention_case(torch.bfloat16, 8, 2, 128, 128, 1000, [1500, 900, 30], [1, 1, 1], 0)


def test_window_attention_mixed_step():
    attention_case(torch.bfloat16, 4, 2, 64, 64, 40, [130, 50, 77, 16], [100, 3, 1, 1], 2)


def features(x, act, dims, base, first, scale):
    if act == "silu":
        x = M.silu(x)
    if dims:
        x = M.rotate_half(x, first, dims, base)
    return x * scale


def linear_case(dtype, h, d, dv, lens, q_lens, prefill, act="none", dims=0, base=5e4, decay=None, key_scale=0.3, seed=2,
                tol=None):
    from ksanallm_b200.ops import cuda_mixer, reference as ref
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g).to(dtype).float()  # noqa: E731
    decay = decay or [1 - 0.5 ** (i % 6 + 1) for i in range(h)]
    B = len(lens)
    slots = list(range(B, 0, -1))
    meta, _, _ = steps(lens, q_lens, prefill, slots)
    width = h * (2 * d + dv)
    x = torch.cat([rnd(q, width) for q in q_lens])
    state = torch.randn(B + 1, h, d, dv, generator=g)
    dev_state = state.clone().to(DEV)
    xd = x.to(dtype).to(DEV)
    cut = (h * d, 2 * h * d)
    q, k, v = (t.unflatten(1, (h, -1)) for t in (xd[:, :cut[0]], xd[:, cut[0]:cut[1]], xd[:, cut[1]:]))
    rotary = ref.rotary_table(dims, base, max(lens), DEV) if dims else None
    out = cuda_mixer.linear_attention(q, k, v, dev_state, meta, torch.tensor(decay, device=DEV), act, rotary, key_scale)
    row = 0
    xs = x.double()
    for b, (n, ql) in enumerate(zip(lens, q_lens)):
        part = xs[row:row + ql]
        qq = features(part[:, :cut[0]].unflatten(1, (h, -1)), act, dims, base, n - ql, 1.0)
        kk = features(part[:, cut[0]:cut[1]].unflatten(1, (h, -1)), act, dims, base, n - ql, key_scale)
        vv = part[:, cut[1]:].unflatten(1, (h, -1))
        if act == "silu":
            vv = M.silu(vv).to(dtype).double()
        S0 = torch.zeros(h, d, dv, dtype=torch.float64) if n == ql else state[slots[b]].double()
        want, S = M.decayed_linear_attention(qq, kk, vv, decay, S0)
        scale = want.abs().max()
        tol_o = tol or (1e-5 if dtype == torch.float32 else 5e-3)
        assert (out[row:row + ql].double().cpu() - want).abs().max() < tol_o * scale, (b, n, ql)
        got = dev_state[slots[b]].double().cpu()
        assert (got - S).abs().max() < (1e-5 if dtype == torch.float32 else 1e-4) * S.abs().max(), (b, n, ql)
        row += ql
    assert torch.equal(dev_state[0].cpu(), state[0])  # a slot nobody holds


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("h,d,dv,dims", [(3, 64, 32, 64), (2, 64, 64, 0), (2, 128, 128, 96), (1, 128, 256, 128),
                                         (2, 40, 72, 32), (2, 24, 20, 12), (1, 16, 136, 16), (2, 192, 48, 192)])
def test_linear_attention_prompts(dtype, h, d, dv, dims):
    linear_case(dtype, h, d, dv, [300, 129, 40, 9], [300, 128, 17, 2], 4, "none", dims)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("h,d,dv", [(3, 64, 32), (2, 128, 128), (1, 96, 256), (2, 20, 18)])
def test_linear_attention_single_tokens(dtype, h, d, dv):
    linear_case(dtype, h, d, dv, [1, 2, 70, 200], [1, 1, 1, 1], 0, "silu")
    linear_case(dtype, h, d, dv, [5, 70], [1, 1], 0, "none", 16)


def test_linear_attention_extreme_decays():
    linear_case(torch.bfloat16, 4, 64, 64, [400, 70], [400, 60], 2, "silu", decay=[1.0, 0.0, 0.05, 0.9999])


def test_linear_attention_mixed_step():
    linear_case(torch.bfloat16, 2, 64, 64, [257, 30, 12, 90, 1], [200, 17, 3, 1, 1], 3, "silu")


def test_linear_attention_cuts_agree():
    """The state and the outputs do not depend on where a prompt was cut, beyond rounding."""
    from ksanallm_b200.ops import cuda_mixer
    h, d, dv, n = 2, 64, 64, 290
    g = torch.Generator().manual_seed(5)
    x = torch.randn(n, h * (2 * d + dv), generator=g).to(torch.bfloat16).to(DEV)
    decay = torch.tensor([0.9, 0.999], device=DEV)
    outs, states = [], []
    for cuts in ([n], [2, 100, 128, 1, 1, 58], [17] * 17 + [1], [130, 160]):
        state, done, rows = torch.randn(1, h, d, dv, device=DEV), 0, []
        for c in cuts:
            meta, _, _ = steps([done + c], [c], 0 if c == 1 and done else 1, [0])
            y = x[done:done + c]
            rows.append(cuda_mixer.linear_attention(y[:, :h * d].unflatten(1, (h, d)), y[:, h * d:2 * h * d].unflatten(1, (h, d)),
                                                    y[:, 2 * h * d:].unflatten(1, (h, dv)), state, meta, decay, "silu", None, 1.0))
            done += c
        outs.append(torch.cat(rows).float())
        states.append(state)
    for o, s in zip(outs[1:], states[1:]):
        assert (s - states[0]).abs().max() < 1e-4 * states[0].abs().max()
        assert (o - outs[0]).abs().max() < 8e-3 * outs[0].abs().max()


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("rows,H", [(5, 256), (3, 1000), (4, 4096), (2, 9000), (3, 333)])
def test_layer_norm_stream(dtype, rows, H):
    from ksanallm_b200.ops import cuda_mixer
    g = torch.Generator().manual_seed(3)
    x = torch.randn(rows, H, generator=g).to(dtype)
    r = torch.randn(rows, H, generator=g) * 3 + 5
    w = torch.randn(H, generator=g).to(dtype)
    stream = r.clone().to(DEV)
    y = cuda_mixer.layer_norm(x.to(DEV), w.to(DEV), None, 1e-5, stream, dtype)
    total = r.double() + x.double()
    assert (stream.double().cpu() - total).abs().max() < 1e-5
    want = M.layer_norm(total, w.double(), 1e-5)
    assert (y.double().cpu() - want).abs().max() < (2e-5 if dtype == torch.float32 else 2e-2) * want.abs().max()
    y2 = cuda_mixer.layer_norm(r.to(DEV), w.to(DEV), None, 1e-5, None, dtype)
    want = M.layer_norm(r.double(), w.double(), 1e-5)
    assert (y2.double().cpu() - want).abs().max() < (2e-5 if dtype == torch.float32 else 2e-2) * want.abs().max()


def test_layer_norm_bias_bf16_stream():
    from ksanallm_b200.ops import cuda_mixer, reference as ref
    g = torch.Generator().manual_seed(3)
    x, r, w, b = (torch.randn(*s, generator=g).to(torch.bfloat16) for s in ((4, 768), (4, 768), (768,), (768,)))
    r1, r2 = r.clone().to(DEV), r.clone()
    y = cuda_mixer.layer_norm(x.to(DEV), w.to(DEV), b.to(DEV), 1e-5, r1)
    want = ref.layer_norm(x, w, b, 1e-5, r2)
    assert torch.equal(r1.cpu(), r2)
    assert (y.float().cpu() - want.float()).abs().max() < 5e-2


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("gate,concat", [("silu", False), ("sigmoid", True)])
@pytest.mark.parametrize("h,dv", [(4, 64), (3, 50), (2, 256)])
def test_gated_norm(dtype, gate, concat, h, dv):
    from ksanallm_b200.ops import cuda_mixer
    g = torch.Generator().manual_seed(4)
    o = torch.randn(7, h, dv, generator=g).to(dtype)
    gt = torch.randn(7, h * dv + 8, generator=g).to(dtype)
    w = torch.randn(h * dv, generator=g) if concat else None
    out = torch.zeros(7, h * dv + 4, dtype=dtype, device=DEV)
    cuda_mixer.gated_norm(o.to(DEV), gt.to(DEV)[:, :h * dv], w.to(DEV) if concat else None, 1e-3, gate, 1.3, out[:, :h * dv])
    od = o.double()
    n = M.unit_rms(od.flatten(1), 1e-3) * w.double() if concat else M.unit_rms(od, 1e-3).flatten(1)
    gd = gt[:, :h * dv].double()
    want = n * (M.silu(gd) if gate == "silu" else M.sigmoid(gd)) * 1.3
    assert (out[:, :h * dv].double().cpu() - want).abs().max() < (1e-5 if dtype == torch.float32 else 2e-2) * want.abs().max()
    assert (out[:, h * dv:] == 0).all()


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("h,hk,d,dv", [(4, 2, 64, 64), (3, 1, 20, 36), (2, 2, 128, 96)])
def test_qk_norm_cache(dtype, h, hk, d, dv):
    from ksanallm_b200.ops import cuda_mixer, reference as ref
    g = torch.Generator().manual_seed(6)
    meta, tables, blocks = steps([40, 7], [23, 7], 2)
    T = meta.total_tokens
    x = torch.randn(T, h * d + hk * (d + dv) + 8, generator=g).to(dtype)
    qw, kw = torch.randn(d, generator=g), torch.randn(d, generator=g)
    xd = x.clone().to(DEV)

    def parts(t):
        return (t[:, :h * d].unflatten(1, (h, d)), t[:, h * d:(h + hk) * d].unflatten(1, (hk, d)),
                t[:, (h + hk) * d:(h + hk) * d + hk * dv].unflatten(1, (hk, dv)))

    cache = torch.full((blocks, hk * BS * (d + dv)), 9.0, dtype=dtype, device=DEV)
    cuda_mixer.qk_norm_cache(*parts(xd), meta.slot_mapping, cache, BS, qw.to(DEV), kw.to(DEV), 1e-4)
    q, k, v = (t.double() for t in parts(x))
    tol = 1e-5 if dtype == torch.float32 else 3e-2
    assert (parts(xd)[0].double().cpu() - M.unit_rms(q, 1e-4) * qw.double()).abs().max() < tol
    K, V = ref.split_kv_cache(cache.cpu(), hk, BS, d, dv)
    slots = meta.slot_mapping.cpu().long()
    assert (K[slots // BS, :, slots % BS].double() - M.unit_rms(k, 1e-4) * kw.double()).abs().max() < tol
    assert torch.equal(V[slots // BS, :, slots % BS], parts(x)[2])
    untouched = torch.ones(blocks * BS, dtype=torch.bool)
    untouched[slots] = False
    assert (K.permute(0, 2, 1, 3).reshape(blocks * BS, -1)[untouched] == 9).all()


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("width", [96, 52])
def test_gelu_softcap_embedding(dtype, width):
    from ksanallm_b200.ops import cuda_mixer
    g = torch.Generator().manual_seed(7)
    x = (torch.randn(9, 2 * width, generator=g) * 3).to(dtype)
    want = M.gelu_tanh(x[:, :width].double()) * x[:, width:].double()
    got = cuda_mixer.gelu_and_mul(x.to(DEV)).double().cpu()
    assert (got - want).abs().max() < (1e-5 if dtype == torch.float32 else 1e-2) * want.abs().max()
    y = torch.randn(4, width, generator=g) * 60
    assert (cuda_mixer.softcap(y.to(DEV), 25.0).double().cpu() - 25 * torch.tanh(y.double() / 25)).abs().max() < 1e-4
    table = torch.randn(11, width, generator=g).to(dtype)
    ids = torch.tensor([3, 0, 10], dtype=torch.int32)
    e = cuda_mixer.embedding(ids.to(DEV), table.to(DEV), 7.5, torch.float32).cpu()
    assert torch.equal(e, table[ids.long()].float() * 7.5)


@pytest.mark.parametrize("rows,K,ff", [(700, 256, 512), (130, 136, 48)])
def test_gelu_gate_as_gemm_epilogue(rows, K, ff):
    from ksanallm_b200.ops import cuda
    g = torch.Generator().manual_seed(8)
    x, w = torch.randn(rows, K, generator=g).to(torch.bfloat16), (torch.randn(2 * ff, K, generator=g) * 0.2).to(torch.bfloat16)
    got = cuda.gemm_bf16_swiglu(x.to(DEV), cuda.interleave_gate_up(w.to(DEV)), "gelu_tanh").double().cpu()
    want = M.gelu_tanh(x.double() @ w[:ff].double().T) * (x.double() @ w[ff:].double().T)
    assert (got - want).abs().max() < 1e-2 * want.abs().max()
