#!/usr/bin/env python
"""Stand-alone cases of the hot kernels with achieved bandwidth / FLOP rates (CUDA events, L2 flushed between
iterations by rotating through operand copies larger than L2). Also the entry point used for `ncu` captures:
each case is small (at most a few GB on the device) and launches its kernel a handful of times.

    python benchmarks/kernel_cases.py gemm [M N K]            # tcgen05 bf16 GEMM
    python benchmarks/kernel_cases.py gemm_fp8 [M N K]        # block-scaled fp8 GEMM
    python benchmarks/kernel_cases.py gemm_int4 [M N K]       # int4 weight-only GEMM (in-pipeline dequant)
    python benchmarks/kernel_cases.py decode [B ctx h hk]     # paged split-KV decode attention
    python benchmarks/kernel_cases.py prefill [T h hk]        # tcgen05 paged prefill attention
    python benchmarks/kernel_cases.py mla [B ctx h q_len]     # tcgen05 absorbed-MLA decode over the latent cache
    python benchmarks/kernel_cases.py rmsnorm [T H]
    python benchmarks/kernel_cases.py moe [T E k H I]
    python benchmarks/kernel_cases.py window_prefill [T h hk d dv window keep shared cap]   # layers with mixers of their own sizes
    python benchmarks/kernel_cases.py window_decode [B ctx h hk d dv window keep shared cap]
    python benchmarks/kernel_cases.py linear_prefill [T h d dv rotary]
    python benchmarks/kernel_cases.py linear_decode [B h d dv rotary]
    python benchmarks/kernel_cases.py mixer_rows [T H h hk d]
    python benchmarks/kernel_cases.py latent_prefill [T h dim rot vdim rank]
    python benchmarks/kernel_cases.py latent_decode [B ctx h dim rot vdim rank]
    python benchmarks/kernel_cases.py recurrence_prefill [T C blocks taps sequences]
    python benchmarks/kernel_cases.py recurrence_decode [B C blocks taps]
    python benchmarks/kernel_cases.py ladusun_rows [T H streams h hk d rank rot]
    python benchmarks/kernel_cases.py talking_prefill [T h hk d dv]
    python benchmarks/kernel_cases.py talking_decode [B ctx h hk d dv]
    python benchmarks/kernel_cases.py timemix_prefill [T heads dim sequences]
    python benchmarks/kernel_cases.py timemix_decode [B heads dim]
    python benchmarks/kernel_cases.py vibunex_rows [T H h hk d]
    python benchmarks/kernel_cases.py all
"""
import json
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
from ksanallm_b200.engine.step_input import make_step_input  # noqa: E402
from ksanallm_b200.ops import cuda, cuda_latent, cuda_mixer, cuda_moe, cuda_recurrence, cuda_talking, cuda_timemix  # noqa: E402
from ksanallm_b200.ops import reference as ref  # noqa: E402

DEV = "cuda"


def peaks():
    p = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
    f = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "MEASURED_PEAKS.json")
    if os.path.exists(f):
        d = json.load(open(f))
        p["hbm_gbs"], p["bf16_tflops"] = float(d["hbm_gbs"]), float(d["bf16_tflops"])
    return p


def timeit(fn, iters=10, warm=3):
    for i in range(warm):
        fn(i)
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for i in range(iters):
        fn(warm + i)
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / iters * 1e3  # us


def timeit_graph(fn, count=48):
    """For kernels shorter than their launch from Python: ``count`` launches in one CUDA graph."""
    for i in range(count):
        fn(i)
    torch.cuda.synchronize()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        for i in range(count):
            fn(i)
    return timeit(lambda i: graph.replay(), iters=5) / count


def args_or(default):
    a = [int(x) for x in sys.argv[2:]]
    return a + default[len(a):]


def case_gemm():
    M, N, K = args_or([4096, 4096, 4096])
    nw = max(2, int(300e6 // (N * K * 2)) + 1)
    ws = [(torch.randn(N, K, device=DEV) * 0.05).to(torch.bfloat16) for _ in range(nw)]
    x = torch.randn(M, K, device=DEV).to(torch.bfloat16)
    us = timeit(lambda i: cuda.gemm_bf16(x, ws[i % nw]))
    us_lib = timeit(lambda i: torch.nn.functional.linear(x, ws[i % nw]))
    fl = 2.0 * M * N * K
    by = (M * K + N * K + M * N) * 2
    p = peaks()
    return dict(kernel="gemm_bf16", M=M, N=N, K=K, us=round(us, 1), tflops=round(fl / us / 1e6, 1),
                frac_of_measured_bf16=round(fl / us / 1e6 / p["bf16_tflops"], 3), gbs=round(by / us / 1e3, 1),
                frac_of_measured_hbm=round(by / us / 1e3 / p["hbm_gbs"], 3), cublas_us=round(us_lib, 1))


def case_gemm_fp8():
    M, N, K = args_or([4096, 4096, 4096])
    nw = max(2, int(300e6 // (N * K)) + 1)
    wq, wsc = [], []
    for _ in range(nw):
        q, s = ref.quant_fp8_block_weight(torch.randn(N, K, device=DEV) * 0.05)
        wq.append(q)
        wsc.append(s)
    x = torch.randn(M, K, device=DEV).to(torch.bfloat16)
    xq, xs = cuda.quant_fp8_group(x)
    us = timeit(lambda i: cuda.gemm_fp8_block(xq, xs, wq[i % nw], wsc[i % nw]))
    fl = 2.0 * M * N * K
    by = M * K + N * K + M * N * 2
    p = peaks()
    return dict(kernel="gemm_fp8_block", M=M, N=N, K=K, us=round(us, 1), tflops=round(fl / us / 1e6, 1),
                gbs=round(by / us / 1e3, 1), frac_of_measured_hbm=round(by / us / 1e3 / p["hbm_gbs"], 3),
                frac_of_2x_measured_bf16=round(fl / us / 1e6 / (2 * p["bf16_tflops"]), 3))


def case_gemm_int4():
    from ksanallm_b200.ops import cuda_int4
    M, N, K = args_or([16, 8192, 8192])
    nw = max(2, int(300e6 // (N * K // 2)) + 1)
    qs = [ref.quant_int4_group(torch.randn(N, K, device=DEV) * 0.05, 128) for _ in range(nw)]
    qs = [(ref.tile_int4(p), s, z, cuda_int4.pack_scale_zero(s, z)) for p, s, z in qs]
    x = torch.randn(M, K, device=DEV).to(torch.bfloat16)
    us = timeit(lambda i: cuda_int4.linear_int4(x, *qs[i % nw][:3], None, 128, sz=qs[i % nw][3]))
    by = N * K / 2 + N * (K // 128) * 8 + M * K * 2 + M * N * 2
    fl = 2.0 * M * N * K
    p = peaks()
    return dict(kernel="gemm_int4", M=M, N=N, K=K, us=round(us, 1), gbs=round(by / us / 1e3, 1),
                frac_of_measured_hbm=round(by / us / 1e3 / p["hbm_gbs"], 3), tflops=round(fl / us / 1e6, 1),
                frac_of_measured_bf16=round(fl / us / 1e6 / p["bf16_tflops"], 3))


def _attn_setup(q_lens, kv_lens, h, hk):
    bs, d = 16, 128
    nblk = [(L + bs - 1) // bs for L in kv_lens]
    total = sum(nblk) + 1
    cache = (torch.randn(total, 2, hk, bs, d, device=DEV) * 0.3).to(torch.bfloat16)
    bt = torch.zeros(len(kv_lens), max(nblk), dtype=torch.int32)
    n = 0
    for b, c in enumerate(nblk):
        bt[b, :c] = torch.arange(n, n + c, dtype=torch.int32)
        n += c
    cu = [0]
    for ql in q_lens:
        cu.append(cu[-1] + ql)
    T = cu[-1]
    q = (torch.randn(T, h, d, device=DEV) * 0.3).to(torch.bfloat16)
    return q, cache, bt, cu


def case_decode():
    B, ctx, h, hk = args_or([64, 2048, 32, 32])
    q, cache, bt, cu = _attn_setup([1] * B, [ctx] * B, h, hk)
    meta = make_step_input([0] * B, [0] * B, [0] * B, cu, [ctx] * B, bt, num_prefill=0, device=DEV)
    us = timeit(lambda i: cuda.paged_attention(q, cache, meta, 128 ** -0.5))
    by = B * ctx * 2 * hk * 128 * 2
    p = peaks()
    return dict(kernel="paged_decode", B=B, ctx=ctx, h=h, hk=hk, us=round(us, 1), kv_gb=round(by / 1e9, 3),
                gbs=round(by / us / 1e3, 1), frac_of_measured_hbm=round(by / us / 1e3 / p["hbm_gbs"], 3))


def case_prefill():
    T, h, hk = args_or([4096, 32, 32])
    q, cache, bt, cu = _attn_setup([T], [T], h, hk)
    meta = make_step_input([0] * T, [0] * T, [0] * T, cu, [T], bt, num_prefill=1, device=DEV)
    us = timeit(lambda i: cuda.paged_attention(q, cache, meta, 128 ** -0.5), iters=5)
    fl = 4.0 * h * 128 * T * T / 2  # causal
    p = peaks()
    return dict(kernel="paged_prefill", T=T, h=h, hk=hk, us=round(us, 1), tflops=round(fl / us / 1e6, 1),
                frac_of_measured_bf16=round(fl / us / 1e6 / p["bf16_tflops"], 3))


def case_mla():
    from ksanallm_b200.ops import cuda_mla
    B, ctx, h, ql = args_or([64, 4096, 128, 1])
    bs = 64
    nb = (ctx + bs - 1) // bs
    cache = (torch.randn(B * nb + 1, bs, 576, device=DEV) * 0.3).to(torch.bfloat16)
    bt = torch.arange(B * nb, dtype=torch.int32).reshape(B, nb)
    cu = [i * ql for i in range(B + 1)]
    T = B * ql
    q_lat = (torch.randn(T, h, 512, device=DEV) * 0.3).to(torch.bfloat16)
    q_rope = (torch.randn(T, h, 64, device=DEV) * 0.3).to(torch.bfloat16)
    meta = make_step_input([0] * T, [0] * T, [0] * T, cu, [ctx] * B, bt, num_prefill=0, device=DEV)
    us = timeit(lambda i: cuda_mla.mla_paged_attention(q_lat, q_rope, cache, meta, 0.1147))
    by = B * ctx * 576 * 2
    fl = 2.0 * T * h * ctx * (576 + 512)
    p = peaks()
    return dict(kernel="mla_decode", B=B, ctx=ctx, h=h, q_len=ql, us=round(us, 1), kv_gb=round(by / 1e9, 3),
                gbs=round(by / us / 1e3, 1), frac_of_measured_hbm=round(by / us / 1e3 / p["hbm_gbs"], 3),
                tflops=round(fl / us / 1e6, 1), frac_of_measured_bf16=round(fl / us / 1e6 / p["bf16_tflops"], 3))


def case_rmsnorm():
    T, H = args_or([16384, 8192])
    xs = [torch.randn(T, H, device=DEV).to(torch.bfloat16) for _ in range(2)]
    rs = [torch.randn(T, H, device=DEV).to(torch.bfloat16) for _ in range(2)]
    w = torch.ones(H, device=DEV, dtype=torch.bfloat16)
    us = timeit(lambda i: cuda.rms_norm(xs[i % 2], w, 1e-6, rs[i % 2]))
    by = T * H * 2 * 4  # x, residual in, residual out, y
    p = peaks()
    return dict(kernel="rms_norm+residual", T=T, H=H, us=round(us, 1), gbs=round(by / us / 1e3, 1),
                frac_of_measured_hbm=round(by / us / 1e3 / p["hbm_gbs"], 3))


def case_moe():
    T, E, k, H, I = args_or([2048, 32, 8, 2048, 1024])
    x = torch.randn(T, H, device=DEV).to(torch.bfloat16)
    ids, w = ref.moe_route(torch.randn(T, E, device=DEV), k, "softmax", True)
    w1 = (torch.randn(E, 2 * I, H, device=DEV) * 0.05).to(torch.bfloat16)
    w2 = (torch.randn(E, H, I, device=DEV) * 0.05).to(torch.bfloat16)
    us = timeit(lambda i: cuda_moe.moe_experts(x, ids, w, w1, w2, 0), iters=5)
    fl = 2.0 * T * k * (2 * I * H + H * I)
    p = peaks()
    return dict(kernel="moe_experts(pipeline)", T=T, E=E, k=k, H=H, I=I, us=round(us, 1),
                tflops=round(fl / us / 1e6, 1), frac_of_measured_bf16=round(fl / us / 1e6 / p["bf16_tflops"], 3))


def _window_setup(q_lens, kv_lens, h, hk, d, dv, window, prefill, keep=0, shared=0, cap=0):
    q, _, bt, cu = _attn_setup(q_lens, kv_lens, h, 1)
    q = (torch.randn(cu[-1], h, d, device=DEV) * 0.3).to(torch.bfloat16)
    cache = (torch.randn(int(bt.max()) + 2, hk * 16 * (d + (0 if shared else dv)), device=DEV) * 0.3).to(torch.bfloat16)
    T = cu[-1]
    meta = make_step_input([0] * T, [0] * T, [0] * T, cu, kv_lens, bt, num_prefill=prefill, device=DEV)
    bias = None if shared or cap else torch.randn(h, max(kv_lens) if keep else window or max(kv_lens), device=DEV)
    out = torch.empty(T, h * dv, dtype=torch.bfloat16, device=DEV)
    gate = torch.randn(T, (h + 7) // 8 * 8, device=DEV).to(torch.bfloat16)[:, :h] if cap else None
    return lambda i: cuda_mixer.window_attention(q, cache, meta, 16, hk, dv, d ** -0.5, window, bias, 1.0, out, keep,
                                                 float(cap), bool(cap), gate)


def case_window_prefill():
    T, h, hk, d, dv, window, keep, shared, cap = args_or([8192, 32, 8, 128, 128, 1024, 0, 0, 0])
    us = timeit(_window_setup([T], [T], h, hk, d, dv, window, 1, keep, shared, cap), iters=5)
    w = min(window or T, T)
    pairs = w * (w + 1) / 2 + (T - w) * w
    fl = 2.0 * h * (d + dv) * pairs
    p = peaks()
    return dict(kernel="window_prefill", T=T, h=h, hk=hk, d=d, dv=dv, window=window, keep=keep, shared=shared, cap=cap, us=round(us, 1),
                tflops=round(fl / us / 1e6, 1), frac_of_measured_bf16=round(fl / us / 1e6 / p["bf16_tflops"], 3))


def case_window_decode():
    B, ctx, h, hk, d, dv, window, keep, shared, cap = args_or([128, 4096, 32, 8, 128, 128, 1024, 0, 0, 0])
    us = timeit(_window_setup([1] * B, [ctx] * B, h, hk, d, dv, window, 0, keep, shared, cap))
    by = B * min(window + keep if window else ctx, ctx) * hk * (d + (0 if shared else dv)) * 2
    p = peaks()
    return dict(kernel="window_decode", B=B, ctx=ctx, h=h, hk=hk, d=d, dv=dv, window=window, keep=keep, shared=shared, cap=cap, us=round(us, 1),
                kv_gb=round(by / 1e9, 3), gbs=round(by / us / 1e3, 1),
                frac_of_measured_hbm=round(by / us / 1e3 / p["hbm_gbs"], 3))


def _linear_setup(lens, q_lens, h, d, dv, rotary, prefill, copies=1):
    B, T = len(lens), sum(q_lens)
    cu = [0]
    for q in q_lens:
        cu.append(cu[-1] + q)
    pos = [n - q + i for n, q in zip(lens, q_lens) for i in range(q)]
    meta = make_step_input([0] * T, pos, [0] * T, cu, lens, torch.zeros(B, 1), num_prefill=prefill, device=DEV,
                           state_slots=list(range(B)))
    width = h * (2 * d + dv)
    xs = [(torch.randn(T, width, device=DEV) * 0.3).to(torch.bfloat16) for _ in range(copies)]
    states = [torch.zeros(B, h, d, dv, device=DEV) for _ in range(copies)]
    decay = torch.full((h,), 0.99, device=DEV)
    table = ref.rotary_table(d, 1e4, max(lens), DEV) if rotary else None

    def run(i):
        x = xs[i % copies]
        q, k, v = x[:, :h * d], x[:, h * d:2 * h * d], x[:, 2 * h * d:]
        cuda_mixer.linear_attention(q.unflatten(1, (h, d)), k.unflatten(1, (h, d)), v.unflatten(1, (h, dv)),
                                    states[i % copies], meta, decay, "none" if rotary else "silu", table, 0.1)
    return run


def case_linear_prefill():
    T, h, d, dv, rotary = args_or([8192, 32, 128, 128, 1])
    us = timeit(_linear_setup([T], [T], h, d, dv, rotary, 1, 2), iters=5)
    by = T * h * (2 * d + 2 * dv) * 2
    fl = T * h * (2.0 * d * dv * 2 + 128 * (d + dv))  # state update and read-out + the causal half of a chunk of 128
    p = peaks()
    floor = max(by / p["hbm_gbs"] / 1e3, fl / p["bf16_tflops"] / 1e6)
    return dict(kernel="linear_chunked", T=T, h=h, d=d, dv=dv, rotary=rotary, us=round(us, 1),
                roofline_us=round(floor, 1), frac_of_roofline=round(floor / us, 3))


def case_linear_decode():
    B, h, d, dv, rotary = args_or([128, 32, 128, 128, 1])
    us = timeit(_linear_setup([100] * B, [1] * B, h, d, dv, rotary, 0, 2))
    by = 2 * B * h * d * dv * 4
    p = peaks()
    return dict(kernel="linear_recurrent", B=B, h=h, d=d, dv=dv, rotary=rotary, us=round(us, 1),
                state_gb=round(by / 2e9, 3), gbs=round(by / us / 1e3, 1),
                frac_of_measured_hbm=round(by / us / 1e3 / p["hbm_gbs"], 3))


def _latent_setup(q_lens, kv_lens, h, dim, rot, vdim, rank, prefill):
    """The operator's inputs, and what its kernels get in between."""
    from ksanallm_b200.models.mixers import LatentWeights
    _, _, bt, cu = _attn_setup(q_lens, kv_lens, 1, 1)
    T = cu[-1]
    bf = lambda *s: (torch.randn(*s, device=DEV) * 0.3).to(torch.bfloat16)  # noqa: E731
    cache = bf(int(bt.max()) + 2, 16 * (rank + rot))
    pos = [n - q + i for n, q in zip(kv_lens, q_lens) for i in range(q)]
    slots = [int(bt[b, p // 16]) * 16 + p % 16 for b, (n, q) in enumerate(zip(kv_lens, q_lens)) for p in range(n - q, n)]
    meta = make_step_input([0] * T, pos, slots, cu, kv_lens, bt, num_prefill=prefill, device=DEV)
    x = bf(T, (h * (dim + rot) + rank + rot + h + 7) // 8 * 8)
    nq, na = h * (dim + rot), rank + rot
    w = LatentWeights(bf(h, dim, rank), bf(h, vdim, rank))
    out, norm, table = bf(T, h * vdim), torch.ones(rank, device=DEV), ref.rotary_table(rot, 1e4, max(kv_lens), DEV)
    return x[:, :nq].unflatten(1, (h, dim + rot)), x[:, nq:nq + na], x[:, nq + na:nq + na + h], w, cache, meta, out, norm, table


def case_latent_prefill():
    """The attention kernel alone, and the whole operator: append, gather, keys and values per head, attention."""
    T, h, dim, rot, vdim, rank = args_or([8192, 32, 128, 64, 128, 512])
    q, a, gate, w, cache, meta, out, norm, table = _latent_setup([T], [T], h, dim, rot, vdim, rank, 1)
    lat = (torch.randn(T, rank + rot, device=DEV) * 0.3).to(torch.bfloat16)
    kv = cuda.gemm_bf16(lat[:, :rank], w.expand)
    st = torch.cuda.current_stream().cuda_stream

    def kernel(i):
        assert cuda.lib().ksana_latent_prefill(
            q.data_ptr(), q.stride(0), T, kv.data_ptr(), kv.stride(0), lat.data_ptr() + 2 * rank, rank + rot, T,
            meta.cu_q.data_ptr(), meta.kv_lens.data_ptr(), h, dim, rot, vdim, 0.07, gate.data_ptr(), gate.stride(0),
            out.data_ptr(), out.stride(0), 0, 1, T, st) == 0
    us = timeit(kernel, iters=5)
    op = timeit(lambda i: cuda_latent.latent_attention(q, a, norm, 1e-6, table, cache, meta, 16, w, 0.07, gate, out), iters=5)
    gather = timeit(lambda i: cuda.lib().ksana_latent_gather(cache.data_ptr(), meta.block_tables.data_ptr(), meta.max_blocks,
                                                             meta.kv_lens.data_ptr(), 0, 1, T, 16, rank + rot, lat.data_ptr(), st))
    fl, p = 2.0 * h * (dim + rot + vdim) * T * (T + 1) / 2, peaks()
    return dict(kernel="latent_prefill", T=T, h=h, dim=dim, rot=rot, vdim=vdim, rank=rank, us=round(us, 1),
                tflops=round(fl / us / 1e6, 1), frac_of_measured_bf16=round(fl / us / 1e6 / p["bf16_tflops"], 3),
                operator_us=round(op, 1), gather_us=round(gather, 1),
                gather_frac_of_measured_hbm=round(T * (rank + rot) * 4 / gather / 1e3 / p["hbm_gbs"], 3))


def case_latent_decode():
    B, ctx, h, dim, rot, vdim, rank = args_or([64, 4096, 32, 128, 64, 128, 512])
    q, a, gate, w, cache, meta, out, norm, table = _latent_setup([1] * B, [ctx] * B, h, dim, rot, vdim, rank, 0)
    qc = (torch.randn(B, h * (rank + rot), device=DEV) * 0.3).to(torch.bfloat16)
    o = torch.empty(B, h * rank, dtype=torch.bfloat16, device=DEV)
    st = torch.cuda.current_stream().cuda_stream

    def kernel(i):
        assert cuda.lib().ksana_latent_decode(
            qc.data_ptr(), qc.stride(0), B, cache.data_ptr(), cache.shape[0], meta.block_tables.data_ptr(), meta.max_blocks,
            meta.cu_q.data_ptr(), meta.kv_lens.data_ptr(), h, rank, rot, 16, 0.07, gate.data_ptr(), gate.stride(0),
            o.data_ptr(), o.stride(0), 0, B, 1, ctx, st) == 0
    us = timeit(kernel)
    op = timeit(lambda i: cuda_latent.latent_attention(q, a, norm, 1e-6, table, cache, meta, 16, w, 0.07, gate, out))
    by, p = B * ctx * (rank + rot) * 2, peaks()
    return dict(kernel="latent_decode", B=B, ctx=ctx, h=h, rank=rank, rot=rot, us=round(us, 1), kv_gb=round(by / 1e9, 3),
                gbs=round(by / us / 1e3, 1), frac_of_measured_hbm=round(by / us / 1e3 / p["hbm_gbs"], 3),
                tflops=round(2.0 * B * h * ctx * (2 * rank + rot) / us / 1e6, 1), operator_us=round(op, 1))


def _recurrence_setup(lens, q_lens, C, blocks, K, prefill, copies=2):
    from ksanallm_b200.models.mixers import RecurrenceWeights
    B, T = len(lens), sum(q_lens)
    cu = [0]
    for q in q_lens:
        cu.append(cu[-1] + q)
    meta = make_step_input([0] * T, [0] * T, [0] * T, cu, lens, torch.zeros(B, 1), num_prefill=prefill, device=DEV,
                           state_slots=list(range(B)))
    s, r = C // blocks, lambda *a: torch.randn(*a, device=DEV) * 0.3  # noqa: E731
    w = RecurrenceWeights({"p.conv": r(C, K), "p.conv_b": r(C), "p.gates": r(2, blocks, s, s).to(torch.bfloat16),
                           "p.gates_b": r(2, C), "p.lam": r(C) - 3}, "p", 8.0)
    xs = [r(T, 2 * C).to(torch.bfloat16) for _ in range(copies)]
    states = [torch.zeros(B, 1, K, C, device=DEV) for _ in range(copies)]
    out = torch.empty(T, C, dtype=torch.bfloat16, device=DEV)
    return lambda i: cuda_recurrence.gated_recurrence(xs[i % copies][:, :C], xs[i % copies][:, C:], states[i % copies], meta, w, out)


def case_recurrence_prefill():
    T, C, blocks, K, n = args_or([8192, 4096, 32, 4, 1])
    us = timeit(_recurrence_setup([T // n] * n, [T // n] * n, C, blocks, K, n), iters=5)
    by, fl, p = T * C * 6, 4.0 * T * C * (C // blocks), peaks()
    floor = max(by / p["hbm_gbs"] / 1e3, fl / p["bf16_tflops"] / 1e6)
    return dict(kernel="recurrence_prompts", T=T, C=C, blocks=blocks, K=K, sequences=n, us=round(us, 1),
                roofline_us=round(floor, 1), frac_of_roofline=round(floor / us, 3))


def case_recurrence_decode():
    B, C, blocks, K = args_or([128, 4096, 32, 4])
    # enough layers' states and inputs that L2 holds none of them
    us = timeit_graph(_recurrence_setup([100] * B, [1] * B, C, blocks, K, 0, 24))
    by, p = B * C * (8 * K + 6) + 4 * C * (C // blocks), peaks()
    return dict(kernel="recurrence_step", B=B, C=C, blocks=blocks, K=K, us=round(us, 1), mb=round(by / 1e6, 1),
                gbs=round(by / us / 1e3, 1), frac_of_measured_hbm=round(by / us / 1e3 / p["hbm_gbs"], 3))


def case_ladusun_rows():
    """Row-wise kernels of hyper-connected streams, latent attention and clamped experts."""
    T, H, S, h, hk, d, rank, rot = args_or([8192, 4096, 4, 32, 8, 128, 512, 64])
    bf = lambda *s: torch.randn(*s, device=DEV).to(torch.bfloat16)  # noqa: E731
    f32 = lambda *s: torch.randn(*s, device=DEV)  # noqa: E731
    p, out, st = peaks(), {}, torch.cuda.current_stream().cuda_stream

    def add(name, us, by):
        out[name] = dict(us=round(us, 1), gbs=round(by / us / 1e3, 1), frac_of_measured_hbm=round(by / us / 1e3 / p["hbm_gbs"], 3))
    xs, streams, w = [bf(T, H) for _ in range(2)], [f32(T, S, H) for _ in range(2)], bf(H)
    mix, ow, iw, ls = torch.eye(S, device=DEV), f32(S), f32(S) / S, torch.ones(H, device=DEV)
    add("hyper_norm", timeit(lambda i: cuda_mixer.hyper_norm(xs[i % 2], ls, None, streams[i % 2], mix, ow, streams[i % 2], iw, w,
                                                             1e-6, torch.bfloat16)), T * H * (8 * S + 4))
    k = 2
    y2, pos, wts = bf(T * k, H), torch.randperm(T * k, dtype=torch.int32, device=DEV), torch.rand(T, k, device=DEV)
    add("hyper_norm_routed", timeit(lambda i: cuda_mixer.hyper_norm(None, ls, (y2, pos, wts), streams[i % 2], mix, ow, streams[i % 2],
                                                                    iw, w, 1e-6, torch.bfloat16)), T * H * (8 * S + 2 + 2 * k))
    add("rms_norm", timeit(lambda i: cuda.rms_norm(xs[i % 2], w, 1e-6, xs[1 - i % 2])), T * H * 8)
    us = [bf(T, 6 * H) for _ in range(2)]
    add("clamped_gate_mul", timeit(lambda i: cuda_mixer.clamped_gate_mul(us[i % 2], 7.0, 1.702)), T * H * 18)
    add("silu_mul", timeit(lambda i: cuda.silu_and_mul(us[i % 2])), T * H * 18)
    add("relu2", timeit(lambda i: cuda_mixer.relu2(us[i % 2])), T * H * 24)
    slots, table = torch.arange(T, dtype=torch.int32, device=DEV), torch.randn(T, d, device=DEV)
    cache = torch.zeros((T + 15) // 16, hk * 16 * 2 * d, dtype=torch.bfloat16, device=DEV)
    qkv = [bf(T, (h + 2 * hk) * d) for _ in range(3)]

    def parts(x):
        return x[:, :h * d].unflatten(1, (h, d)), x[:, h * d:(h + hk) * d].unflatten(1, (hk, d)), x[:, (h + hk) * d:].unflatten(1, (hk, d))
    by = T * d * 2 * (2 * h + 4 * hk)
    add("rotate_cache", timeit(lambda i: cuda_mixer.qk_norm_cache(*parts(qkv[i % 3]), slots, cache, 16, None, None, 1e-6, slots, table)), by)
    add("rope_cache", timeit(lambda i: cuda.rope_qknorm_cache(*parts(qkv[i % 3]), slots, table, slots, cache.view(-1, 2, hk, 16, d))), by)
    lat, lt = torch.zeros((T + 15) // 16, 16 * (rank + rot), dtype=torch.bfloat16, device=DEV), torch.randn(T, rot, device=DEV)
    ql = [bf(T, h * (d + rot) + rank + rot) for _ in range(2)]
    nq, nw = h * (d + rot), torch.ones(rank, device=DEV)

    def append(i):
        x = ql[i % 2]
        assert cuda.lib().ksana_latent_append(x.data_ptr(), x.stride(0), d, None, 0, x.data_ptr() + 2 * nq, x.stride(0), nw.data_ptr(),
                                              1e-6, slots.data_ptr(), lt.data_ptr(), slots.data_ptr(), lat.data_ptr(), T, h, rank, rot, 1, st) == 0
    add("latent_append", timeit(append), T * 4 * (h * rot + rank + rot))
    q, qc = bf(T, h, d + rot), bf(T, h, rank + rot)
    kr, lt2 = bf(T, rot), bf(T, rank)

    def mla_append(i):
        assert cuda.lib().ksana_mla_rope_append(q.data_ptr(), q.stride(0), q.stride(1), d, qc.data_ptr(), kr.data_ptr(), rot, lt2.data_ptr(),
                                                rank, slots.data_ptr(), lt.data_ptr(), slots.data_ptr(), lat.data_ptr(), rank + rot, T, h, rank, rot,
                                                1, st) == 0
    add("mla_rope_append", timeit(mla_append), T * 4 * (h * rot + rank + rot))
    z = torch.randn(T, 16, device=DEV)
    add("moe_topk_groups", timeit(lambda i: cuda_moe.moe_topk(z, 16, 2, None, 4, 2)), T * (16 + 4) * 4)
    add("moe_route", timeit(lambda i: cuda_moe.moe_route(z, 2, "softmax", True, 4, 2)), T * (16 + 4) * 4)
    return dict(kernel="ladusun_rows", T=T, H=H, streams=S, **out)


def _talking_setup(q_lens, kv_lens, h, hk, d, dv, prefill):
    _, _, bt, cu = _attn_setup(q_lens, kv_lens, 1, 1)
    T = cu[-1]
    bf = lambda *s: torch.randn(*s, device=DEV).to(torch.bfloat16)  # noqa: E731
    cache = bf(int(bt.max()) + 2, 16 * hk * (d + dv))
    pos = [n - q + i for n, q in zip(kv_lens, q_lens) for i in range(q)]
    meta = make_step_input([0] * T, pos, [0] * T, cu, kv_lens, bt, num_prefill=prefill, device=DEV)
    x, out = bf(T, h * (d + dv)), bf(T, h * dv)
    sink, talk = torch.randn(h, device=DEV), (torch.eye(h, device=DEV) + 0.3 * torch.randn(h, h, device=DEV)).bfloat16().float()
    return lambda i: cuda_talking.talking_attention(x[:, :h * d].unflatten(1, (h, d)), cache, meta, 16, hk, dv, d ** -0.5, sink,
                                                    talk, 1.0, out, x[:, h * d:])


def case_talking_prefill():
    T, h, hk, d, dv = args_or([8192, 32, 8, 128, 128])
    us = timeit(_talking_setup([T], [T], h, hk, d, dv, 1), iters=5)
    pairs = T * (T + 1) / 2
    fl, mix = 2.0 * h * (d + dv) * pairs, 2.0 * h * h * pairs
    p = peaks()
    return dict(kernel="talking_prefill", T=T, h=h, hk=hk, d=d, dv=dv, us=round(us, 1), tflops=round((fl + mix) / us / 1e6, 1),
                frac_of_measured_bf16=round((fl + mix) / us / 1e6 / p["bf16_tflops"], 3),
                frac_without_the_mix=round(fl / us / 1e6 / p["bf16_tflops"], 3))


def case_talking_decode():
    B, ctx, h, hk, d, dv = args_or([128, 1024, 32, 8, 128, 128])
    us = timeit(_talking_setup([1] * B, [ctx] * B, h, hk, d, dv, 0))
    by, p = B * ctx * hk * (d + dv) * 2, peaks()
    return dict(kernel="talking_decode", B=B, ctx=ctx, h=h, hk=hk, d=d, dv=dv, us=round(us, 1), kv_gb=round(by / 1e9, 3),
                gbs=round(by / us / 1e3, 1), frac_of_measured_hbm=round(by / us / 1e3 / p["hbm_gbs"], 3))


def _timemix_setup(lens, q_lens, h, d, prefill, copies=2):
    B, T, n = len(lens), sum(q_lens), h * d
    cu = [0]
    for q in q_lens:
        cu.append(cu[-1] + q)
    meta = make_step_input([0] * T, [0] * T, [0] * T, cu, lens, torch.zeros(B, 1), num_prefill=prefill, device=DEV,
                           state_slots=list(range(B)))
    xs = [(torch.randn(3, T, n, device=DEV) * 0.3).to(torch.bfloat16) for _ in range(copies)]
    zs = [torch.randn(T, n, device=DEV) for _ in range(copies)]
    states = [torch.zeros(B, 1, 1, h * d * d + n, device=DEV) for _ in range(copies)]
    w0, u = torch.randn(n, device=DEV) - 3, torch.randn(h, d, device=DEV)
    return lambda i: cuda_timemix.time_mix(xs[i % copies][0], xs[i % copies][1], xs[i % copies][2], zs[i % copies], w0, u,
                                           states[i % copies], meta)


def case_timemix_prefill():
    T, h, d, n = args_or([8192, 64, 64, 1])
    us = timeit(_timemix_setup([T // n] * n, [T // n] * n, h, d, n), iters=5)
    by = T * h * d * (4 * 2 + 4)  # r, k, v, o in 16 bits and the decay's exponent in 32
    fl = T * h * (2.0 * d * d * 2 + 64 * 2 * d)  # state update and read-out + the causal half of a chunk of 64
    p = peaks()
    floor = max(by / p["hbm_gbs"] / 1e3, fl / p["bf16_tflops"] / 1e6)
    return dict(kernel="timemix_prefill", T=T, h=h, d=d, sequences=n, us=round(us, 1), roofline_us=round(floor, 1),
                frac_of_roofline=round(floor / us, 3))


def case_timemix_decode():
    B, h, d = args_or([128, 64, 64])
    us = timeit(_timemix_setup([100] * B, [1] * B, h, d, 0))
    by, p = 2 * B * h * d * d * 4, peaks()
    return dict(kernel="timemix_decode", B=B, h=h, d=d, us=round(us, 1), state_gb=round(by / 2e9, 3), gbs=round(by / us / 1e3, 1),
                frac_of_measured_hbm=round(by / us / 1e3 / p["hbm_gbs"], 3))


def case_vibunex_rows():
    """Row-wise kernels of gated residuals, time mixing and weight-mixing attention."""
    T, H, h, hk, d = args_or([8192, 4096, 32, 8, 128])
    bf = lambda *s: torch.randn(*s, device=DEV).to(torch.bfloat16)  # noqa: E731
    p, out = peaks(), {}

    def add(name, us, by):
        out[name] = dict(us=round(us, 1), gbs=round(by / us / 1e3, 1), frac_of_measured_hbm=round(by / us / 1e3 / p["hbm_gbs"], 3))
    xs, r32, w, k = [bf(T, 4 * H) for _ in range(2)], [torch.randn(T, H, device=DEV) for _ in range(2)], bf(H), 2
    y2, pos, wts = bf(T * k, H), torch.randperm(T * k, dtype=torch.int32, device=DEV), torch.rand(T, k, device=DEV)
    z = torch.randn(T, 24, device=DEV)

    def norm(i, routed):
        x = xs[i % 2]
        cuda_mixer.gated_stream_norm(x[:, :H], x[:, H:2 * H], (y2, pos, wts) if routed else None, x[:, 2 * H:3 * H], z[:, 16],
                                     x[:, 3 * H:], 0.5, r32[i % 2], r32[i % 2], [w, w], 1e-6, torch.bfloat16)
    add("gated_stream_norm", timeit(lambda i: norm(i, False)), T * H * 20)
    add("gated_stream_norm_routed", timeit(lambda i: norm(i, True)), T * H * (20 + 2 * k))
    r16 = [bf(T, H) for _ in range(2)]
    add("rms_norm", timeit(lambda i: cuda.rms_norm(r16[i % 2], w, 1e-6, r16[1 - i % 2])), T * H * 8)
    meta = make_step_input([0] * T, [0] * T, [0] * T, [0, T], [T], torch.zeros(1, 1), num_prefill=1, device=DEV, state_slots=[0])
    mu, state = torch.rand(5, H, device=DEV), torch.zeros(1, 1, 1, H, device=DEV)
    add("token_mix", timeit(lambda i: cuda_timemix.token_mix(r16[i % 2], mu, state, meta)), T * H * 12)
    o, g, y, wf = bf(T, H // 64, 64), [bf(T, H) for _ in range(2)], bf(T, H), torch.ones(H, device=DEV)
    add("gated_head_norm_weight", timeit(lambda i: cuda_mixer.gated_norm(o, g[i % 2], wf, 1e-6, "silu", 1.0, y, True)), T * H * 6)
    add("gated_head_norm", timeit(lambda i: cuda_mixer.gated_norm(o, g[i % 2], None, 1e-6, "silu", 1.0, y)), T * H * 6)
    slots, table = torch.arange(T, dtype=torch.int32, device=DEV), torch.randn(T, d // 2, device=DEV)
    cache = torch.zeros((T + 15) // 16, hk * 16 * 2 * d, dtype=torch.bfloat16, device=DEV)
    qkv = [bf(T, (h + 2 * hk) * d) for _ in range(3)]
    wq, wk, wb = torch.ones(h * d, device=DEV), torch.ones(hk * d, device=DEV), torch.ones(d, device=DEV, dtype=torch.bfloat16)

    def parts(x):
        return x[:, :h * d].unflatten(1, (h, d)), x[:, h * d:(h + hk) * d].unflatten(1, (hk, d)), x[:, (h + hk) * d:].unflatten(1, (hk, d))
    by = T * d * 2 * (2 * h + 4 * hk)
    add("qk_row_norm_cache", timeit(lambda i: cuda_mixer.qk_norm_cache(*parts(qkv[i % 3]), slots, cache, 16, wq, wk, 1e-6, slots, table,
                                                                       True, True)), by)
    full = torch.randn(T, d, device=DEV)
    add("rope_cache", timeit(lambda i: cuda.rope_qknorm_cache(*parts(qkv[i % 3]), slots, full, slots, cache.view(-1, 2, hk, 16, d), wb, wb,
                                                              1e-6)), by)
    a32 = torch.randn(T, 64, device=DEV)
    add("tanh_parts", timeit(lambda i: cuda_timemix.tanh_parts(a32, torch.bfloat16)), T * 64 * 8)
    add("moe_topk_sigmoid", timeit(lambda i: cuda_moe.moe_topk(z, 16, 2, None, 1, 1, "sigmoid", 1.5)), T * (16 + 4) * 4)
    add("moe_route", timeit(lambda i: cuda_moe.moe_route(z, 2, "softmax", True)), T * (16 + 4) * 4)
    us = [bf(T, 2 * H) for _ in range(2)]
    add("relu2_strided", timeit(lambda i: cuda_mixer.relu2(us[i % 2][:, H:])), T * H * 4)
    return dict(kernel="vibunex_rows", T=T, H=H, h=h, hk=hk, d=d, **out)


def case_mixer_rows():
    """The row-wise kernels, each beside its counterpart of the dense models."""
    T, H, h, hk, d = args_or([8192, 4096, 32, 8, 128])
    bf = lambda *s: torch.randn(*s, device=DEV).to(torch.bfloat16)  # noqa: E731
    p, out = peaks(), {}

    def add(name, us, by):
        out[name] = dict(us=round(us, 1), gbs=round(by / us / 1e3, 1), frac_of_measured_hbm=round(by / us / 1e3 / p["hbm_gbs"], 3))

    xs, w = [bf(T, H) for _ in range(3)], torch.ones(H, device=DEV, dtype=torch.bfloat16)
    r32, r16 = [torch.randn(T, H, device=DEV) for _ in range(3)], [bf(T, H) for _ in range(3)]
    add("layer_norm", timeit(lambda i: cuda_mixer.layer_norm(xs[i % 3], w, None, 1e-6, r32[i % 3], torch.bfloat16)), T * H * 12)
    add("rms_norm", timeit(lambda i: cuda.rms_norm(xs[i % 3], w, 1e-6, r16[i % 3])), T * H * 8)
    us = [bf(T, 6 * H) for _ in range(2)]
    add("gelu_mul", timeit(lambda i: cuda_mixer.gelu_and_mul(us[i % 2])), T * H * 18)
    add("silu_mul", timeit(lambda i: cuda.silu_and_mul(us[i % 2])), T * H * 18)
    o, g, y = bf(T, h, d), bf(T, 2 * h * d), torch.empty(T, h * d, device=DEV, dtype=torch.bfloat16)
    gs = [g, g.clone()]
    add("gated_head_norm", timeit(lambda i: cuda_mixer.gated_norm(o, gs[i % 2][:, :h * d], None, 1e-6, "silu", 1.1, y)), T * h * d * 6)
    wn = torch.ones(h * d, device=DEV)
    add("gated_row_norm", timeit(lambda i: cuda_mixer.gated_norm(o, gs[i % 2][:, :h * d], wn, 1e-6, "sigmoid", 1.0, y)), T * h * d * 6)
    slots = torch.arange(T, dtype=torch.int32, device=DEV)
    cache = torch.zeros((T + 15) // 16, 2, hk, 16, d, dtype=torch.bfloat16, device=DEV)
    qkv = [bf(T, (h + 2 * hk) * d) for _ in range(3)]
    wf, wb = torch.ones(d, device=DEV), torch.ones(d, device=DEV, dtype=torch.bfloat16)

    def parts(x):
        return x[:, :h * d].unflatten(1, (h, d)), x[:, h * d:(h + hk) * d].unflatten(1, (hk, d)), x[:, (h + hk) * d:].unflatten(1, (hk, d))
    by = T * d * 2 * (2 * h + 4 * hk)
    add("qk_norm_cache", timeit(lambda i: cuda_mixer.qk_norm_cache(*parts(qkv[i % 3]), slots, cache.view(cache.shape[0], -1), 16, wf, wf, 1e-6)), by)
    # cache append beside a plain GELU feed-forward, routed norm, router and sort
    keys = torch.zeros((T + 15) // 16, hk * 16 * d, dtype=torch.bfloat16, device=DEV)
    wide = [bf(T, (h + hk) * d + 4 * H) for _ in range(2)]
    mixed = torch.empty(T, h * d + 4 * H, dtype=torch.bfloat16, device=DEV)
    add("append_act", timeit(lambda i: cuda_mixer.append_act(
        wide[i % 2][:, h * d:(h + hk) * d].unflatten(1, (hk, d)), wide[i % 2][:, (h + hk) * d:], slots, keys, 16,
        mixed[:, h * d:])), T * (hk * d + 4 * H) * 4)
    add("stream_norm", timeit(lambda i: cuda_mixer.stream_norm(xs[i % 3], w, 1e-6, False, r32[i % 3], r32[i % 3], torch.bfloat16)), T * H * 12)
    k, E = 2, 16
    y2, pos = bf(T * k, H), torch.randperm(T * k, dtype=torch.int32, device=DEV)
    z = torch.randn(T, E, device=DEV)
    ids, wts = cuda_moe.moe_topk(z, E, k)
    add("stream_norm_routed", timeit(lambda i: cuda_mixer.stream_norm(xs[i % 3], w, 1e-6, False, r32[i % 3], r32[i % 3], torch.bfloat16,
                                                                      routed=(y2, pos, wts))), T * H * (12 + 2 * k))
    add("stream_norm_pass", timeit(lambda i: cuda_mixer.stream_norm(xs[i % 3], w, 1e-6, False, r32[i % 3], r32[i % 3], torch.bfloat16,
                                                                    add_rows=r32[(i + 1) % 3], add_vec=r32[0][0])), T * H * 16)
    comb = bf(T, H)
    add("moe_combine", timeit(lambda i: cuda.lib().ksana_moe_combine(y2.data_ptr(), pos.data_ptr(), wts.data_ptr(), T, k, H, comb.data_ptr(),
                                                                      torch.cuda.current_stream().cuda_stream)), T * H * (2 + 2 * k))
    add("moe_topk", timeit(lambda i: cuda_moe.moe_topk(z, E, k)), T * (E + 2 * k) * 4)
    add("moe_route", timeit(lambda i: cuda_moe.moe_route(z, k, "softmax", True)), T * (E + 2 * k) * 4)
    offs, src = torch.empty(E + 1, dtype=torch.int32, device=DEV), torch.empty(T * k, dtype=torch.int32, device=DEV)
    add("moe_sort", timeit(lambda i: cuda.lib().ksana_moe_sort(ids.data_ptr(), T * k, 0, E, offs.data_ptr(), pos.data_ptr(), src.data_ptr(),
                                                               torch.cuda.current_stream().cuda_stream)), T * k * 12)
    table = torch.randn(T, d, device=DEV)
    add("rope_cache", timeit(lambda i: cuda.rope_qknorm_cache(*parts(qkv[i % 3]), slots, table, slots, cache, wb, wb, 1e-6)), by)
    return dict(kernel="mixer_rows", T=T, H=H, h=h, hk=hk, d=d, **out)


CASES = dict(gemm=case_gemm, gemm_fp8=case_gemm_fp8, gemm_int4=case_gemm_int4, decode=case_decode, prefill=case_prefill, mla=case_mla, rmsnorm=case_rmsnorm,
             moe=case_moe, window_prefill=case_window_prefill, window_decode=case_window_decode,
             linear_prefill=case_linear_prefill, linear_decode=case_linear_decode, mixer_rows=case_mixer_rows,
             latent_prefill=case_latent_prefill, latent_decode=case_latent_decode, recurrence_prefill=case_recurrence_prefill,
             recurrence_decode=case_recurrence_decode, ladusun_rows=case_ladusun_rows, talking_prefill=case_talking_prefill,
             talking_decode=case_talking_decode, timemix_prefill=case_timemix_prefill, timemix_decode=case_timemix_decode,
             vibunex_rows=case_vibunex_rows)

if __name__ == "__main__":
    which = sys.argv[1] if len(sys.argv) > 1 else "all"
    names = list(CASES) if which == "all" else [which]
    if which == "all":
        sys.argv = sys.argv[:2]
    for n in names:
        print(json.dumps(CASES[n]()))
    print(json.dumps({"kernel_status_word": cuda.read_error()}))
