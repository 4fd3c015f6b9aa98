"""Attention over a window whose edges show: one key per probed query scores far above all others, and sits just inside
or just outside of what the query sees."""
import torch

import molopel_oracle as M
from ksanallm_b200.engine.step_input import make_step_input

BS = 16


def check_window(dtype, device, window, n=180):
    from ksanallm_b200 import ops
    h, hk, d, dv = 2, 1, 64, 64
    for back in sorted({max(window - 1, 0), window, window + 1, 0}):
        g = torch.Generator().manual_seed(window * 7 + back)
        q = torch.randn(n, h, d, generator=g).to(dtype).float()
        k = (0.05 * torch.randn(n, hk, d, generator=g)).to(dtype).float()
        v = torch.randn(n, hk, dv, generator=g).to(dtype).float()
        probes = list(range(max(back, 1) + 3, n, 23)) + [n - 1]
        for p in probes:
            q[p, 1] = q[p, 0]
            k[p - back, 0] = q[p, 0]  # score |q|^2 / 8 = 8 against about 0
        k = k.to(dtype).float()
        rel = torch.randn(8, h, generator=g).to(dtype).float()
        want = M.windowed_attention(q.double(), k.double(), v.double(), 0.125, window, rel.double(), 30)
        wrong = M.windowed_attention(q.double(), k.double(), v.double(), 0.125,
                                     window + 1 if back >= window else max(window - 1, 1), rel.double(), 30)
        if back in (window - 1, window) and window > 1:
            assert (want - wrong)[probes].abs().max() > 0.5  # a window that is one token off shows
        from ksanallm_b200.ops import reference as ref
        bias = ref.distance_bias(rel.to(device), 30, window)
        for cuts in ([n], [n - 40] + [1] * 40, [2, 100, 16, 17, n - 135]):
            pages = list(range((n + BS - 1) // BS))[::-1]
            table = torch.tensor([[p + 1 for p in pages]])
            cache = torch.zeros(len(pages) + 1, hk * BS * (d + dv), dtype=dtype, device=device)
            done, rows = 0, []
            for c in cuts:
                slots = [int(table[0, p // BS]) * BS + p % BS for p in range(done, done + c)]
                meta = make_step_input([0] * c, list(range(done, done + c)), slots, [0, c], [done + c], table,
                                       num_prefill=0 if c == 1 and done else 1, device=device)
                part = slice(done, done + c)
                qq, kk, vv = (x[part].to(dtype).to(device).contiguous() for x in (q, k, v))
                ops.qk_norm_cache(qq, kk, vv, meta.slot_mapping, cache, BS, None, None, 1e-6)
                out = torch.empty(c, h * dv, dtype=dtype, device=device)
                ops.window_attention(qq, cache, meta, BS, hk, dv, 0.125, window, bias, 1.0, out)
                rows.append(out.double().cpu())
                done += c
            err = (torch.cat(rows) - want.flatten(1)).abs().max()
            assert err < (2e-5 if dtype == torch.float32 else 2e-2), (window, back, cuts[:3], err)
