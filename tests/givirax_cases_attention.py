"""Attention over a window and the first tokens, values = keys, with edges that show: one key per probed query scores far
above all others and sits just inside or just outside of what the query sees."""
import torch

import givirax_oracle as O
from ksanallm_b200 import ops
from ksanallm_b200.engine.step_input import make_step_input

BS = 16


def feed(q, k, cuts, dtype, device, scale, window, keep):
    """One sequence's q [n, h, d] and k [n, hk, d] through cache append and attention in portions -> [n, h * d]."""
    n, h, d = q.shape
    hk = k.shape[1]
    pages = list(range((n + BS - 1) // BS))[::-1]  # pages in no natural order; page 0 is somebody else's
    table = torch.tensor([[p + 1 for p in pages]])
    cache = torch.zeros(len(pages) + 1, hk * BS * d, dtype=dtype, device=device)
    done, rows = 0, []
    for c in cuts:
        slots = [int(table[0, p // BS]) * BS + p % BS for p in range(done, done + c)]
        meta = make_step_input([0] * c, list(range(done, done + c)), slots, [0, c], [done + c], table,
                               num_prefill=0 if c == 1 and done else 1, device=device)
        qq, kk = (x[done:done + c].to(dtype).to(device).contiguous() for x in (q, k))
        ops.append_act(kk, None, meta.slot_mapping, cache, BS, None)
        out = torch.empty(c, h * d, dtype=dtype, device=device)
        ops.window_attention(qq, cache, meta, BS, hk, d, scale, window, None, 1.0, out, keep)
        rows.append(out.double().cpu())
        done += c
    assert done == n
    return torch.cat(rows)


def portions(n):
    return ([n], [n - 40] + [1] * 40, [2, 100, 16, 17, n - 135], [1, 2] + [1] * 30 + [n - 33])


def check(dtype, device, window, keep, h=3, hk=1, d=64, n=180, edge="all"):
    """Probes at the window's edge and at the end of the kept tokens, against the oracle; an oracle whose window or kept
    range is one token off must differ visibly at the probes."""
    scale = 8.0 / d  # a probe's own score is about 8
    edges = [("window_in", window - 1), ("window_out", window), ("first_in", -1), ("first_out", 0), ("near", 0)]
    for kind, off in edges:
        if edge not in ("all", kind) or kind == "first_in" and keep == 0:
            continue
        g = torch.Generator().manual_seed(window * 7 + keep * 31 + d + len(kind))
        q = torch.randn(n, h, d, generator=g)
        q = (q * d ** 0.5 / q.norm(dim=-1, keepdim=True)).to(dtype).float()
        k = (0.05 * torch.randn(n, hk, d, generator=g)).to(dtype).float()
        if kind.startswith("first"):
            target = keep + off
            probes = [i for i in range(target + window, n, 29)] + ([n - 1] if target + window <= n - 1 else [])
            k[target, 0] = q[probes[0], 0] if probes else k[target, 0]
            for p in probes:
                q[p, :h // hk] = q[probes[0], :1]
        else:
            probes = [p for p in range(off + 3, n, 23)]
            for p in probes:
                q[p, 1 % h] = q[p, 0]
                k[p - off, 0] = q[p, 0]
        k = k.to(dtype).float()
        want = O.shared_kv_attention(q.double(), k.double(), scale, window, keep)
        if probes and kind != "near":
            wrong = dict(window_in=(max(window - 1, 0), keep), window_out=(window + 1, keep), first_in=(window, keep - 1),
                         first_out=(window, keep + 1))[kind]
            if wrong[0] > 0:
                far = [p for p in probes if not kind.startswith("window") or p - off >= keep]
                bad = O.shared_kv_attention(q.double(), k.double(), scale, *wrong)
                assert not far or (want - bad)[far].abs().max() > 0.5, kind
        for cuts in portions(n):
            err = (feed(q, k, cuts, dtype, device, scale, window, keep) - want.flatten(1)).abs().max()
            assert err < (2e-5 if dtype == torch.float32 else 2e-2), (kind, window, keep, cuts[:3], float(err))
