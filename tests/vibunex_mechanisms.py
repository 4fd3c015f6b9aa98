"""Vibunex' mechanisms one at a time, fed in portions through the package's operators and compared with the oracle, on any
device. Probes make faults show: one key scores far above all others, one head's weights matter to one other head alone, a
token's state is all that is read later."""
import torch

import vibunex_oracle as O
from ksanallm_b200 import ops
from ksanallm_b200.config.model_config import _ladusun_rotary
from ksanallm_b200.engine.step_input import make_step_input
from ksanallm_b200.ops import reference as ref

BS = 16


def tolerance(dtype):
    return 3e-5 if dtype == torch.float32 else 2e-2


def steps(n, cuts, device, slot=1):
    """One sequence of n tokens in portions; its pages lie in no natural order and page 0 is somebody else's."""
    pages = list(range((n + BS - 1) // BS))[::-1]
    table = torch.tensor([[p + 1 for p in pages]])
    done = 0
    for c in cuts:
        slots = [int(table[0, p // BS]) * BS + p % BS for p in range(done, done + c)]
        yield done, c, make_step_input([0] * c, list(range(done, done + c)), slots, [0, c], [done + c], table,
                                       num_prefill=0 if c == 1 and done else 1, device=device, state_slots=[slot])
        done += c
    assert done == n


def portions(n):
    return ([n], [n - 40] + [1] * 40, [2, 100, 16, 17, n - 135], [1, 2] + [1] * 30 + [n - 33], [128, n - 128], [64, 65, n - 129])


# ---- attention with mixed weights ---------------------------------------------------------------------------------
def attention_case(dtype, device, H=4, G=2, d=64, dv=64, dims=16, n=180, kind="random", seed=0):
    """kind: random | far (single keys far back that stand out) | sink (scores below the sinks) | swap (every head hands its
    weights to the next one, so that a head's own weights never meet its own values)"""
    g = torch.Generator().manual_seed(seed + d + H)
    rot = dict(dims=dims, base=200.0, scaling=dict(factor=4.0, fast=8.0, slow=1.0, original=64))
    freqs, mag = O.ramped_frequencies(dims, rot["base"], rot["scaling"])
    rnd = lambda *s: torch.randn(*s, generator=g).to(dtype).float()  # noqa: E731
    q, k, v, gate = rnd(n, H, d), rnd(n, G, d), rnd(n, G, dv), rnd(n, H * dv)
    wq, wk = 1 + 0.3 * rnd(H * d), 1 + 0.3 * rnd(G * d)
    sink = rnd(H)
    talk = (torch.eye(H) + 0.6 * torch.randn(H, H, generator=g)).bfloat16().float()
    scale = 2.0 / d ** 0.5
    if kind == "far":
        k *= 0.02
        wq[:], wk[:] = 1.0, 1.0
        for i in range(60, n, 7):  # queries that ask for one early token by the dimensions that do not turn
            probe = torch.zeros(d)
            probe[dims:] = 3 * torch.randn(d - dims, generator=g)
            q[i], k[(i * 5) % 40] = probe.to(dtype).float(), probe.to(dtype).float()
    if kind == "sink":
        sink = 6.0 + sink
    if kind == "swap":
        talk = torch.roll(torch.eye(H), 1, 0) * 1.5
    k = k.to(dtype).float()
    norm = lambda x, w: O.rms_norm(x.double().flatten(1), w.double(), 1e-5).view(x.shape)  # noqa: E731
    kr = O.rotate_halves(norm(k, wk), range(n), freqs, mag).to(dtype).double()
    qr = O.rotate_halves(norm(q, wq), range(n), freqs, mag).to(dtype).double()
    want = 0.7 * O.talking_attention(qr, kr, v.double(), scale, sink.double(), talk.double()).flatten(1) * O.sigmoid(gate.double())
    r = _ladusun_rotary(rot, "yarn")
    table = ref.rotary_table(r.dims, r.base, n, device, r.scaling)
    pad = -(H * d + G * (d + dv) + H * dv) % 8
    x = torch.cat((q.flatten(1), k.flatten(1), v.flatten(1), gate, torch.zeros(n, pad)), 1).to(dtype)
    at = [0, H * d, (H + G) * d, (H + G) * d + G * dv]
    dev = lambda t: t.to(device)  # noqa: E731
    for cuts in portions(n):
        cache = torch.zeros((n + BS - 1) // BS + 1, G * BS * (d + dv), dtype=dtype, device=device)
        rows = []
        for done, c, meta in steps(n, cuts, device):
            xd = x[done:done + c].clone().to(device)
            qq, kk, vv = (xd[:, a:b].unflatten(1, (h, -1)) for a, b, h in zip(at, at[1:], (H, G, G)))
            ops.qk_norm_cache(qq, kk, vv, meta.slot_mapping, cache, BS, dev(wq), dev(wk), 1e-5, meta.positions, table, True, True)
            out = torch.full((c, H * dv + 8), 7.0, dtype=dtype, device=device)
            ops.talking_attention(qq, cache, meta, BS, G, dv, scale, dev(sink), dev(talk), 0.7, out[:, :H * dv],
                                  xd[:, at[3]:at[3] + H * dv])
            assert (out[:, H * dv:] == 7).all()
            rows.append(out[:, :H * dv].double().cpu())
        err = (torch.cat(rows) - want).abs().max() / want.abs().max()
        assert err < tolerance(dtype), (kind, H, G, d, dv, cuts[:3], float(err))


# ---- time mixing ----------------------------------------------------------------------------------------------------
def token_mix_case(dtype, device, W, rows=5, n=150, seed=0):
    g = torch.Generator().manual_seed(seed + W)
    h, mu = torch.randn(n, W, generator=g).to(dtype), torch.rand(rows, W, generator=g)
    want = torch.stack([O.shifted(h.double(), m.double()) for m in mu])
    for cuts in portions(n):
        state = torch.full((3, 1, 1, W + 8), 5.0, device=device)
        got = [ops.token_mix(h[done:done + c].to(device).contiguous(), mu.to(device), state, meta).double().cpu()
               for done, c, meta in steps(n, cuts, device)]
        assert (torch.cat(got, 1) - want).abs().max() < (1e-6 if dtype == torch.float32 else 3e-2), cuts[:3]
        assert (state[:, ..., :8] == 5).all() and (state[0] == 5).all()
        assert torch.equal(state[1, 0, 0, 8:].cpu(), h[-1].float())


def recurrence_inputs(dtype, h, d, n, z_mean, seed, probe):
    g = torch.Generator().manual_seed(seed + 7 * h + d)
    rnd = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    r, k, v = (rnd(n, h * d).to(dtype) for _ in range(3))
    z, w0, u = rnd(n, h * d), z_mean + rnd(h * d), rnd(h, d)
    if probe:  # from the middle on nothing is written any more: what is read is an early token, through every decay since
        k[n // 2:] = 0
        k[: n // 2] *= 0.01
        k[5] = 3.0
    return r, k, v, z, w0, u


def recurrence_case(dtype, device, h, d, n=180, z_mean=-3.0, seed=0, probe=False, tol=None):
    r, k, v, z, w0, u = recurrence_inputs(dtype, h, d, n, z_mean, seed, probe)
    sh = lambda x: x.double().view(n, h, d)  # noqa: E731
    decay = torch.exp(-torch.exp(z.double() + w0.double()))
    want, last = O.bonus_recurrence(sh(r), sh(k), sh(v), decay.view(n, h, d), u.double())
    pad = -(h * d) % 8
    for cuts in portions(n) if n < 400 else ([n], [n // 2, n - n // 2]):
        state = torch.randn(3, 1, 1, h * d * d + 20, device=device)
        keep = state.clone()
        rows = []
        for done, c, meta in steps(n, cuts, device):
            x = [torch.nn.functional.pad(t[done:done + c], (0, pad)).to(device)[:, :h * d] for t in (r, k, v, z)]
            rows.append(ops.time_mix(*x, w0.to(device), u.to(device), state, meta).double().cpu())
        scale = want.abs().amax((1, 2), keepdim=True).clamp(min=1e-3 * float(want.abs().max()))
        err = ((torch.cat(rows) - want).abs() / scale).max()
        assert err < (tol or tolerance(dtype)), (h, d, cuts[:3], float(err))
        got = state[1, 0, 0, :h * d * d].double().cpu().view(h, d, d)
        assert (got - last).abs().max() < (tol or 1e-4) * last.abs().max().clamp(min=1e-6), cuts[:3]
        assert torch.equal(state[[0, 2]], keep[[0, 2]]) and torch.equal(state[1, ..., h * d * d:], keep[1, ..., h * d * d:])


def recurrence_batch(dtype, device, h, d):
    """Unequal sequences at different places of their own in one step, states in scattered slots."""
    lens, news, slots = [200, 64, 90, 31, 1, 77], [130, 64, 3, 1, 1, 1], [4, 0, 6, 2, 5, 1]
    ins = [recurrence_inputs(dtype, h, d, n, -2.0, i, False) for i, n in enumerate(lens)]
    w0, u = ins[0][4], ins[0][5]
    cu, wants, states, pos = [0], [], torch.randn(7, 1, 1, h * d * d, device=device), []
    for (r, k, v, z, _, _), n, m, s in zip(ins, lens, news, slots):
        sh = lambda x: x.double().view(-1, h, d)  # noqa: E731
        decay = torch.exp(-torch.exp(z.double() + w0.double())).view(n, h, d)
        _, s0 = O.bonus_recurrence(sh(r)[:n - m], sh(k)[:n - m], sh(v)[:n - m], decay[:n - m], u.double())
        if n > m:
            states[s, 0, 0] = s0.flatten().float().to(device)
        wants.append(O.bonus_recurrence(sh(r)[n - m:], sh(k)[n - m:], sh(v)[n - m:], decay[n - m:], u.double(), s0 if n > m else None))
        cu.append(cu[-1] + m)
        pos += range(n - m, n)
    meta = make_step_input([0] * cu[-1], pos, [0] * cu[-1], cu, lens, torch.zeros(len(lens), 1), num_prefill=3, device=device,
                           state_slots=slots)
    pad = -(h * d) % 8
    x = [torch.nn.functional.pad(torch.cat([i[j][n - m:] for i, n, m in zip(ins, lens, news)]), (0, pad)).to(device)[:, :h * d]
         for j in range(4)]
    out = ops.time_mix(*x, w0.to(device), u.to(device), states, meta).double().cpu()
    want = torch.cat([w[0] for w in wants])
    assert (out - want).abs().max() < tolerance(dtype) * want.abs().max()
    for s, (_, last) in zip(slots, wants):
        assert (states[s, 0, 0].double().cpu() - last.flatten()).abs().max() < 1e-4 * last.abs().max()


def tanh_case(device, n):
    x = 3 * torch.randn(40, n, generator=torch.Generator().manual_seed(n))
    want = torch.tanh(x.double())
    a = ops.tanh_parts(x.to(device), torch.float32).double().cpu()
    b = ops.tanh_parts(x.to(device), torch.bfloat16).double().cpu()
    assert b.shape == (40, 2 * n)
    assert (a - want).abs().max() < 1e-6 and (b[:, :n] + b[:, n:] - want).abs().max() < 2e-5
    assert (b[:, :n] - want).abs().max() > 1e-4


def head_norm_case(dtype, device, h, d, n=37):
    g = torch.Generator().manual_seed(h + d)
    o, z = (torch.randn(n, h * d, generator=g).to(dtype) for _ in range(2))
    w = 1 + 0.4 * torch.randn(h * d, generator=g)
    want = 1.3 * O.rms_norm(o.double().view(n, h, d), 1.0, 1e-3).flatten(1) * w.double() * O.silu(z.double())
    wide = torch.zeros(n, h * d + 8, dtype=dtype, device=device)
    zd = torch.cat((z, z), 1).to(device)[:, h * d:]
    ops.gated_norm(o.to(device).view(n, h, d), zd, w.to(device), 1e-3, "silu", 1.3, wide[:, :h * d], per_head=True)
    assert (wide[:, :h * d].double().cpu() - want).abs().max() < (1e-5 if dtype == torch.float32 else 1e-2) * want.abs().max()
    assert (wide[:, h * d:] == 0).all()


# ---- gated residual ---------------------------------------------------------------------------------------------------
def residual_case(dtype, device, H, T=21, top=3):
    g = torch.Generator().manual_seed(H)
    rnd = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    x, xg, y, yg = (rnd(T, H).to(dtype) for _ in range(4))
    rows, pos, wts = rnd(T * top, H).to(dtype), torch.randperm(T * top, generator=g).int(), torch.rand(T, top, generator=g)
    ys, stream, w = rnd(T, 24), rnd(T, H), [rnd(H).to(dtype) for _ in range(2)]
    d64 = lambda t: t.double()  # noqa: E731
    routed = torch.stack([sum(d64(wts)[t, j] * d64(rows)[pos[t * top + j]] for j in range(top)) for t in range(T)])
    gx, gy = d64(x) * O.sigmoid(d64(xg)), O.sigmoid(d64(yg))
    for terms in ("both", "mixers", "shared", "neither"):
        total = torch.zeros(T, H, dtype=torch.float64)
        if terms != "neither":
            total = total + gx
        if terms in ("both", "shared"):
            total = total + ((routed if terms == "both" else 0) + d64(y) * O.sigmoid(d64(ys[:, 5:6]))) * gy
        v = d64(stream) + 0.3 * total
        for norms in (1, 2):
            dev = lambda t: t.to(device)  # noqa: E731
            s = stream.clone().to(device)
            ff = terms in ("both", "shared")
            wide = torch.cat((x, xg, yg), 1).to(device)
            out = ops.gated_stream_norm(
                wide[:, :H] if terms != "neither" else None, wide[:, H:2 * H] if terms != "neither" else None,
                (dev(rows), dev(pos), dev(wts)) if terms == "both" else None, dev(y) if ff else None,
                dev(ys)[:, 5] if ff else None, wide[:, 2 * H:] if ff else None, 0.3, s, s, [dev(w[i]) for i in range(norms)], 1e-4,
                dtype)
            assert out.shape == (norms, T, H)
            assert (s.double().cpu() - v).abs().max() < 1e-5 * v.abs().max()
            for i in range(norms):
                want = O.rms_norm(v, d64(w[i]), 1e-4)
                assert (out[i].double().cpu() - want).abs().max() < (1e-5 if dtype == torch.float32 else 1e-2) * want.abs().max()


# ---- routing and experts ------------------------------------------------------------------------------------------------
def router_case(device, experts, top, scale=1.7):
    z = torch.randn(50, experts + 3, generator=torch.Generator().manual_seed(experts)) * 2
    ids, w = ops.moe_topk(z.to(device), experts, top, None, 1, 1, "sigmoid", scale)
    for t in range(50):
        want_ids, want = O.route(z[t, :experts].double(), top, scale)
        assert ids[t].tolist() == want_ids
        assert (w[t].double().cpu() - torch.stack(want)).abs().max() < 1e-5


def expert_case(dtype, device, T, E, top, H, I):
    g = torch.Generator().manual_seed(T + E)
    x = torch.randn(T, H, generator=g).to(dtype)
    up = (1.5 * torch.randn(E, I, H, generator=g) / H ** 0.5).to(dtype)
    down = (torch.randn(E, H, I, generator=g) / I ** 0.5).to(dtype)
    ids = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)]).int()
    y, pos = ops.moe_expert_rows(x.to(device), ids.to(device), up.to(device), down.to(device), plain=True)
    y, pos = y.double().cpu(), pos.cpu()
    for t in range(0, T, 3):
        for j in range(top):
            e = int(ids[t, j])
            want = O.expert(x[t].double(), {"p.up": up[e].double(), "p.down": down[e].double()}, "p")
            assert (y[int(pos[t * top + j])] - want).abs().max() < (1e-5 if dtype == torch.float32 else 3e-2) * want.abs().max()


def relu2_case(dtype, device, cols):
    x = torch.randn(9, 2 * cols, generator=torch.Generator().manual_seed(cols)).to(dtype).to(device)
    for part in (x, x[:, cols:], x[:, :cols]):
        want = O.squared_relu(part.double().cpu())
        assert (ops.activation(part, "relu2").double().cpu() - want).abs().max() <= (1e-6 if dtype == torch.float32 else 8e-3) * want.max()
