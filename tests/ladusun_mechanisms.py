"""Ladusun's mechanisms one at a time, fed in portions through the package's operators and compared with the oracle, on
any device. Probes make faults show: one key scores far above all others, or hardly any key scores at all."""
import torch

import ladusun_oracle as O
from ksanallm_b200 import ops
from ksanallm_b200.config.model_config import _ladusun_rotary
from ksanallm_b200.engine.step_input import make_step_input
from ksanallm_b200.models.mixers import LatentWeights, RecurrenceWeights
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
    return ([n], [n - 40] + [1] * 40, [2, 100, 16, 17, n - 135], [1, 2] + [1] * 30 + [n - 33], [128, n - 128])


def rotary(rot, kind, length, device):
    r = _ladusun_rotary(rot, kind)
    return ref.rotary_table(r.dims, r.base, length, device, r.scaling)


# ---- capped attention with a sink -----------------------------------------------------------------------------
def attention_case(dtype, device, H=4, G=2, d=64, dv=64, cap=4.0, dims=16, n=180, kind="random", seed=0):
    """kind: random | far (single keys far back that stand out) | faint (scores far below the sink)"""
    g = torch.Generator().manual_seed(seed + d + H)
    rot = dict(dims=dims, base=200.0, scaling=dict(factor=8.0, low=1.0, high=4.0, original=64))
    freqs = O.banded_frequencies(dims, rot["base"], rot["scaling"])
    rnd = lambda *s: torch.randn(*s, generator=g).to(dtype).float()  # noqa: E731
    q, k, v, gate = rnd(n, H, d), rnd(n, G, d), rnd(n, G, dv), rnd(n, H)
    scale = 2.0 / d ** 0.5
    if kind == "far":
        k *= 0.02
        for i in range(60, n, 7):  # queries that ask for one early token by the dimensions that do not turn
            probe = torch.zeros(d)
            probe[dims:] = 3 * torch.randn(d - dims, generator=g)
            q[i], k[(i * 5) % 40] = probe.to(dtype).float(), probe.to(dtype).float()
    if kind == "faint":
        k[:, :, dims:], q[:, :, dims:] = -1.5, 1.5
        scale = 0.2
    k = k.to(dtype).float()
    kr = O.rotate_pairs(k.double(), range(n), freqs).to(dtype).double()
    qr = O.rotate_pairs(q.double(), range(n), freqs).to(dtype).double()
    want = O.capped_sink_attention(qr, kr, v.double(), scale, cap) * O.sigmoid(gate.double()).unsqueeze(2)
    table = rotary(rot, "llama3", n, device)
    x = torch.cat((q.flatten(1), k.flatten(1), v.flatten(1), gate, torch.zeros(n, -gate.shape[1] % 8)), 1).to(dtype)
    at = [0, H * d, (H + G) * d, (H + G) * d + G * dv]
    for cuts in portions(n):
        cache = torch.zeros((n + BS - 1) // BS + 1, G * BS * (d + dv), dtype=dtype, device=device)
        rows = []
        for done, c, meta in steps(n, cuts, device):
            xd = x[done:done + c].clone().to(device)
            qq, kk, vv = (xd[:, a:b].unflatten(1, (h, -1)) for a, b, h in zip(at, at[1:], (H, G, G)))
            gg = xd[:, at[3]:at[3] + H]
            ops.qk_norm_cache(qq, kk, vv, meta.slot_mapping, cache, BS, None, None, 1e-5, meta.positions, table)
            out = torch.full((c, H * dv + 8), 7.0, dtype=dtype, device=device)
            ops.window_attention(qq, cache, meta, BS, G, dv, scale, 0, None, 1.0, out[:, :H * dv], 0, cap, True, gg)
            # a second reader of the same keys: its own queries only
            q2 = x[done:done + c].clone().to(device)[:, :H * d].unflatten(1, (H, d))
            ops.qk_norm_cache(q2, None, None, meta.slot_mapping, cache, BS, None, None, 1e-5, meta.positions, table)
            out2 = torch.zeros(c, (H * dv + 7) // 8 * 8, dtype=dtype, device=device)[:, :H * dv]
            ops.window_attention(q2, cache, meta, BS, G, dv, scale, 0, None, 1.0, out2, 0, cap, True, gg)
            assert torch.equal(out2, out[:, :H * dv])
            assert (out[:, H * dv:] == 7).all()
            rows.append(out[:, :H * dv].double().cpu())
        err = (torch.cat(rows) - want.flatten(1)).abs().max() / want.abs().max()
        assert err < tolerance(dtype), (kind, H, G, d, dv, cap, cuts[:3], float(err))


# ---- latent attention -------------------------------------------------------------------------------------------
def latent_case(dtype, device, H=4, dim=64, rot_dim=32, vdim=64, rank=128, n=180, kind="random", seed=0):
    g = torch.Generator().manual_seed(seed + dim + H)
    rot = dict(dims=rot_dim, base=150.0, scaling=dict(factor=4.0, fast=8.0, slow=1.0, original=64))
    freqs, mag = O.ramped_frequencies(rot_dim, rot["base"], rot["scaling"])
    rnd = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    q, a, gate = rnd(n, H, dim + rot_dim), rnd(n, rank + rot_dim), rnd(n, H).to(dtype).float()
    norm = 1 + 0.3 * rnd(rank)
    uk, uv = (rnd(H, dim, rank) / rank ** 0.5).to(dtype).float(), (rnd(H, vdim, rank) / rank ** 0.5).to(dtype).float()
    scale = 0.7 / (dim + rot_dim) ** 0.5
    if kind == "far":  # every seventh query asks for one early token by its unrotated part
        q *= 0.1
        a[:, rank:] *= 0.05
        lat = O.rms_norm(a[:, :rank], norm, 1e-5)
        for i in range(60, n, 7):
            for h in range(H):
                key = uk[h] @ lat[(i * 5) % 40]
                q[i, h, :dim] = key * (12.0 / (scale * float(key @ key)))
    q, a = q.to(dtype).float(), a.to(dtype).float()
    lat = O.rms_norm(a[:, :rank].double(), norm.double(), 1e-5).to(dtype).double()
    r = O.rotate_pairs(a[:, None, rank:].double(), range(n), freqs, mag)[:, 0].to(dtype).double()
    qr = torch.cat((q[..., :dim].double(), O.rotate_pairs(q[..., dim:].double(), range(n), freqs, mag)), 2)
    want = O.latent_attention(qr, lat, r, uk.double(), uv.double(), scale) * O.sigmoid(gate.double()).unsqueeze(2)
    table = rotary(rot, "yarn", n, device)
    w = LatentWeights(uk.to(dtype).to(device), uv.to(dtype).to(device))
    x = torch.cat((q.flatten(1), a, gate, torch.zeros(n, -(q[0].numel() + a.shape[1] + H) % 8)), 1).to(dtype)
    nq, na = H * (dim + rot_dim), rank + rot_dim
    for cuts in portions(n):
        cache = torch.zeros((n + BS - 1) // BS + 1, BS * na, dtype=dtype, device=device)
        rows = []
        for done, c, meta in steps(n, cuts, device):
            xd = x[done:done + c].clone().to(device)
            out = torch.full((c, H * vdim + 8), 7.0, dtype=dtype, device=device)
            ops.latent_attention(xd[:, :nq].unflatten(1, (H, dim + rot_dim)), xd[:, nq:nq + na], norm.to(device), 1e-5,
                                 table, cache, meta, BS, w, scale, xd[:, nq + na:nq + na + H], out[:, :H * vdim])
            assert (out[:, H * vdim:] == 7).all()
            rows.append(out[:, :H * vdim].double().cpu())
        err = (torch.cat(rows) - want.flatten(1)).abs().max() / want.abs().max()
        assert err < tolerance(dtype) * (1 if dtype == torch.float32 else 1.5), (kind, H, dim, rot_dim, vdim, rank, cuts[:3], float(err))


# ---- gated recurrence -----------------------------------------------------------------------------------------------
def recurrence_weights(C, B, K, dtype, device, g, lam_mean=-3.0):
    rnd = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    s = C // B
    gates = (2 * rnd(2, B, s, s) / s ** 0.5).to(dtype)
    w = {"p.conv": rnd(C, K) / K ** 0.5, "p.conv_b": 0.3 * rnd(C), "p.gates": gates, "p.gates_b": 0.5 * rnd(2, C),
         "p.lam": lam_mean + 1.5 * rnd(C)}
    return w, RecurrenceWeights({k: v.to(device) for k, v in w.items()}, "p", 8.0)


def recurrence_reference(x, y, w, mem, dtype):
    """mem [K, C]: entering state and earlier inputs. Returns (out, new mem) in 64 bits, u rounded as it is stored."""
    C, K = w["p.conv"].shape
    B = w["p.gates"].shape[1]
    xs = torch.cat((mem[1:], x), 0)
    u = O.causal_conv(xs, w["p.conv"].double(), w["p.conv_b"].double())[K - 1:].to(dtype).double()
    gates, gb = w["p.gates"].double(), w["p.gates_b"].double().view(2, B, C // B)
    r, i = (O.sigmoid(O.block_linear(u, gates[n], gb[n])) for n in (0, 1))
    S, last = O.gated_recurrence(u, r, i, w["p.lam"].double(), mem[0])
    return S * O.gelu_tanh(y), torch.cat((last.unsqueeze(0), xs[x.shape[0]:]), 0)


def recurrence_case(dtype, device, C=256, B=2, K=4, n=300, lam_mean=-3.0, seed=0, tol=None):
    g = torch.Generator().manual_seed(seed + C + K)
    w, dev_w = recurrence_weights(C, B, K, dtype, device, g, lam_mean)
    x, y = (torch.randn(n, C, generator=g).to(dtype) for _ in range(2))
    want, mem = recurrence_reference(x.double(), y.double(), w, torch.zeros(K, C, dtype=torch.float64), dtype)
    for cuts in portions(n) + ([3] * (n // 3),):
        state = torch.randn(3, 1, K, C, generator=g).to(device)
        before = state.clone()
        rows = []
        for done, c, meta in steps(n, cuts, device):
            xy = torch.cat((y[done:done + c], x[done:done + c]), 1).to(device)
            out = torch.full((c, C + 8), 7.0, dtype=dtype, device=device)
            ops.gated_recurrence(xy[:, :C], xy[:, C:], state, meta, dev_w, out[:, :C])
            assert (out[:, C:] == 7).all()
            rows.append(out[:, :C].double().cpu())
        tol = tol or tolerance(dtype) * (1 if dtype == torch.float32 else 0.5)
        err = (torch.cat(rows) - want).abs().max() / want.abs().max()
        assert err < tol, (C, B, K, cuts[:3], float(err))
        assert (state[1, 0].double().cpu() - mem).abs().max() < tol * mem.abs().max()
        assert torch.equal(state[[0, 2]], before[[0, 2]])  # slots of other sequences


def recurrence_batch(dtype, device, C=128, B=2, K=4):
    """Unequal sequences in one step: fresh ones and ones that go on, prompts and single tokens, scattered slots."""
    g = torch.Generator().manual_seed(C)
    w, dev_w = recurrence_weights(C, B, K, dtype, device, g)
    lens, new = [300, 260, 2, 40, 33, 1, 500, 7], [300, 130, 2, 1, 1, 1, 1, 1]
    slots, prefill = [5, 0, 7, 2, 9, 1, 3, 8], 3
    state = torch.randn(10, 1, K, C, generator=g)
    cu = [0]
    for q in new:
        cu.append(cu[-1] + q)
    T = cu[-1]
    pos = [n - q + i for n, q in zip(lens, new) for i in range(q)]
    meta = make_step_input([0] * T, pos, [0] * T, cu, lens, torch.zeros(len(lens), 40), num_prefill=prefill, device=device,
                           state_slots=slots)
    xy = torch.randn(T, 2 * C, generator=g).to(dtype)
    dev = state.clone().to(device)
    out = torch.zeros(T, C, dtype=dtype, device=device)
    d = xy.to(device)
    ops.gated_recurrence(d[:, :C], d[:, C:], dev, meta, dev_w, out)
    for b, (n, q) in enumerate(zip(lens, new)):
        mem = state[slots[b], 0].double() if n > q else torch.zeros(K, C, dtype=torch.float64)
        rows = xy[cu[b]:cu[b + 1]].double()
        want, mem = recurrence_reference(rows[:, C:], rows[:, :C], w, mem, dtype)
        tol = tolerance(dtype) * (1 if dtype == torch.float32 else 0.5)
        assert (out[cu[b]:cu[b + 1]].double().cpu() - want).abs().max() < tol * want.abs().max(), b
        assert (dev[slots[b], 0].double().cpu() - mem).abs().max() < tol * mem.abs().max(), b
    assert torch.equal(dev[[4, 6]].cpu(), state[[4, 6]])


# ---- streams ----------------------------------------------------------------------------------------------------------
def hyper_case(dtype, device, S=4, H=128, T=5, k=3):
    g = torch.Generator().manual_seed(S * H)
    rnd = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    x, rows, w = rnd(T, H).to(dtype), rnd(T * k, H).to(dtype), rnd(H).to(dtype)
    ls, mix, out_w, in_w = rnd(H), rnd(S, S), rnd(S), rnd(S)
    pos, wts = torch.randperm(T * k, generator=g).int(), torch.rand(T, k, generator=g)
    pos[4] = -1
    start, streams = rnd(T, H), rnd(T, S, H)
    dev = lambda t: None if t is None else t.to(device)  # noqa: E731
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    norm = lambda v: O.rms_norm(O.combine(v, in_w.double()), w.double(), 1e-5)  # noqa: E731
    for one in (True, False):  # all streams still one row, or apart
        old = (start if one else streams).to(device)
        v = torch.stack([start] * S).double() if one else streams.transpose(0, 1).double()
        got = ops.hyper_norm(None, None, None, old, None, None, None, dev(in_w), dev(w), 1e-5, dtype)
        assert (got.double().cpu() - norm(v)).abs().max() < tol * norm(v).abs().max()
        for use in range(1, 8):
            y = torch.zeros(T, H, dtype=torch.float64)
            if use & 1:
                y += x.double()
            if use & 2:
                for t in range(T):
                    for j in range(k):
                        p = int(pos[t * k + j])
                        if p >= 0:
                            y[t] += wts[t, j].double() * rows[p].double()
            if use & 4:
                y *= ls.double()
            new = O.spread(v, y, mix.double(), out_w.double())
            keep = torch.zeros(T, S, H, device=device) if one else old.clone()
            got = ops.hyper_norm(dev(x) if use & 1 else None, dev(ls) if use & 4 else None,
                                 (dev(rows), dev(pos), dev(wts)) if use & 2 else None, old if one else keep, dev(mix),
                                 dev(out_w), keep, dev(in_w), dev(w), 1e-5, dtype)
            assert (keep.transpose(0, 1).double().cpu() - new).abs().max() < 2e-5 * new.abs().max(), (S, H, use)
            assert (got.double().cpu() - norm(new)).abs().max() < tol * norm(new).abs().max(), (S, H, use)


# ---- feed-forward pieces ------------------------------------------------------------------------------------------------
def router_case(device, experts, top, groups, keep, T=40):
    g = torch.Generator().manual_seed(experts * 7 + groups)
    z = torch.randn(T, (experts + 7) // 8 * 8, generator=g)
    z[:, experts:] = 50.0  # padding columns are no experts, however large
    ids, w = ops.moe_topk(z.to(device), experts, top, None, groups, keep)
    differs = 0
    for t in range(T):
        want, ww = O.route(z[t, :experts].double(), top, groups, keep)
        assert ids[t].tolist() == want
        assert (w[t].double().cpu() - ww).abs().max() < 1e-6
        differs += want != O.route(z[t, :experts].double(), top, 1, 1)[0]
    assert differs or keep >= min(top, groups)  # (the best n experts are in the best n groups)


def activation_case(dtype, device, rows=9, cols=104):
    g = torch.Generator().manual_seed(cols)
    x = (3 * torch.randn(rows, 2 * cols, generator=g)).to(dtype)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    got = ops.activation(x.to(device), "relu2").double().cpu()
    assert (got - O.squared_relu(x.double())).abs().max() < tol * 80
    if device == "cpu":
        f = ref.clamped_gate_mul
    else:
        from ksanallm_b200.ops.cuda_mixer import clamped_gate_mul as f
    for limit in (0.7, 2.0, 50.0):
        gate, up = torch.clamp(x[:, :cols].double(), max=limit), torch.clamp(x[:, cols:].double(), -limit, limit)
        want = gate * O.sigmoid(1.702 * gate) * (up + 1)
        assert (f(x.to(device), limit, 1.702).double().cpu() - want).abs().max() < tol * max(1.0, float(want.abs().max()))
