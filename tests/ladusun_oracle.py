"""A plain, slow statement of the Ladusun decoder: one function per mechanism, whole sequences, explicit loops over
positions where that is the definition. It shares no code with the package and is what the tests compare against.

A model is (config dict, {tensor name: tensor}); everything runs in the dtype the tensors are given in (the tests use
float64 and float32)."""
from __future__ import annotations

import json
import math
import struct
from typing import Dict, List, Optional

import torch


# ---- elementwise pieces ---------------------------------------------------------------------------------------
def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z * z * z)))


def squared_relu(z):
    return torch.clamp(z, min=0) ** 2


# ---- rotation -------------------------------------------------------------------------------------------------
def plain_frequencies(dims, base):
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def banded_frequencies(dims, base, s):
    """Long wavelengths are slowed down by ``factor``, short ones stay, a linear blend in between."""
    out = []
    for f in plain_frequencies(dims, base):
        wl = 2 * math.pi / f
        if wl < s["original"] / s["high"]:
            out.append(f)
        elif wl > s["original"] / s["low"]:
            out.append(f / s["factor"])
        else:
            t = (s["original"] / wl - s["low"]) / (s["high"] - s["low"])
            out.append((1 - t) * f / s["factor"] + t * f)
    return out


def ramped_frequencies(dims, base, s):
    """(frequencies, magnitude): a ramp over the pairs between those that turn ``fast`` and ``slow`` times over the
    original length."""
    def pair_of(turns):
        return dims * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(pair_of(s["fast"])), 0), min(math.ceil(pair_of(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain_frequencies(dims, base)):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * r + f * (1 - r))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate_pairs(x, positions, freqs, magnitude=1.0):
    """x [n, heads, d]: neighbouring entries 2i and 2i + 1 turn by position * freqs[i]; what is beyond stays."""
    out = x.clone()
    for i, f in enumerate(freqs):
        a = torch.tensor([p * f for p in positions], dtype=torch.float64)
        c, s = ((magnitude * t).to(x.dtype).unsqueeze(1) for t in (torch.cos(a), torch.sin(a)))
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i], out[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


# ---- attention ------------------------------------------------------------------------------------------------
def softmax_rows(scores, sink):
    """Weights over the keys of each row; ``sink``: one more score of 0 that belongs to no key."""
    m = scores.max(-1, keepdim=True).values
    if sink:
        m = torch.clamp(m, min=0)
    e = torch.exp(scores - m)
    return e / (e.sum(-1, keepdim=True) + (torch.exp(-m) if sink else 0))


def capped_sink_attention(q, k, v, scale, cap, first=0):
    """q [n, H, d] at positions first .. first + n - 1, k [N, G, d], v [N, G, dv] at positions 0 .. N - 1."""
    n, H = q.shape[:2]
    G = k.shape[1]
    out = q.new_zeros(n, H, v.shape[2])
    for i in range(n):
        for h in range(H):
            g = h // (H // G)
            s = (k[:first + i + 1, g] @ q[i, h]) * scale
            s = cap * torch.tanh(s / cap)
            out[i, h] = softmax_rows(s, True) @ v[:first + i + 1, g]
    return out


def head_gate(o, h, w):
    """o [n, H, dv] times one sigmoid per head of the mixer's input."""
    return o * sigmoid(h @ w.T).unsqueeze(2)


def attention_keys(h, c, w, p):
    n = h.shape[0]
    freqs = banded_frequencies(c["rot"]["dims"], c["rot"]["base"], c["rot"]["scaling"])
    k = (h @ w[p + ".k"].T + w[p + ".k.b"]).view(n, c["kv_heads"], c["dim"])
    v = (h @ w[p + ".v"].T + w[p + ".v.b"]).view(n, c["kv_heads"], c["vdim"])
    return rotate_pairs(k, range(n), freqs), v


def attention_mixer(h, c, w, p, kv):
    """``kv``: rotated keys and values, this layer's own or those of the layer it reads."""
    n = h.shape[0]
    freqs = banded_frequencies(c["rot"]["dims"], c["rot"]["base"], c["rot"]["scaling"])
    q = rotate_pairs((h @ w[p + ".q"].T + w[p + ".q.b"]).view(n, c["heads"], c["dim"]), range(n), freqs)
    o = head_gate(capped_sink_attention(q, *kv, c["scale"], c["softcap"]), h, w[p + ".g"])
    return o.reshape(n, -1) @ w[p + ".o"].T + w[p + ".o.b"]


def latent_attention(q, c, r, uk, uv, scale):
    """q [n, H, dim + rot_dim], latent c [n, rank], shared rotated key part r [n, rot_dim], uk [H, dim, rank],
    uv [H, vdim, rank]; keys and values are written out per head."""
    n, H = q.shape[:2]
    dim = uk.shape[1]
    out = q.new_zeros(n, H, uv.shape[1])
    for h in range(H):
        keys, values = c @ uk[h].T, c @ uv[h].T
        for i in range(n):
            s = (keys[:i + 1] @ q[i, h, :dim] + r[:i + 1] @ q[i, h, dim:]) * scale
            out[i, h] = softmax_rows(s, False) @ values[:i + 1]
    return out


def latent_mixer(h, c, w, p, eps):
    n, H = h.shape[0], c["heads"]
    dim, rd, rank, vdim = c["dim"], c["rot_dim"], c["kv_rank"], c["vdim"]
    freqs, mag = ramped_frequencies(c["rot"]["dims"], c["rot"]["base"], c["rot"]["scaling"])
    q = (h @ w[p + ".q"].T).view(n, H, dim + rd)
    q = torch.cat((q[:, :, :dim], rotate_pairs(q[:, :, dim:], range(n), freqs, mag)), 2)
    a = h @ w[p + ".dkv"].T
    lat = rms_norm(a[:, :rank], w[p + ".dkv.norm"], eps)
    r = rotate_pairs(a[:, None, rank:], range(n), freqs, mag)[:, 0]
    o = latent_attention(q, lat, r, w[p + ".uk"].view(H, dim, rank), w[p + ".uv"].view(H, vdim, rank), c["scale"])
    return head_gate(o, h, w[p + ".g"]).reshape(n, -1) @ w[p + ".o"].T


# ---- gated linear recurrence --------------------------------------------------------------------------------------
def causal_conv(x, taps, bias):
    """x [n, C], taps [C, K]: the last tap meets the current token, what is before the start is zero."""
    n, K = x.shape[0], taps.shape[1]
    out = bias.expand(n, -1).clone()
    for t in range(n):
        for j in range(K):
            if t - (K - 1 - j) >= 0:
                out[t] = out[t] + taps[:, j] * x[t - (K - 1 - j)]
    return out


def block_linear(u, m, b):
    """u [n, C] in B equal parts, part i times m[i] [out, in] plus b[i]."""
    n, (B, s, _) = u.shape[0], m.shape
    return torch.cat([u[:, i * s:(i + 1) * s] @ m[i].T + b[i] for i in range(B)], 1)


def gated_recurrence(u, r, i, lam, s0=None):
    """S_t = a S_(t-1) + sqrt(1 - a^2) i u with log a = -8 r softplus(lam). Returns (all S, the last)."""
    la = -8 * r * softplus(lam)
    a, x = torch.exp(la), torch.sqrt(-torch.expm1(2 * la)) * i * u
    s = torch.zeros_like(u[0]) if s0 is None else s0
    out = []
    for t in range(u.shape[0]):
        s = a[t] * s + x[t]
        out.append(s)
    return torch.stack(out), s


def recurrent_mixer(h, c, w, p):
    y = gelu_tanh(h @ w[p + ".y"].T + w[p + ".y.b"])
    u = causal_conv(h @ w[p + ".x"].T + w[p + ".x.b"], w[p + ".conv"], w[p + ".conv.b"])
    r = sigmoid(block_linear(u, w[p + ".ra"], w[p + ".ra.b"]))
    i = sigmoid(block_linear(u, w[p + ".ri"], w[p + ".ri.b"]))
    return (gated_recurrence(u, r, i, w[p + ".lam"])[0] * y) @ w[p + ".o"].T


# ---- feed-forwards --------------------------------------------------------------------------------------------
def dense_ff(h, w, p):
    return squared_relu(h @ w[p + ".up"].T + w[p + ".up.b"]) @ w[p + ".down"].T + w[p + ".down.b"]


def expert(h, limit, w, p):
    g = torch.clamp(h @ w[p + ".gate"].T, max=limit)
    u = torch.clamp(h @ w[p + ".up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w[p + ".down"].T


def route(z, top, groups, keep):
    """Chosen experts of one token (best first) and their weights: softmax scores, the best ``keep`` of ``groups``
    groups of neighbours by their best score, the ``top`` best experts in those, weights that add up to 1."""
    s = torch.exp(z - z.max())
    s = s / s.sum()
    size = z.shape[0] // groups
    best = sorted(range(groups), key=lambda g: -float(s[g * size:(g + 1) * size].max()))[:keep]
    open_ = [e for g in best for e in range(g * size, (g + 1) * size)]
    ids = sorted(open_, key=lambda e: (-float(s[e]), e))[:top]
    chosen = torch.stack([s[e] for e in ids])
    return ids, chosen / (chosen.sum() + 1e-20)


def choice_margin(z, top, groups, keep):
    """How far (in logits) the token's choice is from another one."""
    size = z.shape[0] // groups
    g = z.view(groups, size).max(1).values.sort(descending=True)
    kept = z.view(groups, size)[g.indices[:keep]].flatten().sort(descending=True).values
    m = float("inf")
    if keep < groups:
        m = min(m, float(g.values[keep - 1] - g.values[keep]))
    if top < kept.shape[0]:
        m = min(m, float(kept[top - 1] - kept[top]))
    return m


def moe_ff(h, c, w, p, margins=None):
    r = c["router"]
    z = h @ w[p + ".router"].T
    rows, close = [], []
    for t in range(h.shape[0]):
        ids, weights = route(z[t], r["top"], r["groups"]["count"], r["groups"]["keep"])
        close.append(choice_margin(z[t], r["top"], r["groups"]["count"], r["groups"]["keep"]))
        rows.append(sum(weights[n] * expert(h[t], c["expert"]["limit"], w, f"{p}.e{e}") for n, e in enumerate(ids)))
    if margins is not None:
        margins.append(torch.tensor(close))
    return torch.stack(rows)


# ---- streams --------------------------------------------------------------------------------------------------
def combine(x, w):
    """x [s, n, W] -> the sublayer's input."""
    return sum(w[s] * x[s] for s in range(x.shape[0]))


def spread(x, y, mix, out):
    """Every stream anew from all old ones (mix [from, to]) and the sublayer's result."""
    n = x.shape[0]
    return torch.stack([sum(mix[s, t] * x[s] for s in range(n)) + out[t] * y for t in range(n)])


# ---- whole model ----------------------------------------------------------------------------------------------
def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], residuals: Optional[list] = None,
            margins: Optional[list] = None):
    """Logits [n, vocab] of one whole sequence; ``residuals`` collects the sum of the streams after every layer,
    ``margins`` how clear each routing decision was."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    x = torch.stack([x] * cfg["streams"])
    shared = {}
    for i, layer in enumerate(cfg["layers"]):
        p, c = f"l{i}", layer["mixer"]

        def sublayer(x, q, f):
            h = rms_norm(combine(x, w[f"{p}.hc{q}.in"]), w[f"{p}.norm{q}"], eps)
            return spread(x, f(h) * w[f"{p}.ls{q}"], w[f"{p}.hc{q}.mix"], w[f"{p}.hc{q}.out"])

        def mixer(h):
            if layer["type"] == "rglru":
                return recurrent_mixer(h, c, w, p + ".mix")
            if layer["type"] == "latent_attention":
                return latent_mixer(h, c, w, p + ".mix", eps)
            if c.get("kv_from") is None:
                shared[i] = attention_keys(h, c, w, p + ".mix")
            return attention_mixer(h, c, w, p + ".mix", shared[i if c.get("kv_from") is None else c["kv_from"]])

        x = sublayer(x, 1, mixer)
        m = layer["mlp"]
        if m is not None:
            x = sublayer(x, 2, lambda h: dense_ff(h, w, p + ".mlp") if m["kind"] == "dense"
                         else moe_ff(h, m, w, p + ".mlp", margins))
        if residuals is not None:
            residuals.append(x.sum(0))
    return rms_norm(x.sum(0), w["final.norm"], eps) @ w["embed"].T


def greedy(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], new: int) -> List[int]:
    out = list(tokens)
    for _ in range(new):
        out.append(int(forward(cfg, w, out)[-1].argmax()))
    return out[len(tokens):]


# ---- random small models --------------------------------------------------------------------------------------
def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    W, S = cfg["width"], cfg["streams"]
    shapes = {"embed": (cfg["vocab"], W), "final.norm": (W,)}
    for i, layer in enumerate(cfg["layers"]):
        c, m, p = layer["mixer"], layer["mlp"], f"l{i}"
        mix = p + ".mix."
        for q in (1,) if m is None else (1, 2):
            shapes[f"{p}.norm{q}"] = shapes[f"{p}.ls{q}"] = (W,)
            shapes[f"{p}.hc{q}.in"] = shapes[f"{p}.hc{q}.out"] = (S,)
            shapes[f"{p}.hc{q}.mix"] = (S, S)
        if layer["type"] == "rglru":
            C, B = c["width"], c["blocks"]
            shapes.update({mix + "y": (C, W), mix + "y.b": (C,), mix + "x": (C, W), mix + "x.b": (C,),
                           mix + "conv": (C, c["conv"]), mix + "conv.b": (C,), mix + "lam": (C,), mix + "o": (W, C)})
            for g in ("ra", "ri"):
                shapes[mix + g], shapes[mix + g + ".b"] = (B, C // B, C // B), (B, C // B)
        elif layer["type"] == "latent_attention":
            H, R = c["heads"], c["kv_rank"]
            shapes.update({mix + "q": (H * (c["dim"] + c["rot_dim"]), W), mix + "dkv": (R + c["rot_dim"], W),
                           mix + "dkv.norm": (R,), mix + "uk": (H * c["dim"], R), mix + "uv": (H * c["vdim"], R),
                           mix + "g": (H, W), mix + "o": (W, H * c["vdim"])})
        else:
            H, G = c["heads"], c["kv_heads"]
            shapes.update({mix + "q": (H * c["dim"], W), mix + "q.b": (H * c["dim"],), mix + "g": (H, W),
                           mix + "o": (W, H * c["vdim"]), mix + "o.b": (W,)})
            if c.get("kv_from") is None:
                shapes.update({mix + "k": (G * c["dim"], W), mix + "k.b": (G * c["dim"],),
                               mix + "v": (G * c["vdim"], W), mix + "v.b": (G * c["vdim"],)})
        if m is None:
            continue
        mlp = p + ".mlp."
        if m["kind"] == "dense":
            shapes.update({mlp + "up": (m["ff"], W), mlp + "up.b": (m["ff"],), mlp + "down": (W, m["ff"]),
                           mlp + "down.b": (W,)})
            continue
        f = m["expert"]["ff"]
        for e in range(m["router"]["experts"]):
            shapes[f"{mlp}e{e}.gate"] = shapes[f"{mlp}e{e}.up"] = (f, W)
            shapes[f"{mlp}e{e}.down"] = (W, f)
        shapes[mlp + "router"] = (m["router"]["experts"], W)
    return shapes


def random_weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """bfloat16 tensors whose sublayers all move the streams by about their own size, with mixes near a permutation of
    the streams and decays from a few tokens to a few hundred."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        r = torch.randn(*shape, generator=g, dtype=torch.float32)
        last = name.split(".")[-1]
        if "norm" in last:
            t = 1 + 0.3 * r
        elif ".hc" in name:
            S = cfg["streams"]
            t = {"in": lambda: (1 + 0.5 * r) / S, "out": lambda: 1 + 0.5 * r,
                 "mix": lambda: torch.eye(S) * 0.8 + 0.15 * r}[last]()
        elif last in ("ls1", "ls2"):
            t = 0.7 + 0.3 * r
        elif last == "lam":
            t = -3 + 1.5 * r
        elif last == "b":
            t = 0.3 * r
        elif last == "conv":
            t = r / math.sqrt(shape[1])
        elif last in ("ra", "ri"):
            t = 2 * r / math.sqrt(shape[2])
        elif name == "embed":
            t = r / cfg["embedding"]["scale"]
        elif last == "router":
            t = 3 * r / math.sqrt(shape[1])
        elif last in ("gate", "up") and ".e" in name:
            t = 2 * r / math.sqrt(shape[1])
        else:
            t = r / math.sqrt(shape[1])
        out[name] = t.to(torch.bfloat16)
    return out


def write_safetensors(path: str, tensors: Dict[str, torch.Tensor]) -> None:
    head, blobs, pos = {}, [], 0
    for name, t in tensors.items():
        raw = t.contiguous().view(torch.int16).numpy().tobytes()
        head[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [pos, pos + len(raw)]}
        blobs.append(raw)
        pos += len(raw)
    text = json.dumps(head).encode()
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text + b"".join(blobs))


def write_model(path, cfg: dict, tensors: Dict[str, torch.Tensor]) -> str:
    path = str(path)
    with open(path + "/config.json", "w") as f:
        json.dump(cfg, f)
    write_safetensors(path + "/model.safetensors", tensors)
    return path
