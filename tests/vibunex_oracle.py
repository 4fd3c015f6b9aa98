"""A plain, slow statement of the Vibunex decoder: one function per mechanism, whole sequences, explicit loops over
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


def silu(z):
    return z * sigmoid(z)


def squared_relu(z):
    return torch.clamp(z, min=0) ** 2


# ---- rotation -------------------------------------------------------------------------------------------------
def ramped_frequencies(dims, base, s):
    """(frequencies, magnitude): a ramp over the pairs between those that turn ``fast`` and ``slow`` times over the
    original length; without ``s`` the plain powers of the base."""
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not s:
        return plain, 1.0

    def pair_of(turns):
        return dims * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(pair_of(s["fast"])), 0), min(math.ceil(pair_of(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * r + f * (1 - r))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate_halves(x, positions, freqs, magnitude=1.0):
    """x [n, heads, d]: of the first 2 len(freqs) entries, i and i + len(freqs) turn by position * freqs[i]."""
    out, half = x.clone(), len(freqs)
    for i, f in enumerate(freqs):
        a = torch.tensor([p * f for p in positions], dtype=torch.float64)
        c, s = ((magnitude * t).to(x.dtype).unsqueeze(1) for t in (torch.cos(a), torch.sin(a)))
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i], out[:, :, i + half] = u * c - v * s, v * c + u * s
    return out


# ---- attention whose heads' weights are mixed -------------------------------------------------------------------
def sink_weights(scores, sink):
    """Softmax weights over the keys of one row whose denominator has one more term exp(sink)."""
    m = torch.maximum(scores.max(), sink)
    e = torch.exp(scores - m)
    return e / (e.sum() + torch.exp(sink - m))


def talking_attention(q, k, v, scale, sink, talk, first=0):
    """q [n, H, d] at positions first .. first + n - 1, k [N, G, d], v [N, G, dv] at positions 0 .. N - 1. The weights of
    all heads are mixed by talk [to, from] before each head sums up the values of its own key/value head."""
    n, H = q.shape[:2]
    mine = [h // (H // k.shape[1]) for h in range(H)]  # every query head's key/value head
    out = q.new_zeros(n, H, v.shape[2])
    for i in range(n):
        N = first + i + 1
        scores = torch.einsum("nhd,hd->hn", k[:N, mine], q[i]) * scale
        p = torch.stack([sink_weights(s, x) for s, x in zip(scores, sink)])
        out[i] = torch.einsum("hn,nhv->hv", talk @ p, v[:N, mine])
    return out


def attention_mixer(h, c, w, p, eps):
    n, H, G = h.shape[0], c["heads"], c["kv_heads"]
    freqs, mag = ramped_frequencies(c["rot"]["dims"], c["rot"]["base"], c["rot"].get("scaling"))
    q = rms_norm(h @ w[p + ".q"].T, w[p + ".q.norm"], eps).view(n, H, c["dim"])
    k = rms_norm(h @ w[p + ".k"].T, w[p + ".k.norm"], eps).view(n, G, c["dim"])
    v = (h @ w[p + ".v"].T).view(n, G, c["vdim"])
    o = talking_attention(rotate_halves(q, range(n), freqs, mag), rotate_halves(k, range(n), freqs, mag), v, c["scale"],
                          w[p + ".sink"], w[p + ".talk"])
    return (o.reshape(n, -1) * sigmoid(h @ w[p + ".g"].T)) @ w[p + ".o"].T


# ---- time mixing ------------------------------------------------------------------------------------------------
def shifted(h, mu, before=None):
    """Every token's h moved towards the previous token's (zeros ahead of the first one) by mu."""
    before = torch.zeros_like(h[:1]) if before is None else before
    return h + (torch.cat((before, h[:-1])) - h) * mu


def decays(m, w1, w2, w0):
    return torch.exp(-torch.exp(torch.tanh(m @ w1.T) @ w2.T + w0))


def bonus_recurrence(r, k, v, w, u, s0=None):
    """r, k, w [n, heads, d], v [n, heads, dv], u [heads, d]: o_t = (S + diag(u) k_t v_t^T)^T r_t, then
    S <- diag(w_t) S + k_t v_t^T. Returns (o [n, heads, dv], the last S [heads, d, dv])."""
    s = r.new_zeros(r.shape[1], r.shape[2], v.shape[2]) if s0 is None else s0
    out = []
    for t in range(r.shape[0]):
        kv = k[t].unsqueeze(2) * v[t].unsqueeze(1)
        out.append(((s + u.unsqueeze(2) * kv) * r[t].unsqueeze(2)).sum(1))
        s = w[t].unsqueeze(2) * s + kv
    return torch.stack(out) if out else torch.zeros_like(v), s


def time_mixer(h, c, w, p, eps):
    n, H, d = h.shape[0], c["heads"], c["dim"]
    m = {x: shifted(h, w[f"{p}.mu.{x}"]) for x in "rkvgw"}
    r, k, v = ((m[x] @ w[f"{p}.{x}"].T).view(n, H, d) for x in "rkv")
    gate = silu(m["g"] @ w[p + ".g"].T)
    dec = decays(m["w"], w[p + ".w1"], w[p + ".w2"], w[p + ".w0"]).view(n, H, d)
    o = rms_norm(bonus_recurrence(r, k, v, dec, w[p + ".u"])[0], 1.0, eps)
    return (o.reshape(n, -1) * w[p + ".norm"] * gate) @ w[p + ".o"].T


# ---- feed-forward -----------------------------------------------------------------------------------------------
def expert(h, w, p):
    return squared_relu(h @ w[p + ".up"].T) @ w[p + ".down"].T


def route(z, top, scale):
    """Chosen experts of one token (best first) and their weights."""
    s = sigmoid(z)
    ids = sorted(range(z.shape[0]), key=lambda e: (-float(s[e]), e))[:top]
    return ids, [s[e] * scale for e in ids]


def choice_margin(z, top):
    """How far (in logits) the token's choice is from another one."""
    s = z.sort(descending=True).values
    return float(s[top - 1] - s[top]) if top < z.shape[0] else float("inf")


def moe_ff(h, c, w, p, margins=None):
    r = c["router"]
    z = h @ w[p + ".router"].T
    rows = []
    for t in range(h.shape[0]):
        ids, weights = route(z[t], r["top"], r["scale"])
        rows.append(sum(a * expert(h[t], w, f"{p}.e{e}") for a, e in zip(weights, ids)))
    if margins is not None:
        margins.append(torch.tensor([choice_margin(x, r["top"]) for x in z]))
    return torch.stack(rows) + expert(h, w, p + ".shared") * sigmoid(h @ w[p + ".shared.sg"].T)


# ---- whole model ------------------------------------------------------------------------------------------------
def gated(y, h, w, p):
    """A sublayer's result times sigmoid(W h + b) of the sublayer's input, number by number."""
    return y * sigmoid(h @ w[p].T + w[p + ".b"])


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], residuals: Optional[list] = None,
            margins: Optional[list] = None):
    """Logits [n, vocab] of one whole sequence; ``residuals`` collects the stream after every layer, ``margins`` how clear
    each routing decision was."""
    eps, scale = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][torch.tensor(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        p, c = f"l{i}", layer["mixer"]
        h = rms_norm(x, w[p + ".norm1"], eps)
        y = c["left_scale"] * attention_mixer(h, c["left"], w, p + ".mix.left", eps) + \
            c["right_scale"] * time_mixer(h, c["right"], w, p + ".mix.right", eps)
        total = gated(y, h, w, p + ".rg1")
        if layer["mlp"] is not None:
            h = rms_norm(x, w[p + ".norm2"], eps)
            total = total + gated(moe_ff(h, layer["mlp"], w, p + ".mlp", margins), h, w, p + ".rg2")
        x = x + scale * total
        if residuals is not None:
            residuals.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T


def greedy(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], new: int) -> List[int]:
    out = list(tokens)
    for _ in range(new):
        out.append(int(forward(cfg, w, out)[-1].argmax()))
    return out[len(tokens):]


# ---- random small models ----------------------------------------------------------------------------------------
def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    W = cfg["width"]
    shapes = {"embed": (cfg["vocab"], W), "head": (cfg["vocab"], W), "final.norm": ()}
    for i, layer in enumerate(cfg["layers"]):
        a, r, m, p = layer["mixer"]["left"], layer["mixer"]["right"], layer["mlp"], f"l{i}"
        for q in (1,) if m is None else (1, 2):
            shapes.update({f"{p}.norm{q}": (), f"{p}.rg{q}": (W, W), f"{p}.rg{q}.b": (W,)})
        H, G, x = a["heads"], a["kv_heads"], p + ".mix.left."
        shapes.update({x + "q": (H * a["dim"], W), x + "k": (G * a["dim"], W), x + "v": (G * a["vdim"], W),
                       x + "q.norm": (H * a["dim"],), x + "k.norm": (G * a["dim"],), x + "talk": (H, H), x + "sink": (H,),
                       x + "g": (H * a["vdim"], W), x + "o": (W, H * a["vdim"])})
        n, x = r["heads"] * r["dim"], p + ".mix.right."
        rank = (6, 16, 11, 3)[i % 4]  # (not part of a configuration: the tensors' shapes tell)
        shapes.update({f"{x}mu.{c}": (W,) for c in "rkvgw"})
        shapes.update({x + c: (n, W) for c in "rkvg"})
        shapes.update({x + "w1": (rank, W), x + "w2": (n, rank), x + "w0": (n,), x + "u": (r["heads"], r["dim"]),
                       x + "norm": (n,), x + "o": (W, n)})
        if m is None:
            continue
        E = m["router"]["experts"]
        for e, ff in [(f"e{j}", m["expert"]["ff"]) for j in range(E)] + [("shared", m["shared"]["ff"])]:
            shapes[f"{p}.mlp.{e}.up"], shapes[f"{p}.mlp.{e}.down"] = (ff, W), (W, ff)
        shapes[p + ".mlp.router"], shapes[p + ".mlp.shared.sg"] = (E, W), (1, W)
    return shapes


def random_weights(cfg: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    """bfloat16-representable float32 weights under which every mechanism matters: sinks and mixed weights of both signs,
    decays between fast and slow, router logits that are apart."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        t = torch.randn(shape, generator=g)
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm2", "norm"):
            t = 1.0 + 0.3 * t
        elif ".mu." in name:
            t = torch.rand(shape, generator=g)
        elif last == "talk":
            t = torch.eye(shape[0]) + 0.5 * t
        elif last == "w0":
            t = -3.0 + 1.7 * t
        elif last == "sink":
            t = 2.0 + t
        elif last == "u":
            pass
        elif last == "b":
            t = 0.5 * t
        elif last == "router":
            t = t * 2.5 / math.sqrt(shape[1])
        elif last == "embed":
            t = t * 2.0
        else:
            t = t * (1.6 if last in ("up", "q", "k") else 1.0) / math.sqrt(shape[-1])
        out[name] = t.bfloat16().float()
    return out


def write_model(path, cfg: dict, w: Dict[str, torch.Tensor]) -> str:
    """config.json and model.safetensors (bfloat16) in the folder ``path``."""
    import os
    with open(os.path.join(path, "config.json"), "w", encoding="utf-8") as f:
        json.dump(cfg, f)
    header, blobs, at = {}, [], 0
    for name, t in w.items():
        raw = t.bfloat16().contiguous().view(torch.int16).numpy().tobytes()
        header[name] = dict(dtype="BF16", shape=list(t.shape), data_offsets=[at, at + len(raw)])
        at += len(raw)
        blobs.append(raw)
    head = json.dumps(header).encode()
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(head)))
        f.write(head)
        f.write(b"".join(blobs))
    return str(path)
