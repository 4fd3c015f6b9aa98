"""A plain, slow statement of the Molopel decoder: one function per mechanism, whole sequences, explicit loops over
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
def layer_norm(x, w, eps):
    mean = x.mean(-1, keepdim=True)
    centred = x - mean
    var = (centred * centred).mean(-1, keepdim=True)
    return centred / torch.sqrt(var + eps) * w


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(x):
    return x / (1 + torch.exp(-x))


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z * z * z)))


# ---- position mechanisms --------------------------------------------------------------------------------------
def distance_bucket(n: int, rows: int, bias_max: int) -> int:
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(bias_max / half) * (rows - half)))


def rotate_half(x, first_pos, dims, base):
    """x [n, heads, d], row r sits at position first_pos + r; the first ``dims`` dimensions of each head turn."""
    out = x.clone()
    half = dims // 2
    for i in range(half):
        f = base ** (-2.0 * i / dims)
        for r in range(x.shape[0]):
            a = (first_pos + r) * f
            c, s = math.cos(a), math.sin(a)
            u, v = x[r, :, i], x[r, :, i + half]
            out[r, :, i] = u * c - v * s
            out[r, :, i + half] = v * c + u * s
    return out


# ---- sequence mixers ------------------------------------------------------------------------------------------
def windowed_attention(q, k, v, scale, window, rel, bias_max):
    """q [n, H, d], k [n, G, d], v [n, G, dv]; softmax over the ``window`` newest keys, plus a per-distance bias."""
    n, H = q.shape[0], q.shape[1]
    G = k.shape[1]
    out = torch.zeros(n, H, v.shape[2], dtype=q.dtype)
    for i in range(n):
        lo = max(0, i - window + 1)
        buckets = torch.tensor([distance_bucket(i - j, rel.shape[0], bias_max) for j in range(lo, i + 1)])
        for h in range(H):
            g = h // (H // G)
            s = k[lo:i + 1, g] @ q[i, h] * scale + rel[buckets, h]
            e = torch.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ v[lo:i + 1, g]
    return out


def decayed_linear_attention(q, k, v, decay, state=None):
    """q, k [n, H, d], v [n, H, dv]; S <- decay S + k v^T, o = S^T q. Returns (o, final S)."""
    n, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    dec = torch.tensor(decay, dtype=q.dtype).view(H, 1, 1)
    out = torch.zeros(n, H, v.shape[2], dtype=q.dtype)
    for t in range(n):
        S = dec * S + k[t].unsqueeze(2) * v[t].unsqueeze(1)
        out[t] = torch.einsum("hde,hd->he", S, q[t])
    return out, S


# ---- sublayers ------------------------------------------------------------------------------------------------
def lightning_mixer(h, c, w, p, eps):
    n, H = h.shape[0], c["heads"]
    q = silu(h @ w[p + ".q"].T).view(n, H, c["dim"])
    k = silu(h @ w[p + ".k"].T).view(n, H, c["dim"])
    v = silu(h @ w[p + ".v"].T).view(n, H, c["vdim"])
    o, _ = decayed_linear_attention(q, k, v, c["decay"])
    o = unit_rms(o.reshape(n, -1), eps) * w[p + ".norm"]
    return (o * sigmoid(h @ w[p + ".g"].T)) @ w[p + ".o"].T


def window_mixer(h, c, w, p, eps):
    n, H, G = h.shape[0], c["heads"], c["kv_heads"]
    q = (h @ w[p + ".q"].T + w[p + ".q.b"]).view(n, H, c["dim"])
    k = (h @ w[p + ".k"].T + w[p + ".k.b"]).view(n, G, c["dim"])
    v = (h @ w[p + ".v"].T + w[p + ".v.b"]).view(n, G, c["vdim"])
    q = unit_rms(q, eps) * w[p + ".q.norm"]
    k = unit_rms(k, eps) * w[p + ".k.norm"]
    o = windowed_attention(q, k, v, c["scale"], c["mask"]["size"], w[p + ".rel"], c["bias_max"])
    return o.reshape(n, -1) @ w[p + ".o"].T


def retention_mixer(h, c, w, p, eps):
    n, H = h.shape[0], c["heads"]
    q = (h @ w[p + ".q"].T).view(n, H, c["dim"])
    k = (h @ w[p + ".k"].T).view(n, H, c["dim"])
    v = (h @ w[p + ".v"].T).view(n, H, c["vdim"])
    q = rotate_half(q, 0, c["rot"]["dims"], c["rot"]["base"])
    k = rotate_half(k, 0, c["rot"]["dims"], c["rot"]["base"]) * c["dim"] ** -0.5
    o, _ = decayed_linear_attention(q, k, v, c["decay"])
    o = unit_rms(o, eps).reshape(n, -1)
    return (o * silu(h @ w[p + ".g"].T)) @ w[p + ".o"].T


def parallel_mixer(h, c, w, p, eps):
    left = window_mixer(h, c["left"], w, p + ".left", eps)
    right = retention_mixer(h, c["right"], w, p + ".right", eps)
    return c["left_scale"] * left + c["right_scale"] * right


def dense_ff(h, w, p):
    return (gelu_tanh(h @ w[p + ".gate"].T) * (h @ w[p + ".up"].T)) @ w[p + ".down"].T


# ---- whole model ----------------------------------------------------------------------------------------------
def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], residuals: Optional[list] = None):
    """Logits [n, vocab] of one whole sequence; ``residuals`` collects the stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        h = layer_norm(x, w[f"l{i}.norm1"], eps)
        mixer = {"lightning": lightning_mixer, "parallel": parallel_mixer}[layer["type"]]
        x = x + mixer(h, layer["mixer"], w, f"l{i}.mix", eps)
        if layer["mlp"] is not None:
            x = x + dense_ff(layer_norm(x, w[f"l{i}.norm2"], eps), w, f"l{i}.mlp")
        if residuals is not None:
            residuals.append(x)
    y = layer_norm(x, w["final.norm"], eps) @ w["embed"].T
    cap = cfg["logit_softcap"]
    return cap * torch.tanh(y / cap)


def greedy(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], new: int) -> List[int]:
    out = list(tokens)
    for _ in range(new):
        out.append(int(forward(cfg, w, out)[-1].argmax()))
    return out[len(tokens):]


# ---- random small models --------------------------------------------------------------------------------------
def tensor_shapes(cfg: dict, bias_rows: int = 16) -> Dict[str, tuple]:
    W = cfg["width"]
    shapes = {"embed": (cfg["vocab"], W), "final.norm": (W,)}
    for i, layer in enumerate(cfg["layers"]):
        p, c = f"l{i}", layer["mixer"]
        shapes[p + ".norm1"] = (W,)

        def proj(pre, heads, kv, d, dv, extra):
            shapes[pre + ".q"] = (heads * d, W)
            shapes[pre + ".k"] = (kv * d, W)
            shapes[pre + ".v"] = (kv * dv, W)
            if extra == "g":
                shapes[pre + ".g"] = (heads * dv, W)
            shapes[pre + ".o"] = (W, heads * dv)

        if layer["type"] == "lightning":
            proj(p + ".mix", c["heads"], c["heads"], c["dim"], c["vdim"], "g")
            shapes[p + ".mix.norm"] = (c["heads"] * c["vdim"],)
        else:
            a, r = c["left"], c["right"]
            proj(p + ".mix.left", a["heads"], a["kv_heads"], a["dim"], a["vdim"], "")
            for t, n in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                shapes[f"{p}.mix.left.{t}.b"] = (n,)
            shapes[p + ".mix.left.q.norm"] = shapes[p + ".mix.left.k.norm"] = (a["dim"],)
            shapes[p + ".mix.left.rel"] = (bias_rows, a["heads"])
            proj(p + ".mix.right", r["heads"], r["heads"], r["dim"], r["vdim"], "g")
        if layer["mlp"] is not None:
            shapes[p + ".norm2"] = (W,)
            shapes[p + ".mlp.gate"] = shapes[p + ".mlp.up"] = (layer["mlp"]["ff"], W)
            shapes[p + ".mlp.down"] = (W, layer["mlp"]["ff"])
    return shapes


def random_weights(cfg: dict, seed: int, bias_rows: int = 16) -> Dict[str, torch.Tensor]:
    """bfloat16 tensors whose sublayers all move the residual stream by about its own size."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, bias_rows).items():
        r = torch.randn(*shape, generator=g, dtype=torch.float32)
        if "norm" in name.split(".")[-1]:
            t = 1 + 0.3 * r
        elif name.endswith(".rel"):
            t = r
        elif name.endswith(".b"):
            t = 0.3 * r
        elif name == "embed":
            t = r / math.sqrt(shape[1]) * 2
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
