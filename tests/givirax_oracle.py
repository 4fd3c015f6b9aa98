"""A plain, slow statement of the Givirax decoder: one function per mechanism, whole sequences, explicit loops over
positions where that is the definition. It shares no code with the package and is what the tests compare against.

A model is (config dict, {tensor name: tensor}); everything runs in the dtype the tensors are given in (the tests use
float64 and float32)."""
from __future__ import annotations

import json
import math
import struct
from typing import Dict, Iterator, List, Optional, Tuple

import torch


# ---- elementwise pieces ---------------------------------------------------------------------------------------
def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def silu(z):
    return z / (1 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z * z * z)))


# ---- start of the stream --------------------------------------------------------------------------------------
def embed(tokens, table, scale, positions):
    """Scaled token rows plus the unscaled learned vector of each position."""
    n = len(tokens)
    return table[torch.tensor(tokens)] * scale + positions[:n]


def layer_runs(n_layers: int, loop: Optional[dict]) -> Iterator[Tuple[int, Optional[int]]]:
    """(layer, number of the pass that starts with it - None inside a pass or outside of the loop)."""
    if not loop:
        yield from ((i, None) for i in range(n_layers))
        return
    for i in range(loop["start"]):
        yield i, None
    for t in range(loop["times"]):
        for i in range(loop["start"], loop["stop"]):
            yield i, t if i == loop["start"] else None
    for i in range(loop["stop"], n_layers):
        yield i, None


# ---- attention whose values are its keys ----------------------------------------------------------------------
def sees(i: int, j: int, window: int, keep_first: int) -> bool:
    return j <= i and (i - j < window or j < keep_first)


def shared_kv_attention(q, k, scale, window, keep_first):
    """q [n, H, d], k [n, G, d]; softmax over the visible keys, which are also the values. Returns [n, H, d]."""
    n, H = q.shape[0], q.shape[1]
    G = k.shape[1]
    out = torch.zeros_like(q)
    for i in range(n):
        js = torch.tensor([j for j in range(i + 1) if sees(i, j, window, keep_first)])
        for g in range(G):
            keys = k[js, g]
            heads = slice(g * (H // G), (g + 1) * (H // G))
            s = (q[i, heads] @ keys.T) * scale
            e = torch.exp(s - s.max(-1, keepdim=True).values)
            out[i, heads] = (e / e.sum(-1, keepdim=True)) @ keys
    return out


def attention_mixer(h, c, w, p):
    n = h.shape[0]
    q = (h @ w[p + ".q"].T).view(n, c["heads"], c["dim"])
    k = (h @ w[p + ".k"].T).view(n, c["kv_heads"], c["dim"])
    o = shared_kv_attention(q, k, c["scale"], c["mask"]["size"], c["mask"]["keep_first"])
    return o.reshape(n, -1) @ w[p + ".o"].T


# ---- feed-forwards --------------------------------------------------------------------------------------------
def dense_ff(h, w, p):
    return gelu_tanh(h @ w[p + ".up"].T) @ w[p + ".down"].T


def expert(h, w, p):
    return (silu(h @ w[p + ".gate"].T) * (h @ w[p + ".up"].T)) @ w[p + ".down"].T


def route(logits, top):
    """The ``top`` experts with the largest logits of one token and the softmax over just their logits."""
    order = sorted(range(logits.shape[0]), key=lambda e: -float(logits[e]))[:top]
    z = torch.stack([logits[e] for e in order])
    x = torch.exp(z - z.max())
    return order, x / x.sum()


def moe_ff(h, top, w, p, margins=None):
    z = h @ w[p + ".router"].T + w[p + ".router.b"]
    if margins is not None and top < z.shape[1]:  # how far each token's choice is from another one
        s = z.sort(-1, descending=True).values
        margins.append(s[:, top - 1] - s[:, top])
    rows = []
    for t in range(h.shape[0]):
        ids, weights = route(z[t], top)
        rows.append(sum(weights[n] * expert(h[t], w, f"{p}.e{e}") for n, e in enumerate(ids)))
    return torch.stack(rows)


def feed_forward(h, mlp, w, p, margins=None):
    return dense_ff(h, w, p) if mlp["kind"] == "dense" else moe_ff(h, mlp["router"]["top"], w, p, margins)


# ---- whole model ----------------------------------------------------------------------------------------------
def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], residuals: Optional[list] = None,
            margins: Optional[list] = None):
    """Logits [n, vocab] of one whole sequence; ``residuals`` collects the stream after every layer run, ``margins`` how
    clear each routing decision was."""
    eps = cfg["norm"]["eps"]
    start = embed(tokens, w["embed"], cfg["embedding"]["scale"], w["pos"])
    x = start
    for i, t in layer_runs(len(cfg["layers"]), cfg.get("loop")):
        layer = cfg["layers"][i]
        if t is not None:
            if t > 0:
                x = x + start
            x = x + w["loop.step"][t]
        h = rms_norm(x, w[f"l{i}.norm1"], eps)
        y = attention_mixer(h, layer["mixer"], w, f"l{i}.mix")
        if layer["mlp"] is not None:
            y = y + feed_forward(h, layer["mlp"], w, f"l{i}.mlp", margins)
        x = x + y
        if residuals is not None:
            residuals.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T


def greedy(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], new: int) -> List[int]:
    out = list(tokens)
    for _ in range(new):
        out.append(int(forward(cfg, w, out)[-1].argmax()))
    return out[len(tokens):]


# ---- random small models --------------------------------------------------------------------------------------
def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    W = cfg["width"]
    shapes = {"embed": (cfg["vocab"], W), "pos": (cfg["max_positions"], W), "final.norm": (W,), "head": (cfg["vocab"], W)}
    if cfg.get("loop"):
        shapes["loop.step"] = (cfg["loop"]["times"], W)
    for i, layer in enumerate(cfg["layers"]):
        c, m, p = layer["mixer"], layer["mlp"], f"l{i}"
        shapes[p + ".norm1"] = (W,)
        shapes[p + ".mix.q"] = (c["heads"] * c["dim"], W)
        shapes[p + ".mix.k"] = (c["kv_heads"] * c["dim"], W)
        shapes[p + ".mix.o"] = (W, c["heads"] * c["vdim"])
        if m is None:
            continue
        if m["kind"] == "dense":
            shapes[p + ".mlp.up"], shapes[p + ".mlp.down"] = (m["ff"], W), (W, m["ff"])
            continue
        for e in range(m["router"]["experts"]):
            f = m["expert"]["ff"]
            shapes[f"{p}.mlp.e{e}.gate"] = shapes[f"{p}.mlp.e{e}.up"] = (f, W)
            shapes[f"{p}.mlp.e{e}.down"] = (W, f)
        shapes[p + ".mlp.router"], shapes[p + ".mlp.router.b"] = (m["router"]["experts"], W), (m["router"]["experts"],)
    return shapes


def random_weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """bfloat16 tensors whose sublayers all move the residual stream by about its own size."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        r = torch.randn(*shape, generator=g, dtype=torch.float32)
        if "norm" in name.split(".")[-1]:
            t = 1 + 0.3 * r
        elif name in ("pos", "loop.step"):
            t = 0.7 * r
        elif name.endswith(".router.b"):
            t = r
        elif name == "embed":
            t = r / cfg["embedding"]["scale"]
        elif name.endswith(".router"):
            t = 3 * r / math.sqrt(shape[1])
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
