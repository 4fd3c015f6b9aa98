"""Small Ladusun configurations shared by the CPU and GPU tests."""
from __future__ import annotations

import copy

import ladusun_oracle as O
from replay_cases import ModelCase


def banded(dims, base, factor=8.0, low=1.0, high=4.0, original=64):
    return dict(dims=dims, base=base, scaling=dict(factor=factor, low=low, high=high, original=original))


def ramped(dims, base, factor=4.0, fast=8.0, slow=1.0, original=64):
    return dict(dims=dims, base=base, scaling=dict(factor=factor, fast=fast, slow=slow, original=original))


def attention(heads, kv, dim, vdim, scale, softcap, rot, mlp=None, kv_from=None):
    m = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale, softcap=softcap, rot=rot)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="attention", mixer=m, mlp=mlp)


def latent(heads, dim, rot_dim, vdim, rank, scale, rot, mlp=None):
    return dict(type="latent_attention", mlp=mlp, mixer=dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=rank,
                                                             scale=scale, rot=rot))


def rglru(width, blocks, conv, mlp=None):
    return dict(type="rglru", mixer=dict(width=width, blocks=blocks, conv=conv), mlp=mlp)


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(experts, top, ff, limit, groups, keep):
    return dict(kind="moe", expert=dict(ff=ff, limit=limit),
                router=dict(experts=experts, top=top, groups=dict(count=groups, keep=keep)))


def model(width, vocab, streams, layers, emb=3.0, eps=1e-5):
    return dict(architecture="Ladusun", width=width, vocab=vocab, streams=streams, embedding=dict(scale=emb),
                norm=dict(eps=eps), layers=layers)


# sizes that are multiples of nothing in particular, layers that all differ, two readers of one layer's keys
ODD = model(84, 203, 3, [
    rglru(60, 3, 3, dense(76)),
    attention(4, 2, 28, 20, 0.35, 2.5, banded(12, 300.0), moe(9, 3, 22, 1.5, 3, 2)),
    latent(3, 20, 12, 28, 36, 0.3, ramped(12, 500.0)),
    attention(4, 2, 28, 20, 0.3, 4.0, banded(12, 300.0), dense(50), kv_from=1),
    rglru(36, 1, 5),
    attention(3, 1, 20, 36, 0.4, 3.0, banded(20, 1000.0, factor=2.0), moe(6, 1, 13, 0.8, 6, 1)),
    attention(2, 2, 28, 20, 0.3, 6.0, banded(12, 300.0), kv_from=1),
    latent(5, 12, 20, 20, 28, 0.35, ramped(20, 90.0, original=40), moe(8, 4, 30, 2.0, 2, 2))])

# sizes that the tensor-core and cache-streaming kernels take
EVEN = model(128, 320, 4, [
    latent(4, 64, 32, 64, 128, 0.12, ramped(32, 800.0), dense(160)),
    rglru(256, 2, 4, moe(16, 4, 48, 1.2, 4, 2)),
    attention(8, 2, 64, 64, 0.18, 3.0, banded(32, 400.0), moe(8, 2, 64, 2.0, 2, 1)),
    rglru(128, 2, 2),
    attention(8, 2, 64, 64, 0.16, 5.0, banded(32, 400.0), dense(320), kv_from=2)], emb=5.0)

# large heads, a long latent, blocks wider than a tile of channels, a long convolution
WIDE = model(136, 256, 2, [
    rglru(192, 1, 6, dense(64)),
    latent(3, 128, 64, 128, 512, 0.1, ramped(64, 2000.0), moe(4, 2, 40, 1.0, 4, 3)),
    attention(3, 3, 128, 64, 0.12, 4.0, banded(128, 3000.0)),
    latent(10, 40, 16, 72, 200, 0.2, ramped(16, 60.0)),
    attention(34, 2, 32, 128, 0.25, 2.0, banded(8, 50.0), moe(5, 2, 24, 0.7, 1, 1))], emb=2.0)

# one of everything: one stream, one head, one block, one tap, one expert, a pair of rotated dimensions
ONE = model(64, 101, 1, [
    rglru(32, 1, 1, moe(1, 1, 40, 1.0, 1, 1)),
    latent(1, 8, 2, 16, 16, 0.5, ramped(2, 10.0)),
    attention(1, 1, 16, 16, 0.3, 1.5, banded(2, 10.0), dense(64)),
    attention(1, 1, 16, 16, 0.3, 1.5, banded(2, 10.0), kv_from=2)], emb=1.0)

# nothing that carries a state
STATELESS = model(72, 77, 2, [
    attention(2, 1, 24, 24, 0.4, 3.0, banded(24, 100.0), moe(4, 2, 24, 1.0, 2, 1)),
    latent(2, 24, 8, 24, 32, 0.3, ramped(8, 100.0), dense(48)),
    attention(4, 1, 24, 24, 0.4, 3.0, banded(24, 100.0), kv_from=0)], emb=7.0)

CASES = {"odd": ODD, "even": EVEN, "wide": WIDE, "one": ONE, "stateless": STATELESS}


class Case(ModelCase):
    """``every_expert``: the router weights all experts and leaves none out. Rounding in 16 bits turns close choices, and a
    token that went elsewhere reaches all later ones through states and keys; without a choice the rest can be compared
    closely."""

    def __init__(self, path, name, every_expert=False, seed=0):
        cfg = copy.deepcopy(CASES[name])
        for layer in cfg["layers"]:
            if every_expert and layer["mlp"] and layer["mlp"]["kind"] == "moe":
                r = layer["mlp"]["router"]
                r["top"], r["groups"]["keep"] = r["experts"], r["groups"]["count"]
        super().__init__(path, O, cfg, O.random_weights(cfg, seed))
