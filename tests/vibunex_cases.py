"""Small Vibunex configurations shared by the CPU and GPU tests."""
from __future__ import annotations

import copy

import vibunex_oracle as O
from replay_cases import ModelCase


def ramped(dims, base, factor=4.0, fast=8.0, slow=1.0, original=64):
    return dict(dims=dims, base=base, scaling=dict(factor=factor, fast=fast, slow=slow, original=original))


def moe(experts, top, ff, shared, scale):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top, scale=scale), shared=dict(ff=shared))


def layer(heads, kv, dim, vdim, scale, rot, mix_heads, mix_dim, left=0.9, right=1.2, mlp=None):
    return dict(type="parallel", mlp=mlp, mixer=dict(
        left=dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale, rot=rot),
        right=dict(heads=mix_heads, dim=mix_dim), left_scale=left, right_scale=right))


def model(width, vocab, mult, layers, eps=1e-5):
    return dict(architecture="Vibunex", width=width, vocab=vocab, residual_mult=mult, norm=dict(eps=eps), layers=layers)


# sizes that are multiples of nothing in particular, layers that all differ
ODD = model(84, 203, 0.6, [
    layer(4, 2, 28, 20, 0.35, ramped(12, 300.0), 3, 20, mlp=moe(9, 3, 22, 30, 1.7)),
    layer(3, 1, 20, 36, 0.4, ramped(20, 90.0, original=40), 2, 12, 1.1, 0.4),
    layer(6, 3, 12, 28, 0.5, dict(dims=6, base=50.0), 5, 7, 0.5, 1.0, moe(5, 5, 13, 9, 0.8)),
    layer(2, 2, 36, 12, 0.3, ramped(36, 1000.0, factor=2.0), 1, 33, 1.3, 0.7, moe(7, 1, 20, 44, 2.5))])

# sizes that the tensor-core and cache-streaming kernels take
EVEN = model(128, 320, 0.7, [
    layer(8, 2, 64, 64, 0.18, ramped(32, 800.0), 4, 64, mlp=moe(16, 4, 48, 160, 1.3)),
    layer(12, 4, 32, 64, 0.25, ramped(16, 400.0), 3, 32, 1.0, 0.8, moe(8, 2, 64, 72, 2.2)),
    layer(4, 4, 64, 128, 0.16, ramped(64, 2000.0), 2, 40, 0.7, 1.1)])

# many heads, large heads, heads that share one key, wide states
WIDE = model(136, 256, 0.4, [
    layer(20, 4, 128, 128, 0.1, ramped(64, 2000.0), 2, 128, mlp=moe(4, 2, 40, 64, 1.0)),
    layer(34, 2, 32, 72, 0.25, ramped(8, 50.0), 6, 72, 0.6, 0.9, moe(5, 2, 24, 32, 1.4)),
    layer(40, 8, 40, 24, 0.2, ramped(40, 700.0), 9, 16),
    layer(33, 11, 24, 136, 0.2, ramped(24, 100.0), 3, 136, 0.8, 0.5, moe(3, 1, 16, 8, 0.9))])

# one of everything: one head, one state, one expert, a pair of rotated dimensions, factors of 1
ONE = model(64, 101, 1.0, [
    layer(1, 1, 16, 8, 0.5, ramped(2, 10.0, factor=1.0), 1, 8, 1.0, 1.0, moe(1, 1, 40, 8, 1.0)),
    layer(2, 1, 8, 16, 0.6, ramped(8, 10.0), 1, 24, 1.0, 1.0, moe(2, 1, 8, 16, 1.0))])

CASES = {"odd": ODD, "even": EVEN, "wide": WIDE, "one": ONE}


class Case(ModelCase):
    """``every_expert``: the router weights all experts and leaves none out. Rounding in 16 bits turns close choices, and a
    token that went elsewhere reaches all later ones through states and keys; without a choice the rest can be compared
    closely."""

    def __init__(self, path, name, every_expert=False, seed=0):
        cfg = copy.deepcopy(CASES[name])
        for entry in cfg["layers"]:
            if every_expert and entry["mlp"]:
                entry["mlp"]["router"]["top"] = entry["mlp"]["router"]["experts"]
        super().__init__(path, O, cfg, O.random_weights(cfg, seed))
