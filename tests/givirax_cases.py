"""Small Givirax configurations shared by the CPU and GPU tests."""
from __future__ import annotations

import torch

import givirax_oracle as O
from replay_cases import ModelCase


def layer(heads, kv, dim, window, keep, scale, mlp=None):
    return dict(type="attention", mlp=mlp, mixer=dict(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=scale,
                                                      mask=dict(size=window, keep_first=keep)))


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(experts, top, ff):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))


def model(width, vocab, layers, loop=None, emb=3.0, eps=1e-5, positions=288):
    return dict(architecture="Givirax", width=width, vocab=vocab, embedding=dict(scale=emb), norm=dict(eps=eps),
                max_positions=positions, loop=loop, layers=layers)


# sizes that are multiples of nothing in particular, layers that all differ, a loop in the middle
ODD = model(92, 203, [
    layer(3, 1, 20, 7, 3, 0.3, dense(76)),
    layer(4, 2, 28, 20, 17, 0.21, moe(5, 3, 22)),
    layer(2, 2, 36, 33, 1, 0.17),
    layer(6, 2, 12, 50, 0, 0.25, moe(11, 1, 13))], loop=dict(start=1, stop=3, times=3))

# sizes that the tensor-core and cache-streaming kernels take: 64 / 128 heads, grouped and single key heads
EVEN = model(128, 320, [
    layer(4, 2, 64, 33, 18, 0.125, dense(160)),
    layer(5, 1, 128, 50, 5, 0.09, moe(9, 2, 48)),
    layer(2, 2, 64, 16, 16, 0.15, dense(320)),
    layer(34, 2, 32, 70, 2, 0.2, moe(6, 4, 104))], loop=dict(start=0, stop=2, times=2), emb=5.0)

# a window of one token, one head, one expert, a loop of one pass over every layer
ONE = model(64, 101, [
    layer(1, 1, 32, 1, 1, 0.2, moe(1, 1, 40)),
    layer(1, 1, 16, 1, 0, 0.3, dense(64))], loop=dict(start=0, stop=2, times=1), emb=1.0)

# no loop at all
FLAT = model(72, 77, [layer(2, 1, 24, 11, 2, 0.25, moe(4, 2, 24)), layer(2, 1, 24, 11, 2, 0.25, dense(48))], emb=7.0)

CASES = {"odd": ODD, "even": EVEN, "one": ONE, "flat": FLAT}


class Case(ModelCase):
    def __init__(self, path, name, seed=0):
        super().__init__(path, O, CASES[name], O.random_weights(CASES[name], seed))
        self._close = {}

    def close_calls(self, tokens):
        """Tokens whose routing 16-bit rounding may turn: their own logits then belong to other experts."""
        key = tuple(tokens)
        if key not in self._close:
            margins = []
            O.forward(self.cfg, self.w64, tokens, margins=margins)
            self._close[key] = torch.stack(margins).min(0).values < 0.1 if margins else torch.zeros(len(tokens), dtype=bool)
        return self._close[key]
