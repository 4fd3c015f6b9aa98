"""Small Molopel configurations and engine helpers shared by the CPU and GPU tests."""
from __future__ import annotations

import molopel_oracle as M
from replay_cases import ModelCase, run_batches, run_long_decode, run_portions, spread  # noqa: F401


def lightning(heads, dim, vdim, decay, ff=0):
    return dict(type="lightning", mlp=dict(kind="dense", ff=ff) if ff else None,
                mixer=dict(heads=heads, dim=dim, vdim=vdim, decay=decay))


def parallel(left, right, scales, ff=0):
    heads, kv, dim, vdim, window, bias_max, scale = left
    rh, rd, rv, decay, rot, base = right
    return dict(type="parallel", mlp=dict(kind="dense", ff=ff) if ff else None, mixer=dict(
        left=dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, mask=dict(size=window), bias_max=bias_max, scale=scale),
        right=dict(heads=rh, dim=rd, vdim=rv, decay=decay, rot=dict(dims=rot, base=base)),
        left_scale=scales[0], right_scale=scales[1]))


def model(width, vocab, layers, emb=3.0, cap=20.0, eps=1e-5):
    return dict(architecture="Molopel", width=width, vocab=vocab, embedding=dict(scale=emb), norm=dict(eps=eps),
                logit_softcap=cap, layers=layers)


# sizes that are multiples of nothing in particular, a partial rotation, a feed-forward behind either kind of layer
ODD = model(92, 203, [
    lightning(3, 20, 36, [0.5, 0.9, 0.99], ff=76),
    parallel((4, 2, 28, 20, 20, 30, 0.21), (2, 44, 12, [0.97, 0.6], 24, 3000.0), (0.8, 1.3), ff=100),
    parallel((3, 1, 16, 52, 7, 40, 0.3), (5, 12, 24, [0.9, 0.8, 0.7, 0.99, 1.0], 12, 500.0), (1.2, 0.4)),
    lightning(1, 48, 16, [0.95])])

# sizes that the tensor-core and cache-streaming kernels take: 64 / 128 heads, grouped and single key heads
EVEN = model(128, 320, [
    parallel((4, 2, 64, 64, 33, 60, 0.125), (2, 64, 128, [0.98, 0.999], 64, 1e4), (1.0, 0.7), ff=256),
    lightning(2, 128, 64, [0.8, 0.995]),
    parallel((5, 1, 128, 128, 50, 90, 0.09), (3, 32, 64, [0.9, 0.95, 0.99], 32, 2e5), (0.5, 1.0), ff=160),
    lightning(4, 64, 32, [0.3, 0.7, 0.9, 0.99], ff=128)], emb=5.0, cap=15.0)

# a window of one token, decays of one, a single head everywhere
ONE = model(64, 101, [
    parallel((1, 1, 32, 64, 1, 20, 0.2), (1, 16, 16, [1.0], 16, 100.0), (1.0, 1.0), ff=64),
    lightning(1, 16, 16, [1.0], ff=40)], emb=1.0, cap=50.0)

CASES = {"odd": (ODD, 12), "even": (EVEN, 16), "one": (ONE, 2)}


class Case(ModelCase):
    def __init__(self, path, name, seed=0):
        cfg, rows = CASES[name]
        super().__init__(path, M, cfg, M.random_weights(cfg, seed, rows))
