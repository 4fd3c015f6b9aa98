"""Small Molopel configurations and engine helpers shared by the CPU and GPU tests."""
from __future__ import annotations

import torch

import molopel_oracle as M


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


class Case:
    """A model on disk, its oracle and an engine over it."""

    def __init__(self, path, name, seed=0):
        self.cfg, rows = CASES[name]
        self.w = M.random_weights(self.cfg, seed, rows)
        self.w64 = {k: v.double() for k, v in self.w.items()}
        self.dir = M.write_model(path, self.cfg, self.w)
        self._cache = {}

    def tokens(self, n, seed):
        return torch.randint(0, self.cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()

    def logits(self, tokens):
        key = tuple(tokens)
        if key not in self._cache:
            self._cache[key] = M.forward(self.cfg, self.w64, tokens)
        return self._cache[key]

    def engine(self, dtype, max_tokens, device):
        from ksanallm_b200.tools.trace_run import build_engine
        return build_engine(self.dir, dtype, max_tokens, device)


class Feed:
    """Feeds sequences to an engine in portions and checks every row of logits against the whole-sequence oracle."""

    def __init__(self, case, engine, tol):
        self.case, self.engine, self.tol = case, engine, tol
        self.at, self.ids, self.fresh, self.worst = {}, {}, 0, 0.0

    def step(self, *portions, end=()):
        """portions: (name, whole token list, how many of its next tokens)."""
        entries, wants = [], []
        for name, tokens, n in portions:
            if name not in self.ids:
                self.fresh += 1
                self.ids[name], self.at[name] = self.fresh, 0
            lo = self.at[name]
            entries.append((self.ids[name], tokens[lo:lo + n], list(range(min(n, len(tokens) - lo)))))
            wants.append(self.case.logits(tokens)[lo:lo + n])
            self.at[name] = min(lo + n, len(tokens))
        got = self.engine.replay(entries, [self.ids.pop(x) for x in end])
        want = torch.cat(wants)
        assert got.shape == want.shape
        err = ((got.double() - want) ** 2).mean(1).sqrt() / self.case_scale(want)
        self.worst = max(self.worst, float(err.max()))
        assert float(err.max()) < self.tol, (portions and [(p[0], self.at[p[0]], p[2]) for p in portions], err)

    def case_scale(self, want):
        return float((want - want.mean(1, keepdim=True)).pow(2).mean().sqrt())

    def whole(self, name, tokens, cuts):
        for i, c in enumerate(cuts):
            self.step((name, tokens, c), end=[name] if i == len(cuts) - 1 else [])
        assert self.at[name] == len(tokens)


def spread(n, sizes):
    """Portions of the given sizes, over and over, that add up to n."""
    out = []
    while sum(out) < n:
        out.append(min(sizes[len(out) % len(sizes)], n - sum(out)))
    return out


def run_portions(case, engine, tol):
    """A sequence cut in many ways gives the same logits as the oracle's whole pass."""
    toks = case.tokens(150, 1)
    feed = Feed(case, engine, tol)
    for i, cuts in enumerate(([150], [1] * 150, [2] * 75, spread(150, [1, 2, 3]), [140] + [1] * 10, spread(150, [16]),
                              spread(150, [17, 1, 33]), [128, 22], [1, 149], [129, 1, 20], spread(150, [64, 2, 1, 1]))):
        feed.whole(f"a{i}", toks, cuts)
    return feed.worst


def run_batches(case, engine, tol):
    """Unequal requests in one batch, portions beside single tokens, requests that pause, slots and pages in reuse."""
    feed = Feed(case, engine, tol)
    t = {c: case.tokens(n, 10 + i) for i, (c, n) in enumerate(dict(a=120, b=45, c=7, d=90, e=33, f=1, g=64).items())}
    feed.step(("a", t["a"], 50), ("b", t["b"], 45), ("c", t["c"], 1))
    feed.step(("b2", t["b"], 2), ("a", t["a"], 1), ("c", t["c"], 1), end=["b"])
    feed.step(("d", t["d"], 80), ("a", t["a"], 20), ("c", t["c"], 1), ("b2", t["b"], 20))
    feed.step(("d", t["d"], 1), ("a", t["a"], 1), ("c", t["c"], 4), ("b2", t["b"], 1), end=["c"])
    feed.step(("d", t["d"], 1), ("f", t["f"], 1), ("b2", t["b"], 22), end=["f", "b2"])
    feed.step(("e", t["e"], 17), ("a", t["a"], 2), ("g", t["g"], 64), ("d", t["d"], 8), end=["g", "d"])
    feed.step(("a", t["a"], 46), ("e", t["e"], 16), ("c2", t["c"], 7), end=["a", "e", "c2"])
    for i in range(6):  # the pool is refilled from its released pages and slots again and again
        feed.step((f"x{i}", t["a"], 70), (f"y{i}", t["d"], 19))
        feed.step((f"x{i}", t["a"], 1), (f"y{i}", t["d"], 1), end=[f"x{i}", f"y{i}"])
    return feed.worst


def run_long_decode(case, engine, tol):
    toks = case.tokens(260, 3)
    feed = Feed(case, engine, tol)
    feed.whole("long", toks, [3] + [1] * 257)
    return feed.worst
