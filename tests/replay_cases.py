"""A model on disk beside a plain oracle, and feeding it token by token, in portions and in mixed batches: shared by the
tests of models whose oracle states whole sequences."""
from __future__ import annotations

import torch


class ModelCase:
    """A model folder, its oracle (``forward(cfg, weights, tokens) -> logits``, ``write_model``) and engines over it."""

    def __init__(self, path, oracle, cfg, weights):
        self.oracle, self.cfg, self.w = oracle, cfg, weights
        self.w64 = {k: v.double() for k, v in self.w.items()}
        self.dir = oracle.write_model(path, cfg, self.w)
        self._cache = {}

    def tokens(self, n, seed):
        return torch.randint(0, self.cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()

    def logits(self, tokens):
        key = tuple(tokens)
        if key not in self._cache:
            self._cache[key] = self.oracle.forward(self.cfg, self.w64, tokens)
        return self._cache[key]

    def close_calls(self, tokens):
        """Tokens whose own logits rounding in 16 bits may change altogether (a discrete choice that is a close one)."""
        return torch.zeros(len(tokens), dtype=torch.bool)

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
        entries, wants, close = [], [], []
        for name, tokens, n in portions:
            if name not in self.ids:
                self.fresh += 1
                self.ids[name], self.at[name] = self.fresh, 0
            lo = self.at[name]
            entries.append((self.ids[name], tokens[lo:lo + n], list(range(min(n, len(tokens) - lo)))))
            wants.append(self.case.logits(tokens)[lo:lo + n])
            if self.engine.model.dtype != torch.float32:
                close.append(self.case.close_calls(tokens)[lo:lo + n])
            self.at[name] = min(lo + n, len(tokens))
        got = self.engine.replay(entries, [self.ids.pop(x) for x in end])
        want = torch.cat(wants)
        assert got.shape == want.shape
        err = ((got.double() - want) ** 2).mean(1).sqrt() / self.case_scale(want)
        if close:
            assert float(torch.cat(close).float().mean()) < 0.5 or len(err) < 20
            err = err.masked_fill(torch.cat(close), 0.0)
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
