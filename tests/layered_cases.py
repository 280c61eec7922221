"""What the GPU tests of the layered models share: small random models on disk with the expected logits of their oracle, and the
comparison of rows of logits: the root mean square of the difference (mean removed) over the spread of the expected ones."""
import tempfile

import numpy as np

import puppygrad_b200 as pg
from puppygrad_b200 import synthetic

BOUND = {"fp32": 3e-5, "bf16": 4e-2}
MODES = ("fp32", "bf16")


def row_errors(got, want):
    d = np.asarray(got, np.float64) - want
    d -= d.mean(axis=-1, keepdims=True)
    return np.sqrt((d * d).mean(axis=-1)) / want.std()


def assert_rows(got, want, mode, factor=1.0):
    err = row_errors(got, want)
    assert err.max() <= BOUND[mode] * factor, (mode, float(err.max()), np.nonzero(err > BOUND[mode] * factor)[0][:8])


class Case:
    """A small random model on disk with its expected logits."""

    def __init__(self, oracle, cfg, seed, rank=5, edit=None):
        self.oracle, self.cfg, self.dir = oracle, cfg, tempfile.mkdtemp()
        self.w = oracle.random_weights(cfg, seed, rank)
        if edit:
            edit(self.w)
            self.w = {k: synthetic.round_bf16(v) for k, v in self.w.items()}  # what the file holds
        synthetic.write_design_dir(self.dir, cfg, self.w)
        self.models, self.known = {}, {}

    def model(self, mode, **kw):
        key = (mode, tuple(sorted(kw.items())))
        if key not in self.models:
            kw.setdefault("max_context", 4096)
            self.models[key] = pg.load_model(self.dir, pg.CudaConfig(math_mode=mode, **kw))
        return self.models[key]

    def ids(self, n, seed=0):
        return np.random.default_rng(1000 + seed).integers(0, self.cfg["vocab"], n)

    def want(self, ids):
        key = tuple(int(t) for t in ids)
        if key not in self.known:
            self.known[key] = self.oracle.forward(self.cfg, self.w, ids)
        return self.known[key]


def cut(ids, sizes):
    out, at, i = [], 0, 0
    while at < len(ids):
        n = sizes[i % len(sizes)]
        out.append(ids[at:at + n])
        at, i = at + n, i + 1
    return out


def run_portions(model, cache, slot, portions):
    return np.concatenate([model.extend([slot], [p], cache, range(len(p))) for p in portions])


def greedy(case, prompt, n):
    """The oracle's greedy continuation, and how far each choice was from the next best (in spreads)."""
    ids, gaps = [int(t) for t in prompt], []
    for _ in range(n):
        row = case.oracle.forward(case.cfg, case.w, ids)[-1]
        top = np.sort(row)
        gaps.append((top[-1] - top[-2]) / row.std())
        ids.append(int(row.argmax()))
    return ids, gaps


def assert_stream(tokens, want, gaps, n_prompt, bound):
    """Equal up to the first choice that is closer than the bound."""
    for i, (a, b) in enumerate(zip(tokens[n_prompt:], want[n_prompt:])):
        if a != b:
            assert gaps[i] < 10 * bound, (i, a, b, gaps[i])
            return
    assert len(tokens) == len(want)
