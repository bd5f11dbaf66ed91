"""What the GPU tests of the layered designs share: a configuration with seeded weights loaded from files, comparison with the
design's numpy oracle, prompts in portions."""
import numpy as np

TOL = {"float32": 3e-5, "bfloat16": 4e-2}


class Case:
    """A configuration with the oracle's seeded weights, loaded from files in one or both number formats."""

    def __init__(self, oracle, qb, ctx, path, cfg, seed=1, edit=None):
        self.oracle, self.qb, self.ctx, self.cfg = oracle, qb, ctx, cfg
        self.W = oracle.random_weights(cfg, seed)
        if edit:
            edit(self.W)
        self.dir = str(path)
        oracle.write_model(self.dir, cfg, self.W)
        self.models = {}
        self.rng = np.random.default_rng(seed + 100)

    def model(self, dtype):
        if dtype not in self.models:
            self.models[dtype] = self.qb.Model.load(self.ctx, self.dir, dtype)
        return self.models[dtype]

    def batch(self, dtype, n_seqs=1, max_ctx=512, **kw):
        return self.qb.Batch(self.model(dtype), n_seqs, max_ctx, 0, **kw)

    def tokens(self, n):
        return self.rng.integers(0, self.cfg["vocab"], n).tolist()

    def want(self, tokens, trace=None):
        return self.oracle.forward(self.cfg, self.W, tokens, np.float64, trace)

    def slack(self, tokens, trace=None):
        """What rounding the operands of the products to bfloat16 does to every row (0 in exact arithmetic)."""
        tr = None if trace is None else []
        d = distance(self.oracle.forward(self.cfg, self.W, tokens, np.float64, tr, self.oracle.to_bf16), self.want(tokens, trace))
        return d if tr is None else (d, [distance(a, b) for a, b in zip(tr, trace)])

    def greedy(self, prompt, n):
        """The oracle's greedy continuation."""
        seq = list(prompt)
        for _ in range(n):
            seq.append(int(self.want(seq)[-1].argmax()))
        return seq[len(prompt):]

    def close(self):
        for m in self.models.values():
            m.close()


def distance(got, want):
    """Root-mean-square difference per row relative to the rms of the whole expected array."""
    return np.sqrt(((got - want) ** 2).mean(-1)) / np.sqrt((want ** 2).mean())


def close_to(got, want, dtype, what="", slack=None):
    """slack (bfloat16): rows that rounding alone moves far may differ by six times that; half of the rows by a third of the
    tolerance at most."""
    assert np.isfinite(got).all(), what
    e = distance(got, want)
    lim = np.full(len(e), TOL[dtype])
    if slack is not None and dtype == "bfloat16":
        lim = np.maximum(lim, 6 * slack)
        assert np.median(e) < max(TOL[dtype] / 3, 2 * np.median(slack)), "%s: the median row differs by %.3g" % (what, np.median(e))
    assert (e < lim).all(), "%s: row %d differs by %.3g" % (what, int((e / lim).argmax()), e[int((e / lim).argmax())])


def in_portions(b, seq, tokens, size):
    """Logits at every position, the tokens cut into portions of `size` (a number, or a list that repeats)."""
    out, at, i = [], 0, 0
    sizes = [size] if isinstance(size, int) else size
    while at < len(tokens):
        n = min(sizes[i % len(sizes)], len(tokens) - at)
        out.append(b.score(seq, tokens[at:at + n], range(n)))
        at, i = at + n, i + 1
    return np.concatenate(out)
