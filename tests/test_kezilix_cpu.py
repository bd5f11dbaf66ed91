"""The plain restatement of the Kezilix design (oracle/kezilix_oracle.py) against closed forms, mistakes planted in it that
have to show, and the serving loop's plain sampled steps against a fake engine.  No GPU."""
import importlib.machinery
import importlib.util
import inspect
import os
import sys

import numpy as np
import pytest

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, os.path.join(ROOT, "oracle"))
import kezilix_oracle as K  # noqa: E402

CFG = {"architecture": "Kezilix", "vocab": 90, "width": 40, "norm": {"eps": 1e-5},
       "layers": [{"type": "retention", "mlp": None, "mixer": {"heads": 3, "dim": 12, "vdim": 20, "rot": {"dims": 8, "base": 900.0}, "decay": [0.9, 0.99, 1.0]}},
                  {"type": "latent_attention", "mlp": {"kind": "dense", "ff": 50},
                   "mixer": {"heads": 2, "dim": 10, "rot_dim": 12, "vdim": 14, "kv_rank": 18, "scale": 0.3,
                             "rot": {"dims": 12, "base": 500.0, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}}}}],
       "loop": {"start": 0, "stop": 2, "times": 2}}


def test_rotation_is_a_turn_of_each_pair():
    rot = {"dims": 6, "base": 100.0}
    x = np.random.default_rng(0).standard_normal((5, 2, 9))
    for inter, pairs in ((True, [(0, 1), (2, 3), (4, 5)]), (False, [(0, 3), (1, 4), (2, 5)])):
        y = K.rotate(x, np.arange(5), rot, inter)
        np.testing.assert_array_equal(y[..., 6:], x[..., 6:])
        np.testing.assert_array_equal(y[0], x[0])
        for i, (u, v) in enumerate(pairs):
            z = (x[..., u] + 1j * x[..., v]) * np.exp(1j * np.arange(5) * 100.0 ** (-i / 3))[:, None]
            np.testing.assert_allclose(y[..., u] + 1j * y[..., v], z, atol=1e-12)


def test_interpolated_frequencies():
    plain, one = K.rotary_frequencies({"dims": 32, "base": 10000.0})
    f, amp = K.rotary_frequencies({"dims": 32, "base": 10000.0, "scaling": {"factor": 8.0, "original": 512, "fast": 32.0, "slow": 1.0}})
    assert one == 1.0 and abs(amp - (1 + 0.1 * np.log(8.0))) < 1e-12
    np.testing.assert_allclose(f[:2], plain[:2])                             # many turns: as they are
    np.testing.assert_allclose(f[-3:], plain[-3:] / 8.0)                     # less than a turn: stretched
    assert (np.diff(f / plain) <= 1e-12).all()


def test_retention_equals_its_sum_form():
    rng = np.random.default_rng(1)
    q, k, v = rng.standard_normal((9, 2, 4)), rng.standard_normal((9, 2, 4)), rng.standard_normal((9, 2, 3))
    dec = np.array([0.8, 1.0])
    o = K.retention_core(q, k, v, dec)
    for t in range(9):
        for h in range(2):
            want = sum(dec[h] ** (t - j) * (q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1))
            np.testing.assert_allclose(o[t, h], want, atol=1e-12)


def test_sink_only_scales_the_attention_output():
    mx = CFG["layers"][1]["mixer"]
    W = K.random_weights(CFG, 5)
    w = {k[len("l1.mix."):]: v.astype(np.float64) for k, v in W.items() if k.startswith("l1.mix.")}
    h = np.random.default_rng(2).standard_normal((7, 40))
    full = K.latent_attention(h, dict(w, sink=np.full(2, -1e9)), mx, 1e-5)
    first = K.latent_attention(h[:1], w, mx, 1e-5)
    q = (h[:1] @ w["q"].T).reshape(2, 22)
    dkv = h[:1] @ w["dkv"].T
    c = K.rms_norm(dkv[:, :18], w["dkv.norm"], 1e-5)
    s = np.array([q[n, :10] @ (w["uk"][n * 10:n * 10 + 10] @ c[0]) + (q[n, 10:] @ dkv[0, 18:]) * (0.1 * np.log(4.0) + 1.0) ** 2 for n in range(2)]) * 0.3
    share = np.exp(s) / (np.exp(s) + np.exp(w["sink"]))
    want = (w["uv"] @ c[0] * np.repeat(share, 14)) @ w["o"].T
    np.testing.assert_allclose(first[0], want, atol=1e-10)
    assert np.isfinite(full).all()


def test_prefix_property_and_loop_runs():
    W = K.random_weights(CFG, 6)
    toks = np.random.default_rng(3).integers(0, 90, 30).tolist()
    trace = []
    a = K.forward(CFG, W, toks, trace=trace)
    np.testing.assert_allclose(K.forward(CFG, W, toks[:11]), a[:11], atol=1e-10)
    assert K.runs(CFG) == [(0, 0), (1, 0), (0, 1), (1, 1)] and len(trace) == 4
    assert K.runs(dict(CFG, loop=None)) == [(0, None), (1, None)]


@pytest.mark.parametrize("mistake", ["sink", "yarn", "amplitude", "embedding_add", "step", "decay", "pairing", "scale"])
def test_planted_mistakes_show(mistake, monkeypatch):
    """What the GPU tests compare against moves by far more than their 32-bit tolerance when a mechanism is wrong."""
    import copy
    W = K.random_weights(CFG, 7)
    toks = np.random.default_rng(4).integers(0, 90, 40).tolist()
    want = K.forward(CFG, W, toks)
    cfg, W2 = copy.deepcopy(CFG), dict(W)
    mx = cfg["layers"][1]["mixer"]
    if mistake == "sink":
        W2["l1.mix.sink"] = np.full(2, -1e9)
    elif mistake == "yarn":
        del mx["rot"]["scaling"]
    elif mistake == "amplitude":
        f = K.rotary_frequencies
        monkeypatch.setattr(K, "rotary_frequencies", lambda rot, dt=np.float64: (f(rot, dt)[0], 1.0))
    elif mistake == "embedding_add":
        ns = dict(vars(K))
        src = inspect.getsource(K.forward)
        exec(src.replace("x = x + emb", "pass"), ns)
        assert "x = x + emb" in src
        monkeypatch.setattr(K, "forward", ns["forward"])
    elif mistake == "step":
        W2["loop.step"] = W["loop.step"][::-1]
    elif mistake == "decay":
        cfg["layers"][0]["mixer"]["decay"] = [0.9, 0.99, 0.999]
    elif mistake == "pairing":
        r = K.rotate
        monkeypatch.setattr(K, "rotate", lambda x, pos, rot, inter: r(x, pos, rot, not inter))
    elif mistake == "scale":
        mx["scale"] *= (0.1 * np.log(4.0) + 1.0) ** 2
    d = K.forward(cfg, W2, toks) - want
    assert np.sqrt((d ** 2).mean()) > 1e-3 * np.sqrt((want ** 2).mean())


class StepEngine:
    """A fake engine with plain steps only: token = floor(100 u), or 0 for greedy steps."""
    k, max_ctx = 0, 64

    def __init__(self, n):
        self.n_seqs, self.out, self.used = n, [[] for _ in range(n)], []

    def reset(self, s):
        self.out[s] = []

    def prefill_sampled(self, s, tokens, u, **kw):
        self.out[s] = [int(100 * u)]

    def sampled_step(self, u, **kw):
        assert len(u) == self.n_seqs and kw == {"temp": 0.5}
        self.used.append(list(u))
        self.out = [[int(100 * x)] for x in u]

    def read_output(self):
        return self.out

    def set_active(self, n):
        pass

    def swap(self, a, b):
        self.out[a], self.out[b] = self.out[b], self.out[a]


@pytest.mark.parametrize("loop", ["run", "run_compact"])
def test_plain_sampled_steps_take_one_draw_each(qb, loop):
    class Rng:
        def __init__(self, rid):
            self.v = iter([(rid * 10 + i) / 100 for i in range(10)])

        def random(self):
            return next(self.v)
    eng = StepEngine(2)
    reqs = [qb.serve.Request(i, [1, 2], n) for i, n in enumerate((3, 5, 2))]
    getattr(qb.serve, loop)(eng, reqs, speculative=False, sampling={"temp": 0.5}, rng_of=lambda r: Rng(r.rid))
    for r, n in zip(reqs, (3, 5, 2)):
        assert [round(t / 1) for t in r.tokens] == [int(100 * ((r.rid * 10 + i) / 100)) for i in range(n)]


def test_trace_slots():
    loader = importlib.machinery.SourceFileLoader("trace_run", os.path.join(ROOT, "bin", "trace_run"))
    spec = importlib.util.spec_from_loader("trace_run", loader)
    mod = importlib.util.module_from_spec(spec)
    loader.exec_module(mod)

    class B:
        n_seqs, resets = 2, []

        def reset(self, s):
            self.resets.append(s)
    r = mod.Requests(B())
    assert (r.of("a"), r.of("b"), r.of("a")) == (0, 1, 0)
    with pytest.raises(RuntimeError):
        r.of("c")
    r.end("a")
    r.end("nobody")
    assert r.of("c") == 0
