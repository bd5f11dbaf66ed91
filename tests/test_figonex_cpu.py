"""The plain restatement of the Figonex design (oracle/figonex_oracle.py) against closed forms, and mistakes planted in it that
have to show in the logits.  No GPU."""
import copy
import os
import sys

import numpy as np
import pytest

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, os.path.join(ROOT, "oracle"))
import figonex_oracle as F  # noqa: E402

ATT = {"type": "attention", "mlp": {"kind": "dense", "ff": 44},
       "mixer": {"heads": 6, "kv_heads": 2, "dim": 14, "vdim": 14, "scale": 0.4, "rot": {"dims": 6, "base": 300.0, "scaling": {"factor": 3.0}}}}
LIG = {"type": "lightning", "mlp": None, "mixer": {"heads": 3, "dim": 10, "vdim": 12, "decay": [0.7, 0.95, 0.999]}}
MLS = {"type": "mlstm", "mlp": {"kind": "dense", "ff": 30}, "mixer": {"heads": 2, "dim": 8, "vdim": 18, "gate_cap": 9.0}}
CFG = {"architecture": "Figonex", "vocab": 80, "width": 36, "norm": {"eps": 1e-5}, "embedding": {"scale": 5.0},
       "layers": [LIG, ATT, MLS, dict(ATT, weights_of=1), dict(MLS, weights_of=2)]}


def mixer_weights(i, seed=5):
    p = "l%d.mix." % i
    return {k[len(p):]: v.astype(np.float64) for k, v in F.random_weights(CFG, seed).items() if k.startswith(p)}


def test_rotation_turns_pairs_at_the_stretched_frequency():
    rot = {"dims": 6, "base": 100.0, "scaling": {"factor": 4.0}}
    x = np.random.default_rng(0).standard_normal((5, 2, 9))
    y = F.rotate(x, np.arange(5), rot)
    np.testing.assert_array_equal(y[..., 6:], x[..., 6:])
    for i in range(3):
        z = (x[..., i] + 1j * x[..., i + 3]) * np.exp(1j * np.arange(5) * 100.0 ** (-i / 3) / 4)[:, None]
        np.testing.assert_allclose(y[..., i] + 1j * y[..., i + 3], z, atol=1e-12)


def test_layer_norm_is_centred():
    x = np.random.default_rng(1).standard_normal((3, 50)) * 4 + 7
    y = F.layer_norm(x, np.ones(50), 0.0)
    np.testing.assert_allclose(y.mean(-1), 0, atol=1e-12)
    np.testing.assert_allclose(y.std(-1), 1, atol=1e-12)
    np.testing.assert_allclose(F.layer_norm(x + 3, np.ones(50), 1e-5), F.layer_norm(x, np.ones(50), 1e-5), atol=1e-10)


def test_first_token_attends_itself_and_the_sink():
    w, mx = mixer_weights(1), ATT["mixer"]
    h = np.random.default_rng(2).standard_normal((1, 36))
    raw, q = (h @ w["k"].T).reshape(2, 14), (h @ w["q"].T).reshape(6, 14)
    want = []
    for n in range(6):
        k = raw[n // 3]
        s = 0.4 * (F.rms(q[n], 1e-5) * w["q.norm"]) @ (F.rms(k, 1e-5) * w["k.norm"])
        want.append(k * np.exp(s) / (1 + np.exp(s)) / (1 + np.exp(-(h[0] @ w["g"][n]))))
    np.testing.assert_allclose(F.attention(h, w, mx, 1e-5)[0], np.concatenate(want) @ w["o"].T, atol=1e-10)


def test_lightning_equals_its_sum_form():
    rng = np.random.default_rng(3)
    q, k, v = rng.standard_normal((9, 2, 4)), rng.standard_normal((9, 2, 4)), rng.standard_normal((9, 2, 3))
    o = F.lightning_core(q, k, v, [0.8, 0.99])
    for t in range(9):
        for h, d in enumerate((0.8, 0.99)):
            np.testing.assert_allclose(o[t, h], sum(d ** (t - j) * (q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1)), atol=1e-12)


def test_mlstm_equals_its_unstabilised_form():
    """Without the running maximum: plain exponentials, the 1e-6 scaled back by exp(m)."""
    rng = np.random.default_rng(4)
    T, H = 12, 2
    q, k, v = rng.standard_normal((T, H, 4)), rng.standard_normal((T, H, 4)), rng.standard_normal((T, H, 3))
    i, f = rng.standard_normal((T, H)) * 2, F.log_sigmoid(rng.standard_normal((T, H)) * 3)
    o = F.mlstm_core(q, k, v, i, f)
    b = f.cumsum(0)
    for t in range(T):
        for h in range(H):
            w = np.exp(b[t, h] - b[:t + 1, h] + i[:t + 1, h])
            num = sum(w[j] * (q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1))
            nq = sum(w[j] * (q[t, h] @ k[j, h]) for j in range(t + 1))
            m = max(b[t, h], (b[t, h] - b[:t + 1, h] + i[:t + 1, h]).max())          # the maximum starts at 0
            np.testing.assert_allclose(o[t, h], num / (max(abs(nq), 1) + 1e-6 * np.exp(m)), rtol=1e-9, atol=1e-12)


def test_log_sigmoid_in_both_tails():
    z = np.array([-40.0, -3.0, 0.0, 3.0, 40.0])
    np.testing.assert_allclose(F.log_sigmoid(z), [-40.0, np.log(1 / (1 + np.exp(3.0))), np.log(0.5), -np.log1p(np.exp(-3.0)), -np.exp(-40.0)], rtol=1e-12)


def test_prefix_property_and_shared_weights():
    W = F.random_weights(CFG, 6)
    assert not any(k.startswith(("l3.", "l4.")) for k in W)
    toks = np.random.default_rng(5).integers(0, 80, 30).tolist()
    trace = []
    a = F.forward(CFG, W, toks, trace=trace)
    np.testing.assert_allclose(F.forward(CFG, W, toks[:11]), a[:11], atol=1e-10)
    assert len(trace) == 5
    own = dict(CFG, layers=[dict(L, weights_of=None) for L in CFG["layers"]])
    W2 = dict(W, **{k.replace("l%d." % j, "l%d." % i): v for i, j in ((3, 1), (4, 2)) for k, v in W.items() if k.startswith("l%d." % j)})
    np.testing.assert_allclose(F.forward(own, W2, toks), a, atol=1e-12)
    assert [F.weights_of(CFG, i) for i in range(5)] == [0, 1, 2, 1, 2]


MISTAKES = ["no_sink", "value_normed", "no_key_norm", "no_query_norm", "gate", "scaling", "scale", "pairs", "rms_for_layer_norm", "layer_scale", "embed_scale",
            "decay", "lightning_silu", "norm_per_head", "mlstm_cap", "mlstm_normaliser", "mlstm_query_scale", "forget_raw", "weights_of"]


@pytest.mark.parametrize("mistake", MISTAKES)
def test_planted_mistakes_show(mistake, monkeypatch):
    """What the GPU tests compare against moves by far more than their 32-bit tolerance when a mechanism is wrong."""
    W, cfg = F.random_weights(CFG, 7), copy.deepcopy(CFG)
    if mistake.startswith("mlstm_"):
        # a head's output is divided by its root mean square: its size shows beside a large eps only
        cfg["norm"]["eps"] = 0.5
        cfg["layers"][2]["mixer"]["gate_cap"] = cfg["layers"][4]["mixer"]["gate_cap"] = 15.0
    toks = np.random.default_rng(6).integers(0, 80, 40).tolist()
    want = F.forward(cfg, W, toks)
    W2 = dict(W)
    att = [L["mixer"] for L in cfg["layers"] if L["type"] == "attention"]

    def rewrite(name, old, new):
        import inspect
        src = inspect.getsource(getattr(F, name))
        assert old in src
        ns = dict(vars(F))
        exec(src.replace(old, new), ns)
        monkeypatch.setattr(F, name, ns[name])
        for t, f in list(F.MIXERS.items()):
            if f.__name__ == name:
                monkeypatch.setitem(F.MIXERS, t, ns[name])
    if mistake == "no_sink":
        rewrite("attention", "+ np.exp(-m)", "")
    elif mistake == "value_normed":
        rewrite("attention", "@ raw[:, g]", "@ rms(raw[:, g], eps)")
    elif mistake == "no_key_norm":
        rewrite("attention", 'rms_norm(raw, w["k.norm"], eps)', 'raw * w["k.norm"]')
    elif mistake == "no_query_norm":
        rewrite("attention", 'rms_norm((h @ w["q"].T).reshape(T, H, d), w["q.norm"], eps)', '(h @ w["q"].T).reshape(T, H, d) * w["q.norm"]')
    elif mistake == "gate":
        rewrite("attention", 'sigmoid(h @ w["g"].T)[:, :, None]', "0.5")
    elif mistake == "scaling":
        for m in att:
            m["rot"].pop("scaling", None)
    elif mistake == "scale":
        for m in att:
            m["scale"] = 14 ** -0.5
    elif mistake == "pairs":
        r = F.rotate
        perm = [0, 2, 4, 1, 3, 5] + list(range(6, 14))
        monkeypatch.setitem(F.MIXERS, "attention", F.attention)
        monkeypatch.setattr(F, "rotate", lambda x, p, rot: r(x[..., perm], p, rot)[..., np.argsort(perm)])
    elif mistake == "rms_for_layer_norm":
        monkeypatch.setattr(F, "layer_norm", lambda x, w, eps: F.rms_norm(x, w, eps))
    elif mistake == "layer_scale":
        W2["l1.ls2"] = np.ones_like(W["l1.ls2"])
    elif mistake == "embed_scale":
        cfg["embedding"]["scale"] = 6.0
    elif mistake == "decay":
        cfg["layers"][0]["mixer"]["decay"] = [0.7, 0.95, 0.99]
    elif mistake == "lightning_silu":
        rewrite("lightning", 'v = silu(h @ w["v"].T)', 'v = (h @ w["v"].T)')
    elif mistake == "norm_per_head":
        rewrite("lightning", 'rms_norm(o, w["norm"], eps)', 'rms(o.reshape(T, H, vd), eps).reshape(T, -1) * w["norm"]')
    elif mistake == "mlstm_cap":
        monkeypatch.setattr(F, "soft_cap", lambda z, cap: z)
    elif mistake == "mlstm_normaliser":
        rewrite("mlstm_core", "np.abs((n * q[t]).sum(-1))", "(n * q[t]).sum(-1)")
    elif mistake == "mlstm_query_scale":
        rewrite("mlstm", "* dt(d ** -0.5)", "")
    elif mistake == "forget_raw":
        monkeypatch.setattr(F, "log_sigmoid", lambda z: np.minimum(z, 0))
    elif mistake == "weights_of":
        cfg["layers"][3]["weights_of"] = None
        W2.update({k.replace("l1.", "l3."): v[..., ::-1] for k, v in W.items() if k.startswith("l1.")})
    d = F.forward(cfg, W2, toks) - want
    assert np.sqrt((d ** 2).mean()) > 1e-3 * np.sqrt((want ** 2).mean())
