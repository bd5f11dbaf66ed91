"""Plain, slow restatement of the Figonex decoder in numpy: one function per mechanism, whole sequences, no cache.

Test infrastructure only: it shares no code with the product path.  `dt` is the number type of everything (float64 unless
a test asks for float32).  Weights are a dict {tensor name: array}, the configuration the parsed config.json.
`rnd` is applied to what enters a matrix product from the right of a weight (identity unless a test asks what rounding those
operands does to a row).
"""
import numpy as np

from kezilix_oracle import bf16_round, rms, rms_norm, silu, write_model  # noqa: F401  (plain helpers, shared between the oracles)


def exact(a):
    return a


def to_bf16(a):
    return bf16_round(a.astype(np.float32)).astype(a.dtype)


def sigmoid(z):
    return 1 / (1 + np.exp(-z))


def layer_norm(x, w, eps):
    """Mean off, divided by the root of the mean squared deviation plus eps, times w."""
    d = x - x.mean(-1, keepdims=True)
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + x.dtype.type(eps)) * w


def frequencies(rot, dt=np.float64):
    """Turn per position of each pair; a scaling entry stretches every pair alike."""
    n = int(rot["dims"])
    f = float(rot["base"]) ** (-2.0 * np.arange(n // 2) / n)
    if rot.get("scaling"):
        f = f / float(rot["scaling"]["factor"])
    return f.astype(dt)


def rotate(x, pos, rot):
    """x [T][heads][d]: element i and element i + dims / 2 of the first rot.dims turn together, the rest passes."""
    dt, n = x.dtype.type, int(rot["dims"])
    a = (pos.astype(dt)[:, None] * frequencies(rot, dt)[None, :])[:, None, :]
    u, v = x[..., :n // 2], x[..., n // 2:n]
    return np.concatenate([u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a), x[..., n:]], -1)


def attention(h, w, mx, eps, pos=None, rnd=exact):
    """Grouped-query attention whose values are the raw key projections, with a zero-score sink and one gate per head."""
    dt = h.dtype.type
    T, H, G, d = len(h), mx["heads"], mx["kv_heads"], mx["dim"]
    pos = np.arange(T) if pos is None else pos
    raw = (h @ w["k"].T).reshape(T, G, d)
    q = rnd(rotate(rms_norm((h @ w["q"].T).reshape(T, H, d), w["q.norm"], eps), pos, mx["rot"]))
    k = rnd(rotate(rms_norm(raw, w["k.norm"], eps), pos, mx["rot"]))
    raw = rnd(raw)
    o = np.zeros((T, H, d), h.dtype)
    for n in range(H):
        g = n // (H // G)
        s = (q[:, n] @ k[:, g].T) * dt(mx["scale"])
        s[~np.tri(T, dtype=bool)] = -np.inf
        m = np.maximum(s.max(-1), 0)
        e = np.exp(s - m[:, None])
        o[:, n] = (e / (e.sum(-1) + np.exp(-m))[:, None]) @ raw[:, g]
    o = o * sigmoid(h @ w["g"].T)[:, :, None]
    return rnd(o.reshape(T, H * d)) @ w["o"].T


def lightning_core(q, k, v, decay):
    """q, k [T][heads][dim], v [T][heads][vdim] -> o, walking the state token by token."""
    T, H, d = q.shape
    S = np.zeros((H, d, v.shape[-1]), q.dtype)
    dec = np.asarray(decay, q.dtype)[:, None, None]
    o = np.zeros(v.shape, q.dtype)
    for t in range(T):
        S = dec * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    return o


def lightning(h, w, mx, eps, pos=None, rnd=exact):
    T, H, d, vd = len(h), mx["heads"], mx["dim"], mx["vdim"]
    q, k = (silu(h @ w[n].T).reshape(T, H, d) for n in ("q", "k"))
    v = silu(h @ w["v"].T).reshape(T, H, vd)
    o = lightning_core(q, k, v, mx["decay"]).reshape(T, H * vd)
    return rnd(rms_norm(o, w["norm"], eps) * sigmoid(h @ w["g"].T)) @ w["o"].T


def log_sigmoid(z):
    return np.where(z > 0, -np.log1p(np.exp(-np.abs(z))), z - np.log1p(np.exp(-np.abs(z))))


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


def mlstm_core(q, k, v, i, f):
    """q, k [T][heads][dim] (q already scaled), v [T][heads][vdim], log gates i, f [T][heads] -> o, token by token."""
    T, H, d = q.shape
    S, n, m = np.zeros((H, d, v.shape[-1]), q.dtype), np.zeros((H, d), q.dtype), np.zeros(H, q.dtype)
    o = np.zeros(v.shape, q.dtype)
    for t in range(T):
        nm = np.maximum(f[t] + m, i[t])
        keep, add = np.exp(f[t] + m - nm), np.exp(i[t] - nm)
        m = nm
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        den = np.maximum(np.abs((n * q[t]).sum(-1)), np.exp(-m)) + q.dtype.type(1e-6)
        o[t] = np.einsum("hdv,hd->hv", S, q[t]) / den[:, None]
    return o


def mlstm_gates(h, w, cap):
    """(log input gate, log forget gate), [T][heads] each."""
    return soft_cap(h @ w["i"].T + w["i.b"], cap), log_sigmoid(soft_cap(h @ w["f"].T + w["f.b"], cap))


def mlstm(h, w, mx, eps, pos=None, rnd=exact):
    dt = h.dtype.type
    T, H, d, vd = len(h), mx["heads"], mx["dim"], mx["vdim"]
    q = (h @ w["q"].T).reshape(T, H, d) * dt(d ** -0.5)
    k = (h @ w["k"].T).reshape(T, H, d)
    v = (h @ w["v"].T).reshape(T, H, vd)
    i, f = mlstm_gates(h, w, dt(mx["gate_cap"]))
    o = rms(mlstm_core(q, k, v, i, f), eps).reshape(T, H * vd)
    return rnd(o * w["norm"] * sigmoid(h @ w["g"].T)) @ w["o"].T


MIXERS = {"attention": attention, "lightning": lightning, "mlstm": mlstm}


def dense_ff(h, w, rnd=exact):
    return rnd(silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def weights_of(cfg, i):
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg, weights, tokens, dt=np.float64, trace=None, rnd=exact):
    """Logits [T][vocab] of one sequence; trace (a list) receives the residual stream after every layer."""
    W = {k: np.asarray(v, dt) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    sub = lambda p: {k[len(p):]: v for k, v in W.items() if k.startswith(p)}
    x = W["embed"][np.asarray(tokens)] * dt(cfg["embedding"]["scale"])
    for i, L in enumerate(cfg["layers"]):
        p = "l%d." % weights_of(cfg, i)
        x = x + layer_norm(MIXERS[L["type"]](rnd(x), sub(p + "mix."), L["mixer"], eps, rnd=rnd), W[p + "norm1"], eps) * W[p + "ls1"]
        if L.get("mlp"):
            x = x + layer_norm(dense_ff(rnd(x), sub(p + "mlp."), rnd), W[p + "norm2"], eps) * W[p + "ls2"]
        if trace is not None:
            trace.append(x.copy())
    return rnd(layer_norm(x, W["final.norm"], eps)) @ W["head"].T


def tensor_shapes(cfg):
    """{name: shape} of every tensor of a configuration, in file order."""
    D = cfg["width"]
    out = {"embed": (cfg["vocab"], D)}
    for i, L in enumerate(cfg["layers"]):
        if L.get("weights_of") is not None:
            continue
        p, m = "l%d." % i, L["mixer"]
        q, H, d, vd = p + "mix.", m["heads"], m["dim"], m["vdim"]
        out[p + "norm1"] = out[p + "ls1"] = (D,)
        if L["type"] == "attention":
            G = m["kv_heads"]
            out.update({q + "q": (H * d, D), q + "k": (G * d, D), q + "q.norm": (d,), q + "k.norm": (d,), q + "g": (H, D)})
        else:
            out.update({q + "q": (H * d, D), q + "k": (H * d, D), q + "v": (H * vd, D), q + "g": (H * vd, D), q + "norm": (H * vd,)})
            if L["type"] == "mlstm":
                out.update({q + "i": (H, D), q + "i.b": (H,), q + "f": (H, D), q + "f.b": (H,)})
        out[q + "o"] = (D, H * vd)
        if L.get("mlp"):
            F = L["mlp"]["ff"]
            out.update({p + "norm2": (D,), p + "ls2": (D,), p + "mlp.gate": (F, D), p + "mlp.up": (F, D), p + "mlp.down": (D, F)})
    out["final.norm"] = (D,)
    out["head"] = (cfg["vocab"], D)
    return out


def random_weights(cfg, seed, gain=1.0):
    """Seeded weights on the bfloat16 grid, float32 arrays: matrices N(0, gain / columns), gains and layer scales around 1,
    biases of the gates spread so that some heads forget quickly and some keep."""
    rng = np.random.default_rng(seed)
    W = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.split(".")[-1]
        if last in ("norm", "norm1", "norm2"):
            a = 1.0 + 0.2 * rng.standard_normal(shape)
        elif last in ("ls1", "ls2"):
            a = 0.6 + 0.2 * rng.standard_normal(shape)
        elif name.endswith(".f.b"):
            a = rng.uniform(-1.0, 5.0, shape)
        elif name.endswith(".i.b"):
            a = rng.standard_normal(shape)
        elif name == "embed":
            a = rng.standard_normal(shape) / float(cfg["embedding"]["scale"])
        else:
            a = rng.standard_normal(shape) * np.sqrt(gain / shape[1])
        W[name] = bf16_round(a.astype(np.float32))
    return W
