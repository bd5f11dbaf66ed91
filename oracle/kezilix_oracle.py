"""Plain, slow restatement of the Kezilix decoder in numpy: one function per mechanism, whole sequences, no cache.

Test infrastructure only: it shares no code with the product path.  `dt` is the number type of everything (float64 unless
a test asks for float32).  Weights are a dict {tensor name: array}, the configuration the parsed config.json.
"""
import numpy as np


def rms(x, eps):
    """Rows divided by their root mean square, eps inside the root."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + x.dtype.type(eps))


def rms_norm(x, w, eps):
    return rms(x, eps) * w


def silu(z):
    return z / (1 + np.exp(-z))


def rotary_frequencies(rot, dt=np.float64):
    """(frequencies [dims / 2], amplitude of cos and sin) of a rotation entry {base, dims[, scaling]}; the interpolation of
    `scaling` divides low frequencies by `factor`, keeps high ones, and blends between the two pair indices at which a
    dimension makes `fast` and `slow` turns over `original` positions."""
    n, base = int(rot["dims"]), float(rot["base"])
    i = np.arange(n // 2, dtype=np.float64)
    f = base ** (-2.0 * i / n)
    s = rot.get("scaling")
    if not s:
        return f.astype(dt), dt(1.0)
    turns = lambda t: n * np.log(s["original"] / (2 * np.pi * t)) / (2 * np.log(base))
    lo = max(np.floor(turns(s["fast"])), 0)
    hi = min(np.ceil(turns(s["slow"])), n - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0, 1)
    return (f / s["factor"] * ramp + f * (1 - ramp)).astype(dt), dt(0.1 * np.log(s["factor"]) + 1.0)


def rotate(x, pos, rot, interleaved):
    """x [T][heads][d] at positions pos [T]: the first rot.dims of d rotated in pairs (2i, 2i+1) or (i, i + dims/2)."""
    dt = x.dtype.type
    f, amp = rotary_frequencies(rot, dt)
    n = 2 * len(f)
    a = pos.astype(dt)[:, None] * f[None, :]
    cos, sin = (np.cos(a) * amp)[:, None, :], (np.sin(a) * amp)[:, None, :]
    iu = np.arange(0, n, 2) if interleaved else np.arange(n // 2)
    iv = iu + 1 if interleaved else iu + n // 2
    u, v = x[..., iu], x[..., iv]
    y = x.copy()
    y[..., iu] = u * cos - v * sin
    y[..., iv] = v * cos + u * sin
    return y


def latent_attention(h, w, mx, eps, pos=None):
    """h [T][width] -> [T][width].  w: the mixer's tensors by short name."""
    dt = h.dtype.type
    T, H, dim, rd, vd, rank = len(h), mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    pos = np.arange(T) if pos is None else pos
    q = (h @ w["q"].T).reshape(T, H, dim + rd)
    qn, qr = q[..., :dim], rotate(q[..., dim:], pos, mx["rot"], True)
    dkv = h @ w["dkv"].T
    c = rms_norm(dkv[:, :rank], w["dkv.norm"], eps)
    kr = rotate(dkv[:, None, rank:], pos, mx["rot"], True)[:, 0]
    kn = (c @ w["uk"].T).reshape(T, H, dim)
    v = (c @ w["uv"].T).reshape(T, H, vd)
    o = np.zeros((T, H, vd), h.dtype)
    for n in range(H):
        s = (qn[:, n] @ kn[:, n].T + qr[:, n] @ kr.T) * dt(mx["scale"])
        s[~np.tri(T, dtype=bool)] = -np.inf
        m = np.maximum(s.max(-1), w["sink"][n])
        e = np.exp(s - m[:, None])
        den = e.sum(-1) + np.exp(w["sink"][n] - m)
        o[:, n] = (e / den[:, None]) @ v[:, n]
    return o.reshape(T, H * vd) @ w["o"].T


def retention_core(q, k, v, decay):
    """q, k [T][heads][dim] (k already scaled), v [T][heads][vdim] -> o, walking the state token by token."""
    T, H, d = q.shape
    S = np.zeros((H, d, v.shape[-1]), q.dtype)
    o = np.zeros(v.shape, q.dtype)
    dec = np.asarray(decay, q.dtype)[:, None, None]
    for t in range(T):
        S = S * dec + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    return o


def retention(h, w, mx, eps, pos=None):
    dt = h.dtype.type
    T, H, dim, vd = len(h), mx["heads"], mx["dim"], mx["vdim"]
    pos = np.arange(T) if pos is None else pos
    q = rotate((h @ w["q"].T).reshape(T, H, dim), pos, mx["rot"], False)
    k = rotate((h @ w["k"].T).reshape(T, H, dim), pos, mx["rot"], False) * dt(dim ** -0.5)
    v = (h @ w["v"].T).reshape(T, H, vd)
    o = rms(retention_core(q, k, v, mx["decay"]), eps).reshape(T, H * vd)
    return (o * silu(h @ w["g"].T)) @ w["o"].T


MIXERS = {"latent_attention": latent_attention, "retention": retention}


def dense_ff(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def runs(cfg):
    """[(layer, pass or None)] in execution order; pass is the pass number of a layer inside the loop."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, None) for i in range(n)]
    a, b = lp["start"], lp["stop"]
    return ([(i, None) for i in range(a)] + [(i, t) for t in range(lp["times"]) for i in range(a, b)]
            + [(i, None) for i in range(b, n)])


def forward(cfg, weights, tokens, dt=np.float64, trace=None):
    """Logits [T][vocab] of one sequence; trace (a list) receives the residual stream after every layer run."""
    W = {k: np.asarray(v, dt) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    sub = lambda p: {k[len(p):]: v for k, v in W.items() if k.startswith(p)}
    x = rms_norm(W["embed"][np.asarray(tokens)], W["embed.norm"], eps)
    emb = x.copy()
    for i, t in runs(cfg):
        L = cfg["layers"][i]
        if t is not None and i == cfg["loop"]["start"]:
            if t > 0:
                x = x + emb
            x = x + W["loop.step"][t]
        x = x + MIXERS[L["type"]](rms_norm(x, W["l%d.norm1" % i], eps), sub("l%d.mix." % i), L["mixer"], eps)
        if L.get("mlp"):
            x = x + dense_ff(rms_norm(x, W["l%d.norm2" % i], eps), sub("l%d.mlp." % i))
        if trace is not None:
            trace.append(x.copy())
    return rms_norm(x, W["final.norm"], eps) @ W["head"].T


def bf16_round(a):
    """float32 values rounded to the nearest bfloat16 (ties to even)."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) & np.uint32(0xFFFF0000)).astype(np.uint32).view(np.float32)


def tensor_shapes(cfg):
    """{name: shape} of every tensor of a configuration, in file order."""
    D, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"]), "embed.norm": (cfg["width"],)}
    if cfg.get("loop"):
        out["loop.step"] = (cfg["loop"]["times"], D)
    for i, L in enumerate(cfg["layers"]):
        p, m = "l%d." % i, L["mixer"]
        out[p + "norm1"] = (D,)
        if L.get("mlp"):
            out[p + "norm2"] = (D,)
        H, vd = m["heads"], m["vdim"]
        if L["type"] == "retention":
            out.update({p + "mix.q": (H * m["dim"], D), p + "mix.k": (H * m["dim"], D), p + "mix.v": (H * vd, D), p + "mix.g": (H * vd, D)})
        else:
            out.update({p + "mix.q": (H * (m["dim"] + m["rot_dim"]), D), p + "mix.dkv": (m["kv_rank"] + m["rot_dim"], D),
                        p + "mix.dkv.norm": (m["kv_rank"],), p + "mix.uk": (H * m["dim"], m["kv_rank"]),
                        p + "mix.uv": (H * vd, m["kv_rank"]), p + "mix.sink": (H,)})
        out[p + "mix.o"] = (D, H * vd)
        if L.get("mlp"):
            F = L["mlp"]["ff"]
            out.update({p + "mlp.gate": (F, D), p + "mlp.up": (F, D), p + "mlp.down": (D, F)})
    out["final.norm"] = (D,)
    out["head"] = (cfg["vocab"], D)
    return out


def random_weights(cfg, seed, gain=1.0):
    """Seeded weights on the bfloat16 grid, float32 arrays: matrices N(0, gain / columns), norm gains around 1."""
    rng = np.random.default_rng(seed)
    W = {}
    for name, shape in tensor_shapes(cfg).items():
        if name.endswith("norm") or name.endswith("norm1") or name.endswith("norm2"):
            a = 1.0 + 0.2 * rng.standard_normal(shape)
        elif name == "loop.step":
            a = 0.3 * rng.standard_normal(shape)
        elif name.endswith(".sink"):
            a = 1.0 + rng.standard_normal(shape)
        elif name == "embed":
            a = rng.standard_normal(shape)
        else:
            a = rng.standard_normal(shape) * np.sqrt(gain / shape[1])
        W[name] = bf16_round(a.astype(np.float32))
    return W


def write_model(path, cfg, weights):
    """Writes config.json and model.safetensors (bfloat16) into the folder `path`."""
    import json
    import os
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, blobs, at = {}, [], 0
    for name, a in weights.items():
        raw = (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype(np.uint16).tobytes()
        head[name] = {"dtype": "BF16", "shape": list(np.shape(a)), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    hj = json.dumps(head).encode()
    hj += b" " * (-len(hj) % 8)
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(len(hj).to_bytes(8, "little") + hj + b"".join(blobs))
