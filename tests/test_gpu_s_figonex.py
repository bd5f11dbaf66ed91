"""The Figonex design (layered models) on the GPU against the plain numpy restatement in oracle/figonex_oracle.py.

Every configuration here is the tests' own: odd head counts, sizes that are no multiples of 16 or 64, rotations over a part
of a head or all of it, layers with and without feed-forward or weights of their own.  32-bit runs are compared tightly,
bfloat16 runs within the rounding of their products.  Where random weights would drown a single key among many, the score
scale is raised so that one key decides the row; where a norm would hide a factor, eps is raised so that it shows."""
import json
import os
import random
import subprocess
import sys

import numpy as np
import pytest

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, os.path.join(ROOT, "oracle"))
sys.path.insert(0, os.path.join(ROOT, "tests"))
import figonex_oracle as F  # noqa: E402
from layered_case import TOL, Case, close_to, distance, in_portions  # noqa: E402


def dense(ff):
    return {"kind": "dense", "ff": ff} if ff else None


def att(heads=6, kv=3, dim=20, rot=12, base=700.0, factor=3.0, scale=0.25, ff=72):
    r = {"dims": rot, "base": base}
    if factor:
        r["scaling"] = {"factor": factor}
    return {"type": "attention", "mlp": dense(ff), "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale, "rot": r}}


def lig(heads=3, dim=24, vdim=40, decay=(0.8, 0.995, 0.95), ff=None):
    return {"type": "lightning", "mlp": dense(ff), "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)[:heads]}}


def mls(heads=3, dim=24, vdim=36, cap=11.0, ff=None):
    return {"type": "mlstm", "mlp": dense(ff), "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def config(layers, width=88, vocab=210, eps=1e-5, scale=6.5):
    return {"architecture": "Figonex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}


def of(layer, i):
    return dict(layer, weights_of=i)


L0, L1, L2, L3 = att(), lig(ff=56), mls(), att(heads=4, kv=1, dim=16, rot=16, factor=None, ff=None)
# (an mLSTM output that nearly cancels is blown up by its norm, rounding included; a larger eps makes such rows rare)
MIXED = config([L0, L1, L2, L3, of(L2, 2), of(L0, 0), of(L1, 1)], eps=1e-2)


@pytest.fixture
def make(qb, ctx, tmp_path):
    made = []

    def f(cfg, **kw):
        made.append(Case(F, qb, ctx, tmp_path / ("m%d" % len(made)), cfg, **kw))
        return made[-1]
    yield f
    for c in made:
        c.close()


# ---- each mechanism alone --------------------------------------------------------------------------------------------------
ALONE = {
    "attention": config([att(ff=None)]),
    "attention_whole_head_rotated": config([att(heads=4, kv=2, dim=32, rot=32, ff=None)]),
    "attention_two_rotated": config([att(heads=5, kv=5, dim=18, rot=2, ff=None)]),
    "attention_one_kv_head": config([att(heads=7, kv=1, dim=48, rot=8, scale=0.15, ff=None)]),
    "attention_one_head": config([att(heads=1, kv=1, dim=16, rot=4, factor=None, ff=None)]),
    "attention_plain_rotation": config([att(factor=None, ff=None)]),
    "attention_wide_heads": config([att(heads=4, kv=2, dim=136, rot=40, scale=0.1, ff=None)]),
    "attention_real_heads": config([att(heads=8, kv=2, dim=128, rot=32, scale=0.09, ff=40)], width=160),
    "lightning": config([lig()]),
    "lightning_one_head": config([lig(heads=1, dim=16, vdim=16, decay=(0.99,))]),
    "lightning_odd": config([lig(heads=2, dim=10, vdim=70, decay=(1.0, 0.5))]),
    "lightning_wide": config([lig(heads=2, dim=72, vdim=136, decay=(0.9, 0.999))]),
    "lightning_large_eps": config([lig()], eps=3.0),
    "mlstm": config([mls()]),
    "mlstm_one_head": config([mls(heads=1, dim=16, vdim=16, cap=4.0)]),
    "mlstm_odd": config([mls(heads=5, dim=9, vdim=35)]),
    "mlstm_wide": config([mls(heads=2, dim=72, vdim=136)]),
    "mlstm_large_eps": config([mls()], eps=0.5),
    "mlstm_small_cap": config([mls(cap=0.7)], eps=0.5),
    "feed_forward": config([lig(ff=40), mls(ff=100)]),
    "shared_weights": config([lig(ff=24), of(lig(ff=24), 0), att(), of(att(), 2), of(lig(ff=24), 1)]),
    "weights_of_a_later_layer": config([of(mls(), 2), lig(), mls()]),
    "odd_width": config([att(heads=3, kv=3, dim=22, rot=10, ff=33), mls(heads=3, dim=18, vdim=17, ff=50), lig(heads=1, dim=7, vdim=5, decay=(0.9,))], width=67, vocab=101),
    "mixed": MIXED,
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ALONE))
def test_mechanism_alone(make, name, dtype):
    c = make(ALONE[name])
    b = c.batch(dtype)
    for n in (1, 2, 65, 150):
        toks, trace = c.tokens(n), []
        slack, layer_slack = c.slack(toks, trace)
        want = c.want(toks)
        b.reset(0)
        b.layer_trace(True)
        got = b.score(0, toks, range(n))
        layers = b.layer_trace_read()
        for i, w in enumerate(trace):
            close_to(layers[i], w, dtype, "%s: residual after layer %d of %d tokens" % (name, i, n), layer_slack[i])
        close_to(got, want, dtype, name, slack)
    b.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("layer", [att(heads=2, kv=1, dim=264, rot=80, scale=0.05, ff=None),
                                   att(heads=2, kv=2, dim=520, rot=8, scale=0.05, ff=None),            # values too wide for the tiled form
                                   lig(heads=2, dim=136, vdim=40, decay=(0.99, 0.8)), lig(heads=1, dim=250, vdim=33, decay=(0.99,)),
                                   lig(heads=1, dim=300, vdim=300, decay=(0.99,)),                      # state too large for a chunk's tiles
                                   mls(heads=2, dim=136, vdim=40), mls(heads=1, dim=255, vdim=70), mls(heads=1, dim=300, vdim=290)])
def test_sizes_beyond_the_usual_tiles(make, layer, dtype):
    c = make(config([layer]))
    b = c.batch(dtype)
    toks = c.tokens(140)
    close_to(in_portions(b, 0, toks, [100, 1, 2, 37]), c.want(toks), dtype, str(layer["mixer"]))
    b.close()


@pytest.mark.parametrize("heads,kv,dim,rot,n_seqs", [(16, 4, 128, 32, 40), (12, 2, 64, 64, 40), (3, 1, 96, 8, 1), (20, 1, 48, 16, 3), (8, 8, 128, 128, 40)])
def test_decode_attention_shapes(make, heads, kv, dim, rot, n_seqs):
    """Decode rows over many keys; a large batch cuts a sequence into few spans of several 128-key tiles, and a raised scale
    lets the running maximum grow from tile to tile."""
    c = make(config([att(heads=heads, kv=kv, dim=dim, rot=rot, scale=4.0 / dim ** 0.5, ff=None)]))
    n = 1300 if n_seqs == 40 else 333
    toks = c.tokens(n + 6)
    want = c.want(toks)[n:]
    b = c.batch("bfloat16", n_seqs=n_seqs, max_ctx=1400, pool_pages=100)
    b.prefill(n_seqs - 1, toks[:n], more=True)
    got = [b.score(n_seqs - 1, [t], [0]) for t in toks[n:n + 3]]
    got.append(b.score(n_seqs - 1, toks[n + 3:], range(3)))
    close_to(np.concatenate(got), want, "bfloat16")
    b.close()


@pytest.mark.parametrize("heads,kv,dim,rot", [(8, 2, 128, 32), (6, 2, 64, 64), (5, 1, 20, 12), (4, 4, 96, 8), (12, 3, 32, 4), (4, 1, 256, 64), (2, 2, 136, 40), (3, 1, 10, 2)])
def test_prompt_attention_shapes(make, heads, kv, dim, rot):
    """Prompt rows in tiles of 128 queries and 128 keys, cut at odd places: part of a tile, tiles across portions; one or two
    buffers of keys, head sizes that are no multiples of 16 or 8; a raised scale lets the running maximum move."""
    c = make(config([att(heads=heads, kv=kv, dim=dim, rot=rot, scale=5.0 / dim ** 0.5, ff=None)], eps=1e-3))
    toks = c.tokens(700)
    want = c.want(toks)
    b = c.batch("bfloat16", max_ctx=704, page_order=1)
    for size in (700, [301, 128, 1, 130]):
        b.reset(0)
        close_to(in_portions(b, 0, toks, size), want, "bfloat16", str(size), c.slack(toks))
    b.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("page", [8, 48])
def test_other_page_sizes(make, page, dtype):
    c = make(config([att(heads=4, kv=2, dim=32, rot=8, scale=0.5), mls()]))
    b = c.batch(dtype, n_seqs=2, page_size=page, pool_pages=40)
    toks = c.tokens(150)
    close_to(in_portions(b, 1, toks, [47, 1, 2, 70]), c.want(toks), dtype)
    b.close()


# ---- gates of the recurrence -------------------------------------------------------------------------------------------------
GATES = {"keeps": (0.0, 14.0), "forgets_at_once": (0.0, -30.0), "large_input": (40.0, 2.0), "small_input": (-40.0, 6.0), "moderate": (1.0, 1.0)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(GATES))
def test_gates_of_the_matrix_memory(make, name, dtype):
    """Biases push the gates to their ends: sums of log forget gates of several hundred inside a block, weights exp(+-15); eps is
    large, so that the size of a head's output shows behind its norm."""
    def edit(W):
        W["l0.mix.i.b"][:], W["l0.mix.f.b"][:] = GATES[name]
        W["l0.mix.i.b"][0], W["l0.mix.f.b"][1] = 0.5, 3.0                     # mixed heads too
    c = make(config([mls(cap=15.0)], eps=0.2), edit=edit)
    b = c.batch(dtype)
    toks = c.tokens(170)
    want = c.want(toks)
    for size in (170, [65, 1, 2, 30], [3]):
        b.reset(0)
        close_to(in_portions(b, 0, toks, size), want, dtype, "%s in portions of %s" % (name, size))
    b.close()


def test_normaliser_counts(make):
    """Small keys: |n . q| stays under its floor and the output is not divided by it."""
    def edit(W):
        W["l0.mix.k"] *= 0.0625
    c = make(config([mls()], eps=0.01), edit=edit)
    toks = c.tokens(100)
    W2 = dict(c.W)
    W2["l0.mix.k"] = c.W["l0.mix.k"] * 64                                     # above the floor the size of the keys cancels
    assert distance(F.forward(c.cfg, W2, toks), c.want(toks)).max() > 100 * TOL["float32"]
    b = c.batch("float32")
    for size in (100, 1):
        b.reset(0)
        close_to(in_portions(b, 0, toks, size), c.want(toks), "float32")
    b.close()


@pytest.mark.parametrize("layer", [lig(heads=2, dim=16, vdim=16, decay=(0.9999, 1.0)), mls(heads=2, dim=16, vdim=16, cap=15.0)])
def test_state_reaches_far_back(make, layer):
    """Hardly any decay: the first token still shows after 260 positions, across block and portion edges."""
    def edit(W):
        if "l0.mix.f.b" in W:
            W["l0.mix.f.b"][:] = 14.0
    c = make(config([layer]), edit=edit)
    toks = c.tokens(260)
    want = c.want(toks)
    other = list(toks)
    other[0] = (other[0] + 1) % c.cfg["vocab"]
    assert distance(c.want(other)[-1:], want[-1:]).max() > 20 * TOL["float32"]
    for dtype in TOL:
        b = c.batch(dtype)
        for size in (260, 64, [63, 1, 66]):
            b.reset(0)
            close_to(in_portions(b, 0, toks, size), want, dtype, str(size))
        b.close()


# ---- schedules ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size", [1, 2, 3, 15, 16, 17, 63, 64, 65, 129, [2, 100, 3, 1, 17]])
def test_portions(make, size, dtype):
    c = make(MIXED)
    toks = c.tokens(70 if size == 1 else 199)
    b = c.batch(dtype, pool_pages=40)
    close_to(in_portions(b, 0, toks, size), c.want(toks), dtype, "portions of %s" % size, c.slack(toks))
    b.close()


def test_engine_chunks(make, monkeypatch):
    """A portion longer than the executor's own chunk, cut inside it."""
    monkeypatch.setenv("QW3B200_PREFILL_CHUNK", "48")
    c = make(MIXED)
    toks = c.tokens(160)
    b = c.batch("float32")
    want = [0, 1, 47, 48, 49, 95, 96, 143, 144, 159, 50]
    close_to(b.score(0, toks, want), c.want(toks)[want], "float32")
    b.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_prompt(make, dtype):
    """More than one of the executor's 1024-token chunks: attention tiles of every fill, many blocks of the recurrences."""
    c = make(config([att(heads=8, kv=2, dim=64, rot=16, scale=0.5), lig(), mls()]))
    toks = c.tokens(1500)
    at = [0, 1, 127, 128, 500, 1022, 1023, 1024, 1025, 1151, 1152, 1498, 1499]
    b = c.batch(dtype, max_ctx=1600, page_order=2)
    close_to(b.score(0, toks, at), c.want(toks)[at], dtype)
    b.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(make, dtype):
    """200 greedy steps through the decode kernels; every step's logits against the whole sequence at once."""
    c = make(MIXED)
    toks = c.tokens(5)
    b = c.batch(dtype, page_order=2)
    b.prefill(0, toks)
    got = [b.last_logits(1)[0].copy()]
    seq = toks + b.read_output()[0]
    for _ in range(200):
        b.greedy_step()
        got.append(b.last_logits(1)[0].copy())
        seq += b.read_output()[0]
    close_to(np.array(got), c.want(seq[:-1])[len(toks) - 1:], dtype, "", c.slack(seq[:-1])[len(toks) - 1:])
    for lg, t in zip(got, seq[len(toks):]):
        assert t == int(lg.argmax())
    b.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_batch_against_each_alone(make, dtype):
    """Prompts of unequal length decoded together; each row against the oracle, and within rounding against the request alone."""
    c = make(MIXED)
    prompts = [c.tokens(n) for n in (1, 67, 16, 130, 15)]
    alone = []
    for p in prompts:
        b = c.batch(dtype)
        b.prefill(0, p)
        lg, seq = [b.last_logits(1)[0].copy()], p + b.read_output()[0]
        for _ in range(20):
            b.greedy_step()
            lg.append(b.last_logits(1)[0].copy())
            seq += b.read_output()[0]
        close_to(np.array(lg), c.want(seq[:-1])[len(p) - 1:], dtype, "alone", c.slack(seq[:-1])[len(p) - 1:])
        alone.append((np.array(lg), seq))
        b.close()
    b = c.batch(dtype, n_seqs=5, page_order=1)
    first = []
    for s, p in enumerate(prompts):
        b.prefill(s, p)
        first.append(b.last_logits(1)[0].copy())
    seqs = [p + t for p, t in zip(prompts, b.read_output())]
    steps = [first]
    for _ in range(20):
        b.greedy_step()
        steps.append([r.copy() for r in b.last_logits(5)])
        for s, t in enumerate(b.read_output()):
            seqs[s] = seqs[s] + t
    for s in range(5):
        got = np.array([st[s] for st in steps])
        slack = c.slack(seqs[s][:-1])[len(prompts[s]) - 1:]
        close_to(got, c.want(seqs[s][:-1])[len(prompts[s]) - 1:], dtype, "sequence %d" % s, slack)
        if seqs[s] == alone[s][1]:
            assert (distance(got, alone[s][0]) < (2e-5 if dtype == "float32" else np.maximum(2e-2, 4 * slack))).all()
    b.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_large_batch(make, dtype):
    """34 sequences decoded together, then the first 9 of them."""
    c = make(MIXED)
    n = 34
    prompts = [c.tokens(1 + (37 * s) % 140) for s in range(n)]
    b = c.batch(dtype, n_seqs=n, max_ctx=160, pool_pages=10 * n)
    for s, p in enumerate(prompts):
        b.prefill(s, p)
    seqs = [p + t for p, t in zip(prompts, b.read_output())]
    for active in (n, n, 9):
        b.set_active(active)
        b.greedy_step()
        got = b.last_logits(active)
        close_to(got, np.stack([c.want(seqs[s])[-1] for s in range(active)]), dtype, "%d active" % active,
                 np.array([c.slack(seqs[s])[-1] for s in range(active)]))
        for s, t in enumerate(b.read_output()[:active]):
            seqs[s] = seqs[s] + t
    b.close()


def test_pages_and_slots_used_again(make):
    """Requests interleaved over a small pool: slots and pages return with other contents."""
    c = make(MIXED)
    b = c.batch("float32", n_seqs=3, max_ctx=128, pool_pages=12)
    for rnd in range(3):
        a, d = c.tokens(50 + 7 * rnd), c.tokens(33)
        wa, wd = c.want(a), c.want(d)
        got_a = [b.score(0, a[:20], range(20))]
        got_d = [b.score(2, d[:17], range(17))]
        got_a.append(b.score(0, a[20:], range(len(a) - 20)))
        b.swap(2, 1)
        got_d.append(b.score(1, d[17:], range(16)))
        close_to(np.concatenate(got_a), wa, "float32", "round %d, slot 0" % rnd)
        close_to(np.concatenate(got_d), wd, "float32", "round %d, slot 2 then 1" % rnd)
        b.reset(1)
        b.reset(0)
        assert b.pool_info()["free"] == 12
    b.close()


def test_pool_exhaustion_is_refused_before_anything_runs(qb, make):
    c = make(MIXED)
    b = c.batch("float32", n_seqs=2, max_ctx=128, pool_pages=4)
    toks = c.tokens(40)
    with pytest.raises(qb.QbError):
        b.score(0, c.tokens(80), [0])
    close_to(b.score(0, toks, range(40)), c.want(toks), "float32")
    b.close()


def test_snapshot_and_prefix(make):
    c = make(MIXED)
    toks = c.tokens(64)
    want = c.want(toks)
    b = c.batch("float32", n_seqs=2, max_ctx=128, pool_pages=20)
    b.prefill(0, toks[:32], more=True)
    px = b.prefix_capture(0, toks[:32])
    snap = b.snapshot()
    close_to(b.score(0, toks[32:], range(32)), want[32:], "float32")
    b.restore(snap)
    b.free_snapshot(snap)
    close_to(b.score(0, toks[32:], range(32)), want[32:], "float32", "after restore")
    b.prefix_attach(1, px)
    close_to(b.score(1, toks[32:], range(32)), want[32:], "float32", "from the shared prefix")
    b.prefix_release(px)
    b.close()


# ---- far keys, page and tile edges, the sink --------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_one_far_key_decides(make, dtype):
    """A raised scale and no weight on the rotated dimensions: the last token's query is answered by the one token that scores
    highest with it, wherever that lies -- at page, tile and span borders, in a prompt and in decoding."""
    cfg = config([att(heads=2, kv=1, dim=32, rot=4, scale=1.5, ff=None)], width=128, vocab=400)

    def edit(W):
        W["l0.mix.q.norm"][:4] = 0
        W["l0.mix.g"][:] = 0
    c = make(cfg, edit=edit)
    w, n = c.W, 300
    h = w["embed"] * 6.5
    k = F.rms_norm(h @ w["l0.mix.k"].T, w["l0.mix.k.norm"], 1e-5)
    s = F.rms_norm(h @ w["l0.mix.q"][:32].T, w["l0.mix.q.norm"], 1e-5) @ k.T     # head 0: query token x key token
    last = int((np.sort(s, 1)[:, -1] - np.sort(s, 1)[:, -2]).argmax())
    star = int(s[last].argmax())
    perm = [int(t) for t in np.random.default_rng(9).permutation(400) if t not in (last, star)]
    for at in (0, 1, 15, 16, 17, 63, 64, 127, 128, 129, 255):
        base = perm[:at] + [star] + perm[at + 1:n]
        toks = base + [last]
        want = c.want(toks)[-1:]
        moved = list(toks)
        moved[at] = perm[at]
        assert distance(c.want(moved)[-1:], want).max() > 5 * TOL[dtype], "the key at %d does not show" % at
        b = c.batch(dtype, pool_pages=24)
        close_to(b.score(0, toks, [n]), want, dtype, "key %d, prompt" % at)
        b.reset(0)
        b.prefill(0, base, more=True)
        close_to(b.score(0, toks[n:], [0]), want, dtype, "key %d, decoded" % at)
        b.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sink_takes_part_from_the_first_token(make, dtype, monkeypatch):
    """A scale near zero: the sink weighs as much as a key, so a row of n tokens keeps n / (n + 1) of its mean.  The norm behind the
    sublayer hides that factor unless its eps is large."""
    c = make(config([att(scale=0.01, ff=None)], eps=0.5))
    toks = c.tokens(40)
    want = c.want(toks)
    import inspect
    ns = dict(vars(F))
    exec(inspect.getsource(F.attention).replace("+ np.exp(-m)", ""), ns)
    with monkeypatch.context() as m:
        m.setitem(F.MIXERS, "attention", ns["attention"])
        assert distance(c.want(toks)[:3], want[:3]).max() > TOL[dtype]
    b = c.batch(dtype)
    close_to(b.score(0, toks, range(40)), want, dtype, "prompt")
    b.reset(0)
    close_to(in_portions(b, 0, toks, 1), want, dtype, "decoded")
    b.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_large_scores(make, dtype):
    """Scores far above and below the sink's: no overflow, and no weight lost against a maximum that is not there."""
    c = make(config([att(heads=4, kv=2, dim=24, rot=8, scale=3.0, ff=None)], eps=1e-3))
    toks = c.tokens(150)
    b = c.batch("float32")
    close_to(in_portions(b, 0, toks, [100, 1, 49]), c.want(toks), "float32")
    b.close()
    b = c.batch(dtype)
    assert np.isfinite(in_portions(b, 0, toks, [100, 1, 49])).all()
    b.close()


# ---- generation through the scheduler -------------------------------------------------------------------------------------------
@pytest.mark.parametrize("loop", ["run", "run_compact", "prefix_cache"])
def test_greedy_generation_through_the_scheduler(qb, make, loop):
    c = make(MIXED)
    shared = c.tokens(32)
    prompts = [shared + c.tokens(9), c.tokens(3), shared + c.tokens(20), c.tokens(70), c.tokens(1)]
    want = [c.greedy(p, 12) for p in prompts]
    reqs = [qb.serve.Request(i, p, 12, arrival_step=6 * i) for i, p in enumerate(prompts)]
    if loop == "run":
        b = c.batch("float32", n_seqs=2, max_ctx=160)
        qb.serve.run(b, reqs, speculative=False)
    else:
        b = c.batch("float32", n_seqs=3, max_ctx=160, pool_pages=24)
        cache = qb.serve.PrefixCache(b) if loop == "prefix_cache" else None
        qb.serve.run_compact(b, reqs, speculative=False, prefill_chunk=13, prefix_cache=cache)
        if cache:
            assert cache.hits >= 1
            cache.clear()
    assert [r.tokens for r in reqs] == want
    b.close()


def test_sampled_generation(qb, make):
    """Top-1 sampling is greedy; draws decide tokens."""
    c = make(MIXED)
    prompts = [c.tokens(n) for n in (5, 40, 17)]

    def serve(sel, n_seqs, **sampling):
        b = c.batch("float32", n_seqs=n_seqs, max_ctx=96, pool_pages=6 * n_seqs)
        reqs = [qb.serve.Request(i, prompts[i], 16) for i in sel]
        qb.serve.run_compact(b, reqs, speculative=False, sampling=sampling, rng_of=lambda r: random.Random(7 + r.rid))
        b.close()
        return [r.tokens for r in reqs]
    assert serve([0, 1, 2], 3, temp=0.8, top_k=1) == [c.greedy(p, 16) for p in prompts]
    together = serve([0, 1, 2], 3, temp=1.1, top_k=20, top_p=0.95)
    assert together == [serve([i], 1, temp=1.1, top_k=20, top_p=0.95)[0] for i in range(3)]
    assert together != [c.greedy(p, 16) for p in prompts]


# ---- loading and the command line -------------------------------------------------------------------------------------------------
def test_loader_errors(qb, ctx, tmp_path):
    W = F.random_weights(MIXED, 3)

    def attempt(cfg, weights, match):
        F.write_model(str(tmp_path), cfg, weights)
        with pytest.raises(qb.QbError, match=match):
            qb.Model.load(ctx, str(tmp_path))

    def layers(i, **kw):
        return dict(MIXED, layers=MIXED["layers"][:i] + [dict(MIXED["layers"][i], **kw)] + MIXED["layers"][i + 1:])
    mixer = lambda i, **kw: layers(i, mixer=dict(MIXED["layers"][i]["mixer"], **kw))
    attempt(MIXED, {k: v for k, v in W.items() if k != "l2.mix.f.b"}, "l2.mix.f.b is missing")
    attempt(MIXED, {k: v for k, v in W.items() if k != "l0.ls2"}, "l0.ls2 is missing")
    attempt(MIXED, dict(W, head=W["head"][:-1]), "head does not have the shape")
    attempt({k: v for k, v in MIXED.items() if k != "embedding"}, W, "embedding is missing")
    attempt(layers(0, type="conv"), W, "mixer conv is not known")
    attempt(layers(5, weights_of=9), W, "weights_of must name a layer")
    attempt(layers(0, weights_of=5), W, "in a circle")
    attempt(layers(5, weights_of=3), W, "must equal the layer")
    attempt(mixer(0, kv_heads=4), W, "multiple of kv_heads")
    attempt(mixer(0, vdim=10), W, "vdim must equal dim")
    attempt(mixer(1, decay=[0.5]), W, "one number per head")
    attempt(mixer(2, gate_cap=0), W, "gate_cap must be positive")


def test_seeded_model_of_a_configuration(qb, ctx):
    m = qb.Model.layered_synth(ctx, MIXED, 11)
    b = qb.Batch(m, 1, 64, 0)
    lg = b.score(0, [1, 2, 3], [2])
    assert np.isfinite(lg).all() and lg.std() > 0.1
    with pytest.raises(qb.QbError):
        qb.Batch(m, 1, 64, 1)                                                # no draft layer
    b.close()
    m.close()


def test_trace_replay_and_generate_programs(make, tmp_path):
    c = make(MIXED)
    a, d = c.tokens(37), c.tokens(20)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:20], "want": [19, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[20:], "want": [16]}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "d", "tokens": d[:-1], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "d", "tokens": d[-1:], "want": [0]}], "end": ["d"]}]
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", c.dir, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "37"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr[-500:]
    assert [ln for ln in p.stdout.splitlines() if ln.startswith("done")] == ["done %d" % i for i in range(4)]
    read = lambda i: np.fromfile(tmp_path / ("%d.f32" % i), np.float32).reshape(-1, MIXED["vocab"])
    close_to(read(0), c.want(a)[[19, 3]], "float32")
    close_to(read(1), c.want(a)[[36]], "float32")
    close_to(read(3), c.want(d)[[19]], "float32")
    assert not (tmp_path / "2.f32").exists()
    p = subprocess.run([os.path.join(ROOT, "bin", "generate"), "--model", c.dir, "--dtype", "float32", "--new-tokens", "8", "--slots", "2",
                        "--prompt", ",".join(map(str, a)), "--prompt", ",".join(map(str, d)), "--prompt", "5"], capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr[-500:]
    assert [[int(t) for t in ln.split(",")] for ln in p.stdout.split()] == [c.greedy(q, 8) for q in (a, d, [5])]
