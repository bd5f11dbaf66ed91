"""The Kezilix design (layered models) on the GPU against the plain numpy restatement in oracle/kezilix_oracle.py.

Every configuration here is the tests' own: odd head counts, sizes that are no multiples of 16 or 64, rotations over a part
of a head, layers with and without feed-forward.  32-bit runs are compared tightly, bfloat16 runs within the rounding of
their products.  Where random weights would drown a single key among many, the score scale is raised so that one key
decides the row."""
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
import kezilix_oracle as K  # noqa: E402
from layered_case import TOL, Case, close_to, in_portions  # noqa: E402

YARN = {"factor": 6.0, "original": 256, "fast": 24.0, "slow": 2.0}


def ret(heads=3, dim=24, vdim=40, rot=16, base=5000.0, decay=(0.97, 0.9995, 0.9), ff=None):
    return {"type": "retention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "rot": {"dims": rot, "base": base}, "decay": list(decay)[:heads]}}


def lat(heads=5, dim=20, rot_dim=12, vdim=28, rank=52, rot=12, scale=0.2, yarn=YARN, ff=72):
    r = {"dims": rot, "base": 8000.0}
    if yarn:
        r["scaling"] = yarn
    return {"type": "latent_attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "rot": r, "scale": scale}}


def config(layers, loop=None, width=88, vocab=210, eps=1e-5):
    return {"architecture": "Kezilix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers, "loop": loop}


MIXED = config([lat(), ret(), ret(heads=2, dim=40, vdim=24, rot=40, decay=(0.99, 0.8), ff=56), lat(heads=3, yarn=None, ff=None), ret()],
               loop={"start": 1, "stop": 4, "times": 2})


@pytest.fixture
def make(qb, ctx, tmp_path):
    made = []

    def f(cfg, **kw):
        made.append(Case(K, qb, ctx, tmp_path / ("m%d" % len(made)), cfg, **kw))
        return made[-1]
    yield f
    for c in made:
        c.close()


# ---- products ----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("N,Kd", [(130, 72), (40, 8), (300, 200), (1024, 1536), (64, 2048)])
def test_dense_product(qb, ctx, N, Kd):
    rng = np.random.default_rng(N)
    w = K.bf16_round(rng.standard_normal((N, Kd)).astype(np.float32))
    dw = qb.binding.DenseWeight(ctx, N, Kd, (w.view(np.uint32) >> 16).astype(np.uint16))
    for M in (1, 3, 16, 17, 32, 33, 64, 65, 100, 129, 300):
        x = rng.standard_normal((M, Kd)).astype(np.float32)
        np.testing.assert_allclose(dw.matmul(x, f32=True), x.astype(np.float64) @ w.T.astype(np.float64), rtol=0, atol=2e-6 * Kd ** 0.5 * 4)
        xb = K.bf16_round(x)
        np.testing.assert_allclose(dw.matmul(x), xb.astype(np.float64) @ w.T.astype(np.float64), rtol=0, atol=4e-6 * Kd ** 0.5 * 4)
    dw.free()


# ---- each mechanism alone --------------------------------------------------------------------------------------------------
ALONE = {
    "retention": config([ret()]),
    "retention_full_rotation": config([ret(heads=1, dim=16, vdim=16, rot=16, decay=(0.99,))]),
    "retention_no_decay": config([ret(heads=2, dim=10, vdim=70, rot=4, decay=(1.0, 0.5))]),
    "retention_wide": config([ret(heads=2, dim=72, vdim=136, rot=64, decay=(0.99, 0.999))]),
    "latent": config([lat(ff=None)]),
    "latent_plain_rotation": config([lat(ff=None, yarn=None)]),
    "latent_part_rotation": config([lat(ff=None, rot_dim=20, rot=8)]),
    "latent_one_head": config([lat(heads=1, dim=16, rot_dim=16, rot=16, vdim=16, rank=16, ff=None)]),
    "latent_ff": config([lat(ff=40)]),
    "loop_from_first": config([ret(), lat()], loop={"start": 0, "stop": 1, "times": 3}),
    "loop_to_last": config([ret(), ret(), lat()], loop={"start": 1, "stop": 3, "times": 4}),
    "loop_once": config([ret(), lat(), ret()], loop={"start": 1, "stop": 2, "times": 1}),
    "odd_width": config([ret(heads=3, dim=22, vdim=30, rot=10, ff=33), lat(heads=3, dim=18, rot_dim=6, rot=6, vdim=17, rank=45, ff=50)], width=90, vocab=131),
    "odd_width_prime": config([lat(heads=1, dim=7, rot_dim=2, rot=2, vdim=5, rank=19, ff=11), ret(heads=1, dim=3, vdim=7, rot=2, decay=(0.9,))], width=67, vocab=101,
                              loop={"start": 0, "stop": 2, "times": 2}),
    "mixed": MIXED,
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ALONE))
def test_mechanism_alone(make, name, dtype):
    c = make(ALONE[name])
    b = c.batch(dtype)
    for n in (1, 2, 65, 150):
        toks, trace = c.tokens(n), []
        want = c.want(toks, trace)
        b.reset(0)
        b.layer_trace(True)
        got = b.score(0, toks, range(n))
        layers = b.layer_trace_read()
        for i, w in enumerate(trace):
            close_to(layers[i], w, dtype, "%s: residual after run %d of %d tokens" % (name, i, n))
        close_to(got, want, dtype, name)
    b.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("layer", [lat(heads=2, dim=16, rot_dim=8, rot=8, vdim=264, rank=40, ff=None),            # values too wide to expand
                                   lat(heads=17, dim=24, rot_dim=8, rot=8, vdim=24, rank=520, ff=None),           # latent too wide for the tiled form
                                   lat(heads=33, dim=8, rot_dim=8, rot=8, vdim=136, rank=264, ff=None),
                                   ret(heads=1, dim=300, vdim=300, rot=300, decay=(0.99,))])                      # state too large for a chunk's tiles
def test_sizes_beyond_the_tiled_kernels(make, layer, dtype):
    c = make(config([layer]))
    b = c.batch(dtype)
    toks = c.tokens(140)
    close_to(in_portions(b, 0, toks, [100, 1, 2, 37]), c.want(toks), dtype, str(layer["mixer"]))
    b.close()


@pytest.mark.parametrize("heads,rank,rot_dim,n_seqs", [(20, 512, 64, 40), (50, 128, 16, 1), (1, 256, 32, 40), (7, 96, 16, 3), (34, 448, 80, 40)])
def test_absorbed_attention_shapes(make, heads, rank, rot_dim, n_seqs):
    """Decode rows over many keys, at several head counts and latent sizes; a large batch cuts a sequence into few spans of
    several 128-key tiles, and a raised scale lets the running maximum grow from tile to tile."""
    c = make(config([lat(heads=heads, dim=16, rot_dim=rot_dim, rot=rot_dim, vdim=24, rank=rank, scale=0.7, ff=None)]))
    n = 1300 if n_seqs == 40 else 333
    toks = c.tokens(n + 6)
    want = c.want(toks)[n:]
    b = c.batch("bfloat16", n_seqs=n_seqs, max_ctx=1400, pool_pages=100)
    b.prefill(n_seqs - 1, toks[:n], more=True)
    got = [b.score(n_seqs - 1, [t], [0]) for t in toks[n:n + 3]]
    got.append(b.score(n_seqs - 1, toks[n + 3:], range(3)))
    close_to(np.concatenate(got), want, "bfloat16")
    b.close()


# ---- schedules ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size", [1, 2, 3, 15, 16, 17, 63, 64, 65, 129, [2, 100, 3, 1, 17]])
def test_portions(make, size, dtype):
    c = make(MIXED)
    toks = c.tokens(70 if size == 1 else 199)
    b = c.batch(dtype, pool_pages=40)
    close_to(in_portions(b, 0, toks, size), c.want(toks), dtype, "portions of %s" % size)
    b.close()


def test_engine_chunks(make, monkeypatch):
    """A portion longer than the executor's own chunk, cut inside it."""
    monkeypatch.setenv("QW3B200_PREFILL_CHUNK", "48")
    c = make(MIXED)
    toks = c.tokens(160)
    b = c.batch("float32")
    want = [0, 1, 47, 48, 49, 95, 96, 143, 144, 159, 50]                  # unordered places too
    close_to(b.score(0, toks, want), c.want(toks)[want], "float32")
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
    close_to(np.array(got), c.want(seq[:-1])[len(toks) - 1:], dtype)
    for lg, t in zip(got, seq[len(toks):]):
        assert t == int(lg.argmax())
    b.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_batch_equals_each_alone(make, dtype):
    c = make(MIXED)
    prompts = [c.tokens(n) for n in (1, 67, 16, 130, 15)]
    alone = []
    for p in prompts:
        b = c.batch(dtype)
        b.prefill(0, p)
        lg = [b.last_logits(1)[0].copy()]
        for _ in range(20):
            b.greedy_step()
            lg.append(b.last_logits(1)[0].copy())
        alone.append(np.array(lg))
        b.close()
    b = c.batch(dtype, n_seqs=5, page_order=1)
    first = []
    for s, p in enumerate(prompts):
        b.prefill(s, p)
        first.append(b.last_logits(1)[0].copy())
    steps = [first]
    for _ in range(20):
        b.greedy_step()
        steps.append([r.copy() for r in b.last_logits(5)])
    for s in range(5):
        np.testing.assert_array_equal(np.array([st[s] for st in steps]), alone[s])
    b.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_large_batch(make, dtype):
    """34 sequences decoded together (more than one 32-row block of the per-head products), then the first 9 of them."""
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
        close_to(got, np.stack([c.want(seqs[s])[-1] for s in range(active)]), dtype, "%d active" % active)
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


# ---- far keys, page edges, sinks -------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_one_far_key_decides(make, dtype):
    """A raised scale, no rotated part in the score: the last token's query is answered by the one token that scores highest
    with it, wherever that lies -- at page and span borders, in a prompt and in decoding."""
    cfg = config([lat(heads=2, dim=32, rot_dim=2, rot=2, vdim=32, rank=64, scale=2.0, yarn=None, ff=None)], width=128, vocab=400)

    def edit(W):
        for h in range(2):
            W["l0.mix.q"][h * 34 + 32:h * 34 + 34] = 0
    c = make(cfg, edit=edit)
    w, n = c.W, 300
    h = K.rms_norm(K.rms_norm(w["embed"], w["embed.norm"], 1e-5), w["l0.norm1"], 1e-5)
    key = K.rms_norm((h @ w["l0.mix.dkv"].T)[:, :64], w["l0.mix.dkv.norm"], 1e-5) @ w["l0.mix.uk"][:32].T
    s = (h @ w["l0.mix.q"][:32].T) @ key.T                                  # head 0: query token x key token
    last = int((np.sort(s, 1)[:, -1] - np.sort(s, 1)[:, -2]).argmax())
    star = int(s[last].argmax())
    perm = [int(t) for t in np.random.default_rng(9).permutation(400) if t not in (last, star)]
    for at in (0, 1, 15, 16, 17, 127, 128, 129, 255):
        base = perm[:at] + [star] + perm[at + 1:n]
        toks = base + [last]
        want = c.want(toks)[-1:]
        moved = list(toks)
        moved[at] = perm[at]
        assert np.sqrt(((c.want(moved)[-1:] - want) ** 2).mean()) > 5 * TOL[dtype] * np.sqrt((want ** 2).mean()), "the key at %d does not show" % at
        b = c.batch(dtype, pool_pages=24)
        close_to(b.score(0, toks, [n]), want, dtype, "key %d, prompt" % at)
        b.reset(0)
        b.prefill(0, base, more=True)
        close_to(b.score(0, toks[n:], [0]), want, dtype, "key %d, decoded" % at)
        b.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sink_counts_once(make, dtype):
    """A large sink: the attention output of the first tokens is mostly removed, later less so."""
    def edit(W):
        W["l0.mix.sink"][:] = [3.0, -20.0, 0.0, 6.0, 1.0]
    c = make(config([lat(ff=None)]), edit=edit)
    toks = c.tokens(40)
    want = c.want(toks)
    for s in ([-20.0] * 5,):                                                 # without a sink the rows differ visibly
        W2 = dict(c.W)
        W2["l0.mix.sink"] = np.array(s, np.float32)
        d = K.forward(c.cfg, W2, toks) - want
        assert np.sqrt((d ** 2).mean()) > 2 * TOL[dtype] * np.sqrt((want ** 2).mean())
    b = c.batch(dtype)
    close_to(b.score(0, toks, range(40)), want, dtype, "prompt")
    b.reset(0)
    close_to(in_portions(b, 0, toks, 1), want, dtype, "decoded")
    b.close()


def test_state_reaches_far_back(make):
    """Decay near 1: the first tokens still carry weight after 260 positions, across chunk and portion edges."""
    c = make(config([ret(heads=2, dim=16, vdim=16, rot=4, decay=(0.9999, 1.0))]))
    toks = c.tokens(260)
    want = c.want(toks)
    other = list(toks)
    other[0] = (other[0] + 1) % c.cfg["vocab"]
    assert np.sqrt(((c.want(other)[-1] - want[-1]) ** 2).mean()) > 20 * TOL["float32"] * np.sqrt((want ** 2).mean())
    b = c.batch("float32")
    for size in (260, 64, [63, 1, 66]):
        b.reset(0)
        close_to(in_portions(b, 0, toks, size), want, "float32", str(size))
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
    """Top-1 sampling is greedy; a sampled stream does not depend on the other requests of the batch; draws decide tokens."""
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
    pen = serve([0, 1, 2], 3, temp=0.01, presence=50.0)                       # a heavy presence penalty: no token twice
    assert all(len(set(p + t)) == len(set(p)) + len(t) for p, t in zip(prompts, pen))


# ---- loading and the command line -------------------------------------------------------------------------------------------------
def test_loader_errors(qb, ctx, tmp_path):
    W = K.random_weights(MIXED, 3)

    def attempt(cfg, weights, match):
        K.write_model(str(tmp_path), cfg, weights)
        with pytest.raises(qb.QbError, match=match):
            qb.Model.load(ctx, str(tmp_path))
    attempt(MIXED, {k: v for k, v in W.items() if k != "l1.mix.g"}, "l1.mix.g is missing")
    attempt(MIXED, dict(W, head=W["head"][:-1]), "head does not have the shape")
    attempt(dict(MIXED, architecture="Other"), W, "'Other' is not known")
    attempt(dict(MIXED, layers=[dict(MIXED["layers"][0], type="conv")]), W, "mixer conv is not known")
    attempt(dict(MIXED, loop={"start": 3, "stop": 9, "times": 2}), W, "loop")
    with open(tmp_path / "config.json", "w") as f:
        f.write("{")
    with pytest.raises(qb.QbError, match="not JSON"):
        qb.Model.load(ctx, str(tmp_path))
    with pytest.raises(qb.QbError):
        qb.Model.load(ctx, str(tmp_path / "none"))


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
             {"step": 1, "entries": [{"id": "d", "tokens": d, "want": []}], "end": ["d"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[20:], "want": [16]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "d", "tokens": d[:2], "want": [1]}], "end": ["d"]}]
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", c.dir, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "57"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr[-500:]
    assert [ln for ln in p.stdout.splitlines() if ln.startswith("done")] == ["done %d" % i for i in range(4)]
    read = lambda i: np.fromfile(tmp_path / ("%d.f32" % i), np.float32).reshape(-1, MIXED["vocab"])
    close_to(read(0), c.want(a)[[19, 3]], "float32")
    close_to(read(2), c.want(a)[[36]], "float32")
    close_to(read(3), c.want(d)[[1]], "float32")
    assert not (tmp_path / "1.f32").exists()
    p = subprocess.run([os.path.join(ROOT, "bin", "generate"), "--model", c.dir, "--dtype", "float32", "--new-tokens", "8", "--slots", "2",
                        "--prompt", ",".join(map(str, a)), "--prompt", ",".join(map(str, d)), "--prompt", "5"], capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr[-500:]
    assert [[int(t) for t in ln.split(",")] for ln in p.stdout.split()] == [c.greedy(q, 8) for q in (a, d, [5])]
