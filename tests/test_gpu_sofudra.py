"""GPU parity of the Sofudra decoders (grouped attention, linear attention, loops) against the plain oracle."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import hybrid_util as U
import kalosm_b200 as kb
import sofudra_util as V
from gpu_util import dev  # noqa: F401
from kalosm_b200 import models, sofudra
from kalosm_b200.__main__ import generate

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = ["float32", "bfloat16"]


def toks(cfg, n, seed=1):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n)


def check(dev, cfg, w, tokens, dtype, sizes, m=None, **kw):
    """The logits of every position, fed in portions, against the oracle; `sizes` may be a list of such lists."""
    own = m is None
    m = m or V.gpu_model(dev, cfg, w, dtype, **kw)
    want = V.oracle_logits(cfg, w, tokens)
    tol = V.tolerance(cfg, w, tokens, want, dtype)
    for cut in sizes if isinstance(sizes[0], list) else [sizes]:
        e = U.err(U.run_portions(m, tokens, cut), want)
        assert e < tol, (cut, e, tol)
    assert dev.status() == 0
    if own:
        m.free()


def alone(layers, **kw):
    """One kind of layer with an identity head: the logits are the normalised residual stream."""
    return V.config(layers, width=80, vocab=80, mult=1.0, embed=1.0, cap=kw.pop("cap", 0.0), **kw)


# ---- each mechanism alone ------------------------------------------------------------------------------------

ATTENTIONS = [dict(), dict(heads=1, kv_heads=1, dim=8, vdim=8, window=1, rot=V.rotary(8)),
              dict(heads=5, kv_heads=5, dim=33, vdim=17, window=33, rot=V.rotary(4, 50.0)),
              dict(heads=6, kv_heads=1, dim=64, vdim=96, window=64, rot=V.rotary(64, 1000.0, 4.0, 32, 16.0, 1.0)),
              dict(heads=8, kv_heads=2, dim=128, vdim=128, window=50, rot=V.rotary(64, 500000.0, 8.0, 512, 32.0, 2.0)),
              dict(heads=4, kv_heads=4, dim=200, vdim=64, window=100, rot=V.rotary(200, 100.0, 1.5)),
              dict(heads=4, kv_heads=2, dim=40, vdim=250, window=7, scale=0.4),
              dict(heads=3, kv_heads=1, dim=300, vdim=30, window=90), dict(heads=2, kv_heads=2, dim=24, vdim=400, window=5000, rot=V.rotary(24)),
              dict(heads=14, kv_heads=2, dim=16, vdim=8, window=20)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", range(len(ATTENTIONS)))
def test_attention_layer(dev, dtype, shape):
    cfg = alone([V.attention(mlp=0, **ATTENTIONS[shape])])
    w = V.weights(cfg, shape, U.identity_head(cfg))
    check(dev, cfg, w, toks(cfg, 150), dtype, [[150], [70, 3, 40, 2, 1]])


LEFTS = [dict(), dict(heads=1, kv_heads=1, dim=8, vdim=8, softcap=1.0), dict(heads=6, kv_heads=3, dim=40, vdim=33, softcap=30.0, scale=0.5),
         dict(heads=8, kv_heads=1, dim=128, vdim=64, softcap=2.0), dict(heads=4, kv_heads=2, dim=256, vdim=200, softcap=9.0),
         dict(heads=4, kv_heads=1, dim=20, vdim=264, softcap=5.0)]
RIGHTS = [dict(), dict(heads=1, dim=8, vdim=8, decay=[0.9]), dict(heads=5, dim=33, vdim=17), dict(heads=2, dim=64, vdim=96, decay=[1.0, 0.0]),
          dict(heads=4, dim=128, vdim=128), dict(heads=2, dim=200, vdim=40, decay=[0.99, 0.05]), dict(heads=2, dim=300, vdim=31)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", range(len(LEFTS)))
def test_left_side_alone(dev, dtype, shape):
    cfg = alone([V.parallel(V.left(**LEFTS[shape]), left_scale=1.3, mlp=0)])
    ident = U.identity_head(cfg)
    w = V.weights(cfg, 20 + shape, lambda n, a: np.zeros_like(a) if n.endswith("right.o") else ident(n, a))
    check(dev, cfg, w, toks(cfg, 150), dtype, [[150], [66, 3, 40, 2, 1]])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", range(len(RIGHTS)))
def test_right_side_alone(dev, dtype, shape):
    cfg = alone([V.parallel(b=V.right(**RIGHTS[shape]), right_scale=0.6, mlp=0)])
    ident = U.identity_head(cfg)
    w = V.weights(cfg, 40 + shape, lambda n, a: np.zeros_like(a) if n.endswith("left.o") else ident(n, a))
    check(dev, cfg, w, toks(cfg, 210), dtype, [[210], [70, 3, 65, 2, 17, 1], [64, 64, 64, 18], [16, 48, 128, 18]])


@pytest.mark.parametrize("dim,vdim", [(128, 100), (40, 64)])
def test_linear_attention_in_segments(dev, dim, vdim):
    # prompts long enough to be cut into segments that run side by side, also behind earlier tokens
    cfg = alone([V.parallel(b=V.right(2, dim, vdim, [0.9995, 0.9]), mlp=0)])
    ident = U.identity_head(cfg)
    w = V.weights(cfg, 62, lambda n, a: np.zeros_like(a) if n.endswith("left.o") else ident(n, a))
    check(dev, cfg, w, toks(cfg, 1700), "bfloat16", [[1700], [37, 1100, 513, 50]], max_seq_len=1704)


@pytest.mark.parametrize("window,sizes", [(1, [700]), (70, [700]), (200, [650, 50]), (64, [300, 400]), (5000, [257, 443])], ids=str)
@pytest.mark.parametrize("vdim", [64, 128])
def test_attention_many_rows(dev, window, sizes, vdim):
    # enough heads and rows for two groups of rows per CTA in the prompt kernel, with and without a softcap
    cfg = alone([V.attention(heads=64, kv_heads=16, dim=40, vdim=vdim, window=window, mlp=0)])
    check(dev, cfg, V.weights(cfg, 60, U.identity_head(cfg)), toks(cfg, 700), "bfloat16", sizes, max_seq_len=704)
    if window == 5000:
        cfg = alone([V.parallel(V.left(heads=64, kv_heads=16, dim=40, vdim=vdim), mlp=0)])
        check(dev, cfg, V.weights(cfg, 61, U.identity_head(cfg)), toks(cfg, 700), "bfloat16", sizes, max_seq_len=704)


@pytest.mark.parametrize("dtype", DTYPES)
def test_feed_forward_alone(dev, dtype):
    cfg = alone([V.attention(mlp=201), V.attention(mlp=7)])
    ident = U.identity_head(cfg)
    w = V.weights(cfg, 5, lambda n, a: np.zeros_like(a) if n.endswith("mix.o") else ident(n, a))
    check(dev, cfg, w, toks(cfg, 300), dtype, [[300], [36, 1, 200, 2]])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("loop", [None, (0, 3, 2), (0, 1, 1), (2, 3, 4), (1, 3, 3)], ids=str)
def test_loops(dev, dtype, loop):
    # every pass has its own cache and state; the first layer, the last layer, one pass, all layers
    cfg = V.config([V.attention(window=12), V.parallel(), V.attention(mlp=0, window=40)], loop=loop)
    check(dev, cfg, V.weights(cfg, 70), toks(cfg, 90), dtype, [[90], [50, 2, 30, 1]])


@pytest.mark.parametrize("dtype", DTYPES)
def test_factors_around_the_layers(dev, dtype):
    for kw in (dict(cap=0.0, mult=1.0, embed=1.0), dict(cap=1.5, mult=2.0, embed=0.25), dict(eps=0.3)):
        cfg = V.config([V.parallel(), V.attention()], **kw)
        check(dev, cfg, V.weights(cfg, 71), toks(cfg, 50), dtype, [45, 2, 1])
    bare = V.config([V.attention(), V.parallel()])
    for key in ("embedding", "residual_mult", "logit_softcap"):
        del bare[key]
    check(dev, bare, V.weights(bare, 72), toks(bare, 50), dtype, [45, 2, 1])


# ---- whole models: prompts, decoding, portions -----------------------------------------------------------------

def mixed(width=72, vocab=101):
    return V.config([V.parallel(), V.attention(window=37), V.parallel(V.left(5, 1, 40, 16), V.right(4, 40, 24), mlp=0, name="parallel_2"),
                     V.attention(heads=4, kv_heads=4, dim=32, vdim=32, window=9, rot=V.rotary(32), name="attention_2")], width, vocab, loop=(1, 3, 2))


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions(dev, dtype):
    cfg = mixed()
    check(dev, cfg, V.weights(cfg, 7), toks(cfg, 200), dtype,
          [[200], [1], [2], [3, 2, 5], [64, 64, 8], [16, 15, 17, 2], [130, 1], [199, 1]])


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_agree_with_each_other(dev, dtype):
    cfg = mixed()
    w = V.weights(cfg, 8)
    m = V.gpu_model(dev, cfg, w, dtype)
    t = toks(cfg, 140)
    whole = U.run_portions(m, t, [140])
    tol = V.tolerance(cfg, w, t, V.oracle_logits(cfg, w, t), dtype)
    for sizes in ([1], [33, 2, 1], [140]):
        assert U.err(U.run_portions(m, t, sizes), whole) < tol
    assert np.array_equal(U.run_portions(m, t, [140]), whole)  # the same cut gives the same bits


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens(dev, dtype):
    cfg = mixed()
    w = V.weights(cfg, 9)
    m = V.gpu_model(dev, cfg, w, dtype)
    for n in range(1, 7):
        check(dev, cfg, w, toks(cfg, n, seed=n), dtype, [[n], [1]], m=m)


@pytest.mark.parametrize("dtype", DTYPES)
def test_state_of_an_earlier_request_is_gone(dev, dtype):
    cfg = mixed()
    w = V.weights(cfg, 10)
    m = V.gpu_model(dev, cfg, w, dtype)
    a, b = toks(cfg, 90, 1), toks(cfg, 60, 2)
    fresh = U.run_portions(m, b, [40, 1])
    U.run_portions(m, a, [90])
    assert np.array_equal(U.run_portions(m, b, [40, 1]), fresh)
    U.run_portions(m, a, [50, 1])
    single = U.run_portions(m, b[:20], [1])
    m2 = V.gpu_model(dev, cfg, w, dtype)
    assert np.array_equal(U.run_portions(m2, b[:20], [1]), single)


@pytest.mark.parametrize("dtype", DTYPES)
def test_batch_equals_each_sequence_alone(dev, dtype):
    cfg = mixed()
    w = V.weights(cfg, 11)
    m = V.gpu_model(dev, cfg, w, dtype, max_batch=3)
    seqs = np.stack([toks(cfg, 150, s) for s in (1, 2, 3)])
    want = np.stack([V.oracle_logits(cfg, w, s) for s in seqs])
    got = []
    for a, b in [(0, 130), (130, 132), (132, 142)] + [(i, i + 1) for i in range(142, 150)]:
        m.forward(seqs[:, a:b], want_logits=False)
        got.append(m.logits_at(range(3 * (b - a))).reshape(3, b - a, -1))
    got = np.concatenate(got, axis=1)
    for i in range(3):
        assert U.err(got[i], want[i]) < V.tolerance(cfg, w, seqs[i], want[i], dtype), i


@pytest.mark.parametrize("dtype", DTYPES)
def test_odd_sizes(dev, dtype):
    cfg = V.config([V.parallel(V.left(3, 3, 7, 5), V.right(3, 9, 7), mlp=37), V.attention(5, 1, 11, 3, 9, V.rotary(6, 77.0, 2.0), mlp=13),
                    V.parallel(V.left(2, 1, 13, 9), V.right(1, 5, 1), mlp=0)], width=75, vocab=53, loop=(0, 2, 2))
    check(dev, cfg, V.weights(cfg, 23), toks(cfg, 90), dtype, [[90], [40, 2, 31, 1]])


def test_larger_sizes(dev):
    # sizes that real layers have: 128-wide heads, many weight tiles
    att = V.attention(heads=8, kv_heads=2, dim=128, vdim=128, window=130, rot=V.rotary(128, 500000.0, 8.0, 64), mlp=1024)
    cfg = V.config([V.parallel(V.left(8, 2, 128, 128, softcap=20.0), V.right(8, 128, 128), mlp=1024), att], width=1024, vocab=700, loop=(1, 2, 2))
    w = V.weights(cfg, 12)
    t = toks(cfg, 300)
    check(dev, cfg, w, t, "bfloat16", [257, 41, 1])
    check(dev, cfg, w, t[:80], "float32", [70, 1])


# ---- distances that have to show: window edges, far keys, sinks, far memory ----------------------------------

def marker_model(layer, width=64):
    """One layer in which token 1 (a query) scores high on token 0 (a key) and low on everything else, so that whether that key
    is visible decides the query's output. The scores sit on a dimension that is not rotated."""
    cfg = V.config([layer], width, width, mult=1.0, embed=1.0, cap=0.0)
    ident = U.identity_head(cfg)
    mx = layer["mixer"].get("left", layer["mixer"])

    def edit(name, a):
        if name == "embed":
            a = np.random.default_rng(5).standard_normal(a.shape) * 0.3
            a[:, :2] = 0.0
            a[0, 0] = a[1, 1] = 6.0
            return a
        if ".right." in name:
            return np.zeros_like(a) if name.endswith(".o") else None
        for short, token in (("q", 1), ("k", 0)):
            if name.endswith(f".{short}"):
                a = a.reshape(-1, mx["dim"], width) * 0.5
                a[:, :, :2] = 0.0
                a[:, -1, token] = 8.0
                return a.reshape(-1, width)
            if name.endswith((f".{short}.b", f".{short}.norm")):
                return np.zeros_like(a) if name.endswith("b") else np.ones_like(a)
        if name.endswith("sink"):
            return np.full(a.shape, 1.0)
        return ident(name, a)
    return cfg, V.weights(cfg, 13, edit)


def windowed(window):
    return V.attention(4, 2, 16, 16, window, V.rotary(8, 1000.0, 2.0), scale=0.8, mlp=0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 2, 15, 63, 64, 65, 127, 129])
def test_window_edges(dev, dtype, window):
    cfg, w = marker_model(windowed(window))
    m = V.gpu_model(dev, cfg, w, dtype)
    for dist in sorted({max(0, window - 2), window - 1, window, window + 1, window + 70}):
        for at in (dist + 1, dist + 66):  # position of the query
            t = np.random.default_rng(at).integers(2, cfg["vocab"], at + 3)
            t[at] = 1
            if dist:
                t[at - dist] = 0
            want = V.oracle_logits(cfg, w, t)
            for sizes in ([len(t)], [at, 1], [max(1, at - 5), 2, 3]):
                assert U.err(U.run_portions(m, t, sizes), want) < U.TOL[dtype], (dist, at, sizes)
    # the test has teeth: a key just inside changes the query's row far beyond the tolerance
    if window > 1:
        t = np.random.default_rng(3).integers(2, cfg["vocab"], window + 3)
        t[-1] = 1
        base = V.oracle_logits(cfg, w, t)[-1]
        inside, outside = t.copy(), t.copy()
        inside[-window] = 0
        outside[-window - 1] = 0
        assert U.err(V.oracle_logits(cfg, w, inside)[-1], base) > 0.15
        assert U.err(V.oracle_logits(cfg, w, outside)[-1], base) < 1e-9


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["windowed", "capped"])
def test_far_key_among_hundreds(dev, dtype, kind):
    cfg, w = marker_model(windowed(1000) if kind == "windowed" else V.parallel(V.left(4, 2, 16, 16, 0.8, 15.0), mlp=0))
    m = V.gpu_model(dev, cfg, w, dtype, max_seq_len=1024)
    for at, key in ((700, 0), (700, 63), (700, 64), (511, 511 - 447), (699, 320)):
        t = np.random.default_rng(key).integers(2, cfg["vocab"], at + 1)
        t[at], t[key] = 1, 0
        want = V.oracle_logits(cfg, w, t)
        without = t.copy()
        without[key] = 2
        assert U.err(want[at], V.oracle_logits(cfg, w, without)[at]) > 0.15
        for sizes in ([at + 1], [at, 1], [300, 200, 150, 2]):
            assert U.err(U.run_portions(m, t, sizes)[at], want[at]) < U.TOL[dtype], (at, key, sizes)


@pytest.mark.parametrize("dtype", DTYPES)
def test_sinks_gates_and_caps_count(dev, dtype):
    # leaving one out moves the oracle far beyond the tolerance that the library meets with it
    cfg = alone([V.attention(mlp=0), V.parallel(mlp=0)])
    w = V.weights(cfg, 14, U.identity_head(cfg))
    t = toks(cfg, 60)
    want = V.oracle_logits(cfg, w, t)
    tol = V.tolerance(cfg, w, t, want, dtype)
    zero = {n: np.zeros_like(w[n]) for n in w}
    for name, value in (("l0.mix.sink", U.to_bf16(np.full(6, -50.0))), ("l1.mix.left.g", zero["l1.mix.left.g"]), ("l1.mix.left.q.b", zero["l1.mix.left.q.b"]),
                        ("l1.mix.left.v.b", zero["l1.mix.left.v.b"]), ("l1.mix.right.g", zero["l1.mix.right.g"])):
        assert U.err(V.oracle_logits(cfg, dict(w, **{name: value}), t), want) > 2 * tol, name
    check(dev, cfg, w, t, dtype, [[60], [30, 2, 1]])
    # a sink far above and far below the scores, also across many splits of the keys
    for level in (-30.0, 12.0, 60.0):
        cfg = alone([V.attention(window=3000, mlp=0)])
        ident = U.identity_head(cfg)
        w = V.weights(cfg, 15, lambda n, a, level=level: np.full(a.shape, level) if n.endswith("sink") else ident(n, a))
        check(dev, cfg, w, toks(cfg, 330), dtype, [[330], [320, 1]])


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_memory_of_the_linear_attention(dev, dtype):
    # slow decay: the first tokens are still in the state hundreds of tokens later; the fast head forgets at once
    cfg = alone([V.parallel(b=V.right(2, 96, 16, [0.9995, 0.2]), mlp=0)])
    ident = U.identity_head(cfg)
    w = V.weights(cfg, 16, lambda n, a: np.zeros_like(a) if n.endswith("left.o") else ident(n, a))
    t = toks(cfg, 400)
    other = t.copy()
    other[0] = (t[0] + 1) % 64
    want = V.oracle_logits(cfg, w, t)
    assert U.err(V.oracle_logits(cfg, w, other)[-1], want[-1]) > 20 * U.TOL["float32"]
    m = V.gpu_model(dev, cfg, w, dtype)
    for sizes in ([400], [1, 399], [2], [301, 50, 1], [65, 63, 129]):
        assert U.err(U.run_portions(m, t, sizes), want) < U.TOL[dtype], sizes


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dev, dtype):
    cfg = mixed()
    check(dev, cfg, V.weights(cfg, 17), toks(cfg, 420), dtype, [20, 1])


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompt(dev, dtype):
    cfg = mixed()
    w = V.weights(cfg, 18)
    check(dev, cfg, w, toks(cfg, 1500), dtype, [[1500], [1023, 450, 2, 1]], max_seq_len=1536)


# ---- generation, session, command line --------------------------------------------------------------------

def greedy_ok(cfg, w, prompt, out, slack):
    """Every generated id is the oracle's choice for the sequence so far, up to `slack` of logit."""
    lg = V.oracle_logits(cfg, w, list(prompt) + list(out))[len(prompt) - 1:-1]
    gap = lg.max(-1) - lg[np.arange(len(out)), out]
    return np.all(gap <= slack * np.sqrt((lg * lg).mean())), float((gap > 0).mean())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("prompt_len", [1, 2, 40])
def test_greedy_generation(dev, dtype, prompt_len, tmp_path):
    cfg = mixed()
    w = V.weights(cfg, 24)
    V.write_checkpoint(str(tmp_path), cfg, w)
    m = models.load_model(dev, str(tmp_path), max_seq_len=256, dtype=dtype)
    prompt = [int(x) for x in toks(cfg, prompt_len, 4)]
    out = generate(m, prompt, 60)
    ok, changed = greedy_ok(cfg, w, prompt, out, 5 * U.TOL[dtype])
    assert ok and changed < 0.2
    assert generate(m, prompt, 60) == out and m.position == prompt_len - 1 + 60
    m.reset()
    step, nxt = [], m.forward(prompt)[1]
    for _ in range(60):
        step.append(int(nxt[0]))
        nxt = m.forward(step[-1:])[1]
    assert greedy_ok(cfg, w, prompt, step, 5 * U.TOL[dtype])[0]
    assert generate(m, prompt, 60, kb.SamplerConfig(temperature=0.0, top_k=8)) == out
    assert len(generate(m, prompt, 10, kb.SamplerConfig(temperature=1.0, seed=3))) == 10


@pytest.mark.parametrize("dtype", DTYPES)
def test_batched_greedy_generation(dev, dtype):
    cfg = mixed()
    w = V.weights(cfg, 25)
    m = V.gpu_model(dev, cfg, w, dtype, max_batch=2)
    p = np.stack([toks(cfg, 30, 1), toks(cfg, 30, 2)])
    m.forward(p[:, :-1], want_logits=False)
    out = m.generate_greedy(p[:, -1], 24)
    for i in range(2):
        assert greedy_ok(cfg, w, p[i], out[i], 5 * U.TOL[dtype])[0]


def test_session_rules(dev):
    cfg = mixed()
    w = V.weights(cfg, 26)
    m = V.gpu_model(dev, cfg, w, "float32", max_seq_len=32)
    t = toks(cfg, 40)
    m.forward(t[:30])
    for bad, code in ((lambda: m.forward(t[:3]), kb.ERR_CAPACITY), (lambda: m.truncate(10), kb.ERR_INVALID_ARGUMENT)):
        with pytest.raises(kb.FusorError) as e:
            bad()
        assert e.value.code == code
    m.truncate(0)
    assert U.err(U.run_portions(m, t[:30], [30], reset=False), V.oracle_logits(cfg, w, t[:30])) < U.TOL["float32"]
    # a model with attention layers only can be rewound
    cfg2 = V.config([V.attention(), V.attention(window=9)], loop=(0, 1, 2))
    w2 = V.weights(cfg2, 27)
    m2 = V.gpu_model(dev, cfg2, w2, "float32")
    t2 = toks(cfg2, 40)
    m2.forward(t2)
    m2.truncate(25)
    assert U.err(U.run_portions(m2, t2[25:], [15], reset=False), V.oracle_logits(cfg2, w2, t2)[25:]) < U.TOL["float32"]


@pytest.mark.parametrize("tensor", ["l0.mix.q", "l0.mix.sink", "l1.mix.left.k.norm", "l1.mix.left.v.b", "l1.mix.right.norm", "l1.mix.right.g", "l0.norm2", "loop.in"])
def test_wrong_shapes_are_refused(dev, tensor):
    cfg = V.config([V.attention(), V.parallel()], loop=(0, 1, 2))
    sh = V.shapes(cfg)
    bad = dict(sh, **{tensor: (sh[tensor][0] + 1,) + sh[tensor][1:]})
    with pytest.raises(kb.FusorError) as e:
        sofudra.build(dev, cfg, lambda n: (kb.BF16, bad[n], np.zeros(int(np.prod(bad[n])), np.uint16)), 64)
    assert e.value.code == kb.ERR_INVALID_SHAPE


def test_bad_configurations_and_missing_tensors_are_refused(dev):
    good = [e[0] for L in (V.attention(), V.parallel()) for e in sofudra.layer_entries(0, L)]
    make = dict(hidden=72, vocab=50, max_seq_len=64)
    for layers, stack in (([dict(good[0], kv_heads=4)], None), ([dict(good[0], rot_dim=7)], None), ([dict(good[0], rot_dim=26)], None),
                          ([dict(good[2], dim=600)], None), ([good[2]], None), ([good[0], dict(good[2], ffn=8)], None),
                          (good, dict(loop_start=1, loop_stop=3, loop_times=2)), (good, dict(loop_start=1, loop_stop=1, loop_times=1))):
        with pytest.raises(kb.FusorError):
            kb.HybridDecoder(dev, layers=layers, stack=stack, **make)
    m = kb.HybridDecoder(dev, layers=good, **make)
    with pytest.raises(kb.FusorError) as e:
        m.forward([1, 2])
    assert e.value.code == kb.ERR_INVALID_ARGUMENT


def test_poisoned_scratch(dev, monkeypatch):
    # activation buffers start as NaN: nothing may read what the pass did not write
    monkeypatch.setenv("FB200_POISON", "1")
    own = kb.Device(0)
    cfg = mixed()
    w = V.weights(cfg, 21)
    for dtype in DTYPES:
        check(own, cfg, w, toks(cfg, 60), dtype, [40, 3, 1])
    own.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_and_command_line(dtype, tmp_path):
    cfg = mixed()
    w = V.weights(cfg, 22)
    folder, out = str(tmp_path / "model"), str(tmp_path / "out")
    V.write_checkpoint(folder, cfg, w)
    os.makedirs(out)
    a, b = [int(x) for x in toks(cfg, 50, 1)], [int(x) for x in toks(cfg, 30, 2)]
    steps = [dict(entries=[dict(id="a", tokens=a[:40], want=[0, 39])], end=[]), dict(entries=[dict(id="a", tokens=a[40:42], want=[])], end=[]),
             dict(entries=[dict(id="a", tokens=a[42:], want=[7, 1])], end=["a"]), dict(entries=[dict(id="b", tokens=b[:29], want=[28])], end=[]),
             dict(entries=[dict(id="b", tokens=b[29:], want=[0])], end=["b"])]
    text = "".join(json.dumps(dict(step=i, **s)) + "\n" for i, s in enumerate(steps))
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", out, "--max-tokens", "64"],
                       input=text, capture_output=True, text=True)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(5)]
    la, lb = V.oracle_logits(cfg, w, a), V.oracle_logits(cfg, w, b)

    def read(i):
        return np.fromfile(os.path.join(out, f"{i}.f32"), "<f4").reshape(-1, cfg["vocab"])
    assert U.err(read(0), la[[0, 39]]) < U.TOL[dtype] and U.err(read(2), la[[49, 43]]) < U.TOL[dtype]
    assert U.err(read(3), lb[[28]]) < U.TOL[dtype] and U.err(read(4), lb[[29]]) < U.TOL[dtype]
    if dtype == "float32":
        r = subprocess.run([sys.executable, "-m", "kalosm_b200", "--model", folder, "--tokens", ",".join(map(str, b)), "--steps", "12",
                            "--dtype", dtype], capture_output=True, text=True, cwd=ROOT)
        assert r.returncode == 0, r.stderr
        assert greedy_ok(cfg, w, b, json.loads(r.stdout)["generated"], 1e-3)[0]
