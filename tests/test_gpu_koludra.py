"""GPU parity of the Koludra decoders (delta rule and latent attention layers) against the plain oracle."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import hybrid_util as U
import kalosm_b200 as kb
from gpu_util import dev  # noqa: F401
from kalosm_b200 import models
from kalosm_b200.__main__ import generate

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = ["float32", "bfloat16"]


def toks(cfg, n, seed=1):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n)


def check(dev, cfg, w, tokens, dtype, sizes, **kw):
    m = U.gpu_model(dev, cfg, w, dtype, **kw)
    got = U.run_portions(m, tokens, sizes)
    want = U.oracle_logits(cfg, w, tokens)
    e, tol = U.err(got, want), U.tolerance(cfg, w, tokens, want, dtype)
    assert e < tol, (e, tol)
    assert dev.status() == 0
    m.free()
    return got


# ---- products with dense weights --------------------------------------------------------------------------

@pytest.mark.parametrize("m,n,k", [(1, 130, 72), (1, 4099, 1024), (1, 20001, 264), (1, 9472, 64), (2, 65, 40), (5, 300, 264), (33, 129, 64), (64, 1000, 520),
                                   (130, 257, 2048), (257, 4000, 128), (700, 260, 1032)])
@pytest.mark.parametrize("ty", ["bf16", "f32"])
def test_dense_products(dev, m, n, k, ty):
    rng = np.random.default_rng(m + n + k)
    w = U.to_bf16(rng.standard_normal((n, k)))
    x = rng.standard_normal((m, k)).astype(np.float32)
    if ty == "bf16":
        q = kb.QMatrix.from_raw_bytes(dev, (n, k), w, kb.BF16)
        xr = x if m == 1 else U.from_bf16(U.to_bf16(x))  # one row keeps f32 activations
    else:
        q = kb.QMatrix.from_raw_bytes(dev, (n, k), U.from_bf16(w), kb.F32)
        xr = x
    want = xr.astype(np.float64) @ U.from_bf16(w).astype(np.float64).T
    got = dev.tensor(x).q_mat_mul(q).as_slice()
    assert np.linalg.norm(got - want) < 3e-6 * np.linalg.norm(want), np.linalg.norm(got - want) / np.linalg.norm(want)
    assert dev.status() == 0
    assert np.array_equal(q.dequantize().as_slice(), U.from_bf16(w))


# ---- each mechanism alone ------------------------------------------------------------------------------------

DELTAS = [dict(), dict(heads=1, kv_heads=1, dim=8, vdim=8, conv=1), dict(heads=6, kv_heads=1, dim=33, vdim=17, conv=2),
          dict(heads=3, kv_heads=3, dim=64, vdim=96, conv=3), dict(heads=4, kv_heads=2, dim=128, vdim=128, conv=4),
          dict(heads=2, kv_heads=2, dim=200, vdim=64, conv=6), dict(heads=2, kv_heads=1, dim=300, vdim=40, conv=4),
          dict(heads=2, kv_heads=1, dim=20, vdim=300, conv=4)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", range(len(DELTAS)))
def test_delta_layer(dev, dtype, shape):
    cfg = U.config([U.delta(ff=0, **DELTAS[shape])], width=88, vocab=88)
    w = U.weights(cfg, shape, U.identity_head(cfg))
    t = toks(cfg, 45)
    check(dev, cfg, w, t, dtype, [len(t)])
    check(dev, cfg, w, t, dtype, [17, 1])


LATENTS = [dict(), dict(heads=1, dim=8, rot=2, vdim=8, rank=8, window=1), dict(heads=5, dim=24, rot=8, vdim=48, rank=72, window=33, base=50.0),
           dict(heads=2, dim=20, rot=6, vdim=12, rank=30, window=7), dict(heads=4, dim=128, rot=64, vdim=128, rank=512, window=50),
           dict(heads=2, dim=64, rot=32, vdim=200, rank=136, window=64), dict(heads=3, dim=192, rot=72, vdim=72, rank=200, window=40, scale=0.2),
           dict(heads=17, dim=16, rot=16, vdim=16, rank=32, window=90)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", range(len(LATENTS)))
def test_latent_layer(dev, dtype, shape):
    cfg = U.config([U.latent(ff=0, **LATENTS[shape])], width=80, vocab=80)
    w = U.weights(cfg, 20 + shape, U.identity_head(cfg))
    t = toks(cfg, 150)
    check(dev, cfg, w, t, dtype, [len(t)])
    check(dev, cfg, w, t, dtype, [70, 3, 40, 2, 1])


@pytest.mark.parametrize("window,sizes", [(1, [700]), (70, [700]), (200, [650, 50]), (64, [300, 400]), (5000, [257, 443])], ids=str)
@pytest.mark.parametrize("vdim", [64, 128])
def test_latent_layer_many_rows(dev, window, sizes, vdim):
    # enough heads and rows for two groups of rows per CTA in the prompt kernel
    cfg = U.config([U.latent(ff=0, heads=64, dim=16, rot=16, vdim=vdim, rank=24, window=window)], width=64, vocab=64)
    w = U.weights(cfg, 40, U.identity_head(cfg))
    check(dev, cfg, w, toks(cfg, 700), "bfloat16", sizes, max_seq_len=704)


@pytest.mark.parametrize("dtype", DTYPES)
def test_layers_that_share_latents(dev, dtype):
    # the second reader has another window, other heads and value size; the third reads the first one's latents as well
    cfg = U.config([U.latent(window=12, ff=40), U.latent(kv_from=0, window=50, heads=4, dim=16, vdim=32, ff=0), U.delta(),
                    U.latent(kv_from=0, window=3, scale=0.4), U.latent(rank=24, rot=8, base=77.0), U.latent(kv_from=4, rank=24, rot=8, base=77.0)])
    w = U.weights(cfg, 3)
    t = toks(cfg, 120)
    for sizes in ([120], [50, 2, 30, 1]):
        check(dev, cfg, w, t, dtype, sizes)


@pytest.mark.parametrize("dtype", DTYPES)
def test_feed_forward_alone(dev, dtype):
    cfg = U.config([U.delta(ff=200)], width=64, vocab=64)
    ident = U.identity_head(cfg)
    w = U.weights(cfg, 5, lambda n, a: np.zeros_like(a) if n.endswith("mix.o") else ident(n, a))
    check(dev, cfg, w, toks(cfg, 37), dtype, [36, 1])


# ---- whole models: prompts, decoding, portions -----------------------------------------------------------------

def mixed(width=72, vocab=101):
    return U.config([U.delta(), U.latent(window=37), U.delta(heads=5, kv_heads=5, dim=40, vdim=16, conv=2, ff=0, name="delta_2"),
                     U.latent(kv_from=1, window=37, ff=0), U.delta(heads=6, kv_heads=3, dim=16, vdim=24, conv=5)], width, vocab)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[200], [1], [2], [3, 2, 5], [64, 64, 8], [16, 15, 17, 2], [130, 1], [199, 1]], ids=str)
def test_portions(dev, dtype, sizes):
    cfg = mixed()
    w = U.weights(cfg, 7)
    check(dev, cfg, w, toks(cfg, 200), dtype, sizes)


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_agree_with_each_other(dev, dtype):
    cfg = mixed()
    w = U.weights(cfg, 8)
    m = U.gpu_model(dev, cfg, w, dtype)
    t = toks(cfg, 140)
    whole = U.run_portions(m, t, [140])
    tol = U.tolerance(cfg, w, t, U.oracle_logits(cfg, w, t), dtype)
    for sizes in ([1], [33, 2, 1], [140]):
        assert U.err(U.run_portions(m, t, sizes), whole) < tol
    assert np.array_equal(U.run_portions(m, t, [140]), whole)  # the same cut gives the same bits


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [1, 2, 3, 4, 5, 6])
def test_first_tokens(dev, dtype, n):
    cfg = mixed()
    w = U.weights(cfg, 9)
    t = toks(cfg, n, seed=n)
    check(dev, cfg, w, t, dtype, [n])
    check(dev, cfg, w, t, dtype, [1])


@pytest.mark.parametrize("dtype", DTYPES)
def test_state_of_an_earlier_request_is_gone(dev, dtype):
    cfg = mixed()
    w = U.weights(cfg, 10)
    m = U.gpu_model(dev, cfg, w, dtype)
    a, b = toks(cfg, 90, 1), toks(cfg, 60, 2)
    fresh = U.run_portions(m, b, [40, 1])
    U.run_portions(m, a, [90])
    assert np.array_equal(U.run_portions(m, b, [40, 1]), fresh)
    # also after decoding, and for a request that starts with single tokens
    U.run_portions(m, a, [50, 1])
    single = U.run_portions(m, b[:20], [1])
    m2 = U.gpu_model(dev, cfg, w, dtype)
    assert np.array_equal(U.run_portions(m2, b[:20], [1]), single)


@pytest.mark.parametrize("dtype", DTYPES)
def test_batch_equals_each_sequence_alone(dev, dtype):
    cfg = mixed()
    w = U.weights(cfg, 11)
    m = U.gpu_model(dev, cfg, w, dtype, max_batch=3)
    seqs = np.stack([toks(cfg, 80, s) for s in (1, 2, 3)])
    want = np.stack([U.oracle_logits(cfg, w, s) for s in seqs])
    got = []
    for a, b in [(0, 50), (50, 52), (52, 70)] + [(i, i + 1) for i in range(70, 80)]:
        m.forward(seqs[:, a:b], want_logits=False)
        got.append(m.logits_at(range(3 * (b - a))).reshape(3, b - a, -1))
    got = np.concatenate(got, axis=1)
    for i in range(3):
        assert U.err(got[i], want[i]) < U.TOL[dtype], i


@pytest.mark.parametrize("dtype", DTYPES)
def test_odd_sizes(dev, dtype):
    cfg = U.config([U.delta(heads=3, kv_heads=1, dim=9, vdim=7, conv=7, ff=37), U.latent(heads=3, dim=7, rot=2, vdim=5, rank=11, window=9, ff=0),
                    U.latent(heads=1, dim=5, rot=2, vdim=3, rank=11, window=31, kv_from=1, ff=13)], width=75, vocab=53)
    w = U.weights(cfg, 23)
    for sizes in ([90], [40, 2, 31, 1]):
        check(dev, cfg, w, toks(cfg, 90), dtype, sizes)


def test_larger_sizes(dev):
    # sizes of the kernels that real layers use: 128-wide heads, 512-wide latents, many weight tiles
    cfg = U.config([U.delta(heads=8, kv_heads=4, dim=128, vdim=128, conv=4, ff=1024),
                    U.latent(heads=8, dim=128, rot=64, vdim=128, rank=512, window=130, ff=1024)], width=1024, vocab=700)
    w = U.weights(cfg, 12)
    t = toks(cfg, 300)
    check(dev, cfg, w, t, "bfloat16", [257, 41, 1])
    check(dev, cfg, w, t[:80], "float32", [70, 1])


# ---- distances that have to show: window edges, far keys, far memory ---------------------------------------

def marker_model(window, width=64, rot=8):
    """One latent layer in which token 1 (a query) scores high on token 0 (a key) and flat on everything else, so that
    whether that key is visible decides the query's output."""
    cfg = U.config([U.latent(heads=2, dim=16, rot=rot, vdim=16, rank=24, window=window, ff=0)], width, width)
    ident = U.identity_head(cfg)

    def edit(name, a):
        if name == "embed":
            a = np.random.default_rng(5).standard_normal(a.shape) * 0.3
            a[:, :2] = 0.0
            a[0, 0] = a[1, 1] = 6.0
            return a
        if name.endswith("mix.dkv"):
            a = a.copy()
            a[:24, :2] = 0.0
            a[0, 0] = 4.0  # the key token's latent points along the first axis
            return a
        if name.endswith("mix.uk"):
            a = a * 0.2
            for h in range(2):
                a[h * 16:(h + 1) * 16, 0] = 0.0
                a[h * 16, 0] = 3.0
            return a
        if name.endswith("mix.q"):
            a = a.reshape(2, 16 + rot, -1) * 0.2
            a[:, :, :2] = 0.0
            a[:, 0, 1] = 4.0  # the query token looks along it
            return a.reshape(-1, a.shape[-1])
        return ident(name, a)
    return cfg, U.weights(cfg, 13, edit)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 2, 15, 63, 64, 65, 127, 129])
def test_window_edges(dev, dtype, window):
    cfg, w = marker_model(window)
    m = U.gpu_model(dev, cfg, w, dtype)
    seen = {}
    for dist in sorted({max(0, window - 2), window - 1, window, window + 1, window + 70}):
        for at in (dist + 1, dist + 66):  # position of the query
            t = np.random.default_rng(at).integers(2, cfg["vocab"], at + 3)
            t[at] = 1
            if dist:
                t[at - dist] = 0
            want = U.oracle_logits(cfg, w, t)
            for sizes in ([len(t)], [at, 1], [max(1, at - 5), 2, 3]):
                got = U.run_portions(m, t, sizes)
                assert U.err(got, want) < U.TOL[dtype], (dist, at, sizes)
            seen.setdefault(dist, []).append(want[at])
    # the test has teeth: a key just inside changes the query's row far beyond the tolerance
    if window > 1:
        t = np.random.default_rng(3).integers(2, cfg["vocab"], window + 3)
        t[-1] = 1
        base = U.oracle_logits(cfg, w, t)[-1]
        inside, outside = t.copy(), t.copy()
        inside[-window] = 0
        outside[-window - 1] = 0
        assert U.err(U.oracle_logits(cfg, w, inside)[-1], base) > 0.3
        assert U.err(U.oracle_logits(cfg, w, outside)[-1], base) < 1e-9


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_key_among_hundreds(dev, dtype):
    cfg, w = marker_model(1000)
    m = U.gpu_model(dev, cfg, w, dtype, max_seq_len=1024)
    for at, key in ((700, 0), (700, 63), (700, 64), (511, 511 - 447), (699, 320)):
        t = np.random.default_rng(key).integers(2, cfg["vocab"], at + 1)
        t[at], t[key] = 1, 0
        want = U.oracle_logits(cfg, w, t)
        without = t.copy()
        without[key] = 2
        assert U.err(want[at], U.oracle_logits(cfg, w, without)[at]) > 0.3
        for sizes in ([at + 1], [at, 1], [300, 200, 150, 2]):
            m.reset()
            got = U.run_portions(m, t, sizes)
            assert U.err(got[at], want[at]) < U.TOL[dtype], (at, key, sizes)


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_memory_of_the_delta_rule(dev, dtype):
    # slow decay: the first tokens are still in the state hundreds of tokens later
    cfg = U.config([U.delta(heads=2, kv_heads=2, dim=96, vdim=16, conv=3, ff=0)], 64, 64)
    ident = U.identity_head(cfg)

    def edit(name, a):
        if name.endswith("A_log"):
            return np.full_like(a, -9.0)
        if name.endswith("mix.b"):
            return a * 0.3
        return ident(name, a)
    w = U.weights(cfg, 14, edit)
    t = toks(cfg, 400)
    other = t.copy()
    other[0] = (t[0] + 1) % 64
    want = U.oracle_logits(cfg, w, t)
    assert U.err(U.oracle_logits(cfg, w, other)[-1], want[-1]) > 20 * U.TOL["float32"]
    m = U.gpu_model(dev, cfg, w, dtype)
    for sizes in ([400], [1, 399], [2], [301, 50, 1]):
        assert U.err(U.run_portions(m, t, sizes), want) < U.TOL[dtype], sizes


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dev, dtype):
    cfg = mixed()
    w = U.weights(cfg, 15)
    check(dev, cfg, w, toks(cfg, 420), dtype, [20, 1])


# ---- generation, session, command line --------------------------------------------------------------------

def greedy_ok(cfg, w, prompt, out, slack):
    """Every generated id is the oracle's choice for the sequence so far, up to `slack` of logit."""
    lg = U.oracle_logits(cfg, w, list(prompt) + list(out))[len(prompt) - 1:-1]
    gap = lg.max(-1) - lg[np.arange(len(out)), out]
    return np.all(gap <= slack * np.sqrt((lg * lg).mean())), float((gap > 0).mean())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("prompt_len", [1, 2, 40])
def test_greedy_generation(dev, dtype, prompt_len, tmp_path):
    cfg = mixed()
    w = U.weights(cfg, 16)
    U.write_checkpoint(str(tmp_path), cfg, w)
    m = models.load_model(dev, str(tmp_path), max_seq_len=256, dtype=dtype)
    prompt = [int(x) for x in toks(cfg, prompt_len, 4)]
    out = generate(m, prompt, 60)
    ok, changed = greedy_ok(cfg, w, prompt, out, 5 * U.TOL[dtype])
    assert ok and changed < 0.2
    assert generate(m, prompt, 60) == out and m.position == prompt_len - 1 + 60
    # stepping through forward gives the same ids
    m.reset()
    step, nxt = [], m.forward(prompt)[1]
    for _ in range(60):
        step.append(int(nxt[0]))
        nxt = m.forward(step[-1:])[1]
    assert greedy_ok(cfg, w, prompt, step, 5 * U.TOL[dtype])[0]
    # a sampler at temperature 0 follows the greedy ids
    assert generate(m, prompt, 60, kb.SamplerConfig(temperature=0.0, top_k=8)) == out
    assert len(generate(m, prompt, 10, kb.SamplerConfig(temperature=1.0, seed=3))) == 10


def test_batched_greedy_generation(dev):
    cfg = mixed()
    w = U.weights(cfg, 17)
    m = U.gpu_model(dev, cfg, w, "float32", max_batch=2)
    p = np.stack([toks(cfg, 30, 1), toks(cfg, 30, 2)])
    m.forward(p[:, :-1], want_logits=False)
    out = m.generate_greedy(p[:, -1], 24)
    for i in range(2):
        assert greedy_ok(cfg, w, p[i], out[i], 1e-3)[0]


def test_session_rules(dev):
    cfg = mixed()
    w = U.weights(cfg, 18)
    m = U.gpu_model(dev, cfg, w, "float32", max_seq_len=32)
    t = toks(cfg, 40)
    m.forward(t[:30])
    for bad, code in ((lambda: m.forward(t[:3]), kb.ERR_CAPACITY), (lambda: m.truncate(10), kb.ERR_INVALID_ARGUMENT),
                      (lambda: m.logits_at([30]), kb.ERR_INVALID_ARGUMENT),
                      (lambda: m.set_tensor("mix_q", 0, kb.F32, (1, 1), np.zeros(1, np.float32)), kb.ERR_INVALID_ARGUMENT)):
        with pytest.raises(kb.FusorError) as e:
            bad()
        assert e.value.code == code
    m.truncate(30)
    m.truncate(0)
    assert U.err(U.run_portions(m, t[:30], [30], reset=False), U.oracle_logits(cfg, w, t[:30])) < U.TOL["float32"]
    # a model with latent layers only can be rewound
    cfg2 = U.config([U.latent(), U.latent(kv_from=0)])
    w2 = U.weights(cfg2, 19)
    m2 = U.gpu_model(dev, cfg2, w2, "float32")
    t2 = toks(cfg2, 40)
    m2.forward(t2)
    m2.truncate(25)
    assert U.err(U.run_portions(m2, t2[25:], [15], reset=False), U.oracle_logits(cfg2, w2, t2)[25:]) < U.TOL["float32"]


def test_wrong_shapes_and_missing_tensors_are_refused(dev):
    cfg = U.config([U.latent()])
    w = U.weights(cfg)
    sh = U.shapes(cfg)
    import kalosm_b200.koludra as K
    bad = dict(sh, **{"l0.mix.uk": (sh["l0.mix.uk"][0], sh["l0.mix.uk"][1] + 1)})
    with pytest.raises(kb.FusorError) as e:
        K.build(dev, cfg, lambda n: (kb.BF16, bad[n], np.zeros(int(np.prod(bad[n])), np.uint16)), 64)
    assert e.value.code == kb.ERR_INVALID_SHAPE
    m = kb.HybridDecoder(dev, hidden=72, vocab=50, layers=[K.layer_config(0, cfg["layers"][0])], max_seq_len=64)
    with pytest.raises(kb.FusorError) as e:
        m.forward([1, 2])
    assert e.value.code == kb.ERR_INVALID_ARGUMENT
    with pytest.raises(kb.FusorError):
        kb.HybridDecoder(dev, hidden=72, vocab=50, layers=[K.layer_config(0, U.latent(kv_from=0))], max_seq_len=64)


def test_poisoned_scratch(dev, monkeypatch):
    # activation buffers start as NaN: nothing may read what the pass did not write
    monkeypatch.setenv("FB200_POISON", "1")
    own = kb.Device(0)
    cfg = mixed()
    w = U.weights(cfg, 21)
    for dtype in DTYPES:
        check(own, cfg, w, toks(cfg, 60), dtype, [40, 3, 1])
    own.close()


def test_logits_of_chosen_rows_of_a_llama(dev):
    from llama_util import build_models, tiny_cfg
    cfg = tiny_cfg()
    gpu, cpu = build_models(dev, cfg, batch=1, seed=3)
    t = np.random.default_rng(1).integers(0, cfg["vocab"], (1, 9), dtype=np.uint32)
    gpu.forward(t)
    got = gpu.logits_at(range(9))
    want = np.concatenate([cpu.forward(t[:, i:i + 1]) for i in range(9)])
    assert U.err(got, want) < 4e-3


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_program(dtype, tmp_path):
    cfg = mixed()
    w = U.weights(cfg, 22)
    folder, out = str(tmp_path / "model"), str(tmp_path / "out")
    U.write_checkpoint(folder, cfg, w)
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
    la, lb = U.oracle_logits(cfg, w, a), U.oracle_logits(cfg, w, b)

    def read(i):
        return np.fromfile(os.path.join(out, f"{i}.f32"), "<f4").reshape(-1, cfg["vocab"])
    assert U.err(read(0), la[[0, 39]]) < U.TOL[dtype] and U.err(read(2), la[[49, 43]]) < U.TOL[dtype]
    assert U.err(read(3), lb[[28]]) < U.TOL[dtype] and U.err(read(4), lb[[29]]) < U.TOL[dtype]
    assert not os.path.exists(os.path.join(out, "1.f32"))
    if dtype == "float32":
        r = subprocess.run([sys.executable, "-m", "kalosm_b200", "--model", folder, "--tokens", ",".join(map(str, b)), "--steps", "12",
                            "--dtype", dtype], capture_output=True, text=True, cwd=ROOT)
        assert r.returncode == 0, r.stderr
        assert greedy_ok(cfg, w, b, json.loads(r.stdout)["generated"], 1e-3)[0]
