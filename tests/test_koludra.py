"""Koludra without a GPU: configuration, checkpoint files, registry, and the oracle's own mechanisms."""
import json
import subprocess
import sys
import os

import numpy as np
import pytest

import hybrid_util as U
import kalosm_b200 as kb
from kalosm_b200 import koludra, models
from kalosm_b200.safetensors import SafetensorsError, SafetensorsFile, write_safetensors
from oracle import hybrid as HY

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def test_layer_configs_carry_every_constant():
    d = koludra.layer_config(0, U.delta(heads=6, kv_heads=3, dim=20, vdim=12, conv=5, ff=0, name="delta_2"))
    assert d == dict(mixer=kb.MIX_DELTA, ffn=0, heads=6, kv_heads=3, dim=20, vdim=12, conv=5)
    a = koludra.layer_config(3, U.latent(heads=2, dim=8, rot=4, vdim=6, rank=10, window=7, base=500.0, scale=0.3, kv_from=1, ff=9))
    assert a == dict(mixer=kb.MIX_LATENT, ffn=9, heads=2, dim=8, rot_dim=4, vdim=6, kv_rank=10, window=7, kv_from=1,
                     rope_base=500.0, scale=0.3)
    assert "mix.dkv" not in koludra.layer_tensors(U.latent(kv_from=1)) and "mix.dkv" in koludra.layer_tensors(U.latent())
    assert "mlp.up" not in koludra.layer_tensors(U.delta(ff=0))


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0].update(type="mamba"), lambda c: c["layers"][0]["mlp"].update(kind="moe"),
    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=2)])
def test_unknown_layers_are_refused(change):
    cfg = U.config([U.delta(), U.latent()])
    change(cfg)
    with pytest.raises(koludra.ConfigError):
        [koludra.layer_config(i, L) for i, L in enumerate(cfg["layers"])]


def test_tensor_names_cover_the_configuration():
    cfg = U.config([U.delta(), U.latent(ff=0), U.delta(ff=0, name="delta_2"), U.latent(kv_from=1)])
    names = {"embed", "head", "final.norm"} | {f"l{i}.{s}" for i, L in enumerate(cfg["layers"]) for s in koludra.layer_tensors(L)}
    assert names == set(U.shapes(cfg))
    assert all(t in kb.Decoder.TENSORS for L in cfg["layers"] for t in koludra.layer_tensors(L).values())


def test_safetensors_round_trip_and_refusals(tmp_path):
    p = str(tmp_path / "a.safetensors")
    a, b = np.arange(6, dtype=np.float32), np.arange(4, dtype=np.uint16)
    write_safetensors(p, [("a", "F32", (2, 3), a), ("b", "BF16", (4,), b), ("t", "I32", (1,), np.int32([7]))])
    f = SafetensorsFile(p)
    ty, shape, raw = f.raw("a")
    assert (ty, shape) == (kb.F32, (2, 3)) and np.array_equal(np.frombuffer(bytes(raw), np.float32), a)
    ty, shape, raw = f.raw("b")
    assert (ty, shape) == (kb.BF16, (4,)) and np.array_equal(np.frombuffer(bytes(raw), np.uint16), b)
    for name in ("t", "missing"):
        with pytest.raises(SafetensorsError):
            f.raw(name)
    with open(p, "r+b") as fh:
        fh.truncate(os.path.getsize(p) - 1)
    with pytest.raises(SafetensorsError):
        SafetensorsFile(p)


def test_registry_picks_the_loader_by_architecture(tmp_path):
    folder = str(tmp_path / "m")
    cfg = U.config([U.delta()])
    U.write_checkpoint(folder, cfg, U.weights(cfg))
    assert models.architecture(folder) == "Koludra" and models.REGISTRY["Koludra"] is koludra.load
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(dict(cfg, architecture="Other"), f)
    with pytest.raises(ValueError, match="Other"):
        models.load_model(None, folder)


def test_command_lines_have_help():
    for cmd in ([os.path.join(ROOT, "bin", "trace_run"), "--help"], [sys.executable, "-m", "kalosm_b200", "--help"]):
        r = subprocess.run(cmd, capture_output=True, text=True, cwd=ROOT)
        assert r.returncode == 0 and "--model" in r.stdout, r.stderr


def test_trace_replay_feeds_one_request_at_a_time(tmp_path):
    from kalosm_b200 import trace
    calls = []

    class Fake:
        vocab = 3

        def reset(self):
            calls.append("reset")

        def forward(self, tokens, want_logits=True):
            calls.append(list(tokens))

        def logits_at(self, rows):
            return np.array([[r, r, r] for r in rows], np.float32).reshape(-1, 3)
    lines = ['{"step": 0, "entries": [{"id": "a", "tokens": [1, 2, 3], "want": [0, 2]}], "end": []}',
             '{"step": 1, "entries": [{"id": "a", "tokens": [4], "want": []}], "end": ["a"]}',
             '{"step": 2, "entries": [{"id": "b", "tokens": [5, 6], "want": [1]}], "end": ["b"]}']
    done = []
    trace.replay(Fake(), lines, str(tmp_path), done.append)
    assert done == ["done 0", "done 1", "done 2"]
    assert np.array_equal(np.fromfile(tmp_path / "0.f32", "<f4"), [0, 0, 0, 2, 2, 2])
    assert not (tmp_path / "1.f32").exists() and (tmp_path / "2.f32").exists()
    assert [c for c in calls if c != "reset"] == [[1, 2, 3], [4], [5, 6]]
    with pytest.raises(RuntimeError):
        trace.replay(Fake(), [lines[0], lines[2]], str(tmp_path), done.append)


# ---- the oracle's mechanisms against independent statements of the same equations

def test_oracle_conv_equals_numpy_convolve():
    rng = np.random.default_rng(1)
    x, w = rng.standard_normal((9, 3)), rng.standard_normal((3, 4))
    for c in range(3):
        # correlation with the last column on the current token = convolution with the reversed taps
        assert np.allclose(HY.causal_conv(x, w)[:, c], np.convolve(x[:, c], w[c, ::-1])[:9])


def test_oracle_delta_rule_closed_forms():
    rng = np.random.default_rng(2)
    T, D = 5, 6
    k = np.linalg.qr(rng.standard_normal((D, D)))[0][:T][:, None, :]  # orthonormal keys
    v, q = rng.standard_normal((T, 1, 3)), rng.standard_normal((T, 1, D))
    one = np.ones((T, 1))
    o, S = HY.delta_rule(q, k, v, one, one)
    # orthonormal keys, full writes, no decay: the state is the plain sum of outer products
    assert np.allclose(S[0], sum(np.outer(k[t, 0], v[t, 0]) for t in range(T)))
    assert np.allclose(o[-1, 0], S[0].T @ q[-1, 0])
    # writing the same key twice replaces the value
    o, S = HY.delta_rule(np.stack([k[0]] * 2), np.stack([k[0]] * 2), v[:2], one[:2], one[:2])
    assert np.allclose(S[0].T @ k[0, 0], v[1, 0])
    # decay acts before the write
    g = np.array([[1.0], [0.25]])
    o, S = HY.delta_rule(k[:2], k[:2], v[:2], g, one[:2])
    assert np.allclose(S[0].T @ k[0, 0], 0.25 * v[0, 0]) and np.allclose(o[1, 0], v[1, 0])


def test_oracle_rotation_is_a_relative_position():
    rng = np.random.default_rng(3)
    q, k = rng.standard_normal(8), rng.standard_normal(8)

    def score(i, j):
        a = HY.rotate_half(q[None], np.array([i]), 100.0, 8)[0]
        b = HY.rotate_half(k[None], np.array([j]), 100.0, 8)[0]
        return a @ b
    assert np.isclose(score(7, 3), score(104, 100)) and not np.isclose(score(7, 3), score(7, 4))
    part = HY.rotate_half(q[None], np.array([5]), 100.0, 4)[0]
    assert np.array_equal(part[4:], q[4:]) and not np.allclose(part[:4], q[:4])


def test_oracle_window():
    s = np.zeros((6, 6))
    p = HY.window_softmax(s, 3)
    assert np.allclose(p[5], [0, 0, 0, 1 / 3, 1 / 3, 1 / 3]) and np.allclose(p[1, :2], 0.5) and np.allclose(p[0, 0], 1)


def test_oracle_is_causal_and_layers_add_in_parallel():
    cfg = U.config([U.delta(), U.latent(ff=0), U.latent(kv_from=1)])
    w = U.weights(cfg, 4)
    toks = np.random.default_rng(5).integers(0, cfg["vocab"], 30)
    full = U.oracle_logits(cfg, w, toks)
    assert np.allclose(U.oracle_logits(cfg, w, toks[:17]), full[:17])
    # without mixer output (o = 0) a layer adds its feed-forward of the same norm
    z = dict(w)
    for i in range(3):
        z[f"l{i}.mix.o"] = np.zeros_like(w[f"l{i}.mix.o"])
    t = U.oracle_model(cfg, z)["tensors"]
    x = t["embed"][toks].astype(np.float64)
    for i in (0, 2):
        h = HY.rms_norm(x, t[f"l{i}.norm1"], cfg["norm"]["eps"])
        x = x + HY.dense_ff(h, lambda n, i=i: t[f"l{i}.mlp.{n}"].astype(np.float64))
    want = HY.rms_norm(x, t["final.norm"], cfg["norm"]["eps"]) @ t["head"].T
    assert np.allclose(U.oracle_logits(cfg, z, toks), want)
