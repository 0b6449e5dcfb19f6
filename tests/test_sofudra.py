"""Sofudra without a GPU: configuration, tensor names, registry, and the oracle's own mechanisms."""
import math
import os

import numpy as np
import pytest

import hybrid_util as U
import kalosm_b200 as kb
import sofudra_util as V
from kalosm_b200 import models, sofudra
from kalosm_b200.checkpoint import ConfigError
from oracle import hybrid as HY
from oracle import sofudra as SO


def test_layer_entries_carry_every_constant():
    (a, names, decay), = sofudra.layer_entries(0, V.attention(heads=6, kv_heads=3, dim=20, vdim=12, window=7, scale=0.3, mlp=9, name="attention_2",
                                                             rot=V.rotary(10, 500.0, 2.5, 96, 20.0, 2.0)))
    assert a == dict(mixer=kb.MIX_ATTENTION, heads=6, kv_heads=3, dim=20, vdim=12, window=7, scale=0.3, softcap=0.0, ffn=9, two_norms=1,
                     ffn_act=kb.FFN_GELU, rot_dim=10, rope_base=500.0, yarn_factor=2.5, yarn_fast=20.0, yarn_slow=2.0, yarn_original=96,
                     parts=kb.ATTN_QK_NORM | kb.ATTN_SINK)
    assert decay is None and "mix.sink" in names and "mix.g" not in names and "norm2" in names
    (l, ln, _), (r, rn, decay) = sofudra.layer_entries(1, V.parallel(V.left(softcap=2.5), V.right(2, 8, 4, [0.5, 0.25]), 0.3, 0.6, mlp=0))
    assert l == dict(mixer=kb.MIX_ATTENTION, heads=4, kv_heads=2, dim=16, vdim=24, window=0, scale=0.25, softcap=2.5, out_scale=0.3,
                     parts=kb.ATTN_QK_NORM | kb.ATTN_BIAS | kb.ATTN_GATE)
    assert r == dict(mixer=kb.MIX_LINEAR, beside=1, heads=2, dim=8, vdim=4, out_scale=0.6) and decay == [0.5, 0.25]
    assert "mix.left.v.b" in ln and "mix.left.sink" not in ln and "norm2" not in ln and "mix.right.norm" in rn
    s = sofudra.stack(V.config([V.parallel()] * 4, loop=(1, 3, 2), mult=0.2, embed=5.0, cap=7.0))
    assert s == dict(embed_scale=5.0, residual_mult=0.2, logit_softcap=7.0, loop_start=1, loop_stop=3, loop_times=2)
    assert sofudra.stack({"layers": []}) == dict(embed_scale=1.0, residual_mult=1.0, logit_softcap=0.0, loop_start=0, loop_stop=0, loop_times=0)


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0].update(type="mamba"), lambda c: c["layers"][0]["mlp"].update(kind="moe"),
    lambda c: c["layers"][1]["mixer"]["right"].update(decay=[0.5]), lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0.0)])
def test_unknown_layers_are_refused(change):
    cfg = V.config([V.attention(), V.parallel()])
    change(cfg)
    with pytest.raises(ConfigError):
        [sofudra.layer_entries(i, L) for i, L in enumerate(cfg["layers"])]


def test_tensor_names_cover_the_configuration():
    cfg = V.config([V.attention(), V.parallel(mlp=0), V.attention(mlp=0), V.parallel(name="parallel_2")], loop=(0, 2, 2))
    names = {"embed", "head", "final.norm", "loop.in"}
    for i, L in enumerate(cfg["layers"]):
        for _, tensors, _ in sofudra.layer_entries(i, L):
            names |= {f"l{i}.{s}" for s in tensors}
            assert all(t in kb.Decoder.TENSORS for t in tensors.values())
    assert names == set(V.shapes(cfg))


def test_registry_picks_the_loader_by_architecture(tmp_path):
    cfg = V.config([V.attention()])
    V.write_checkpoint(str(tmp_path), cfg, V.weights(cfg))
    assert models.architecture(str(tmp_path)) == "Sofudra" and models.REGISTRY["Sofudra"] is sofudra.load and "Sofudra" in models.DENSE
    assert os.path.exists(tmp_path / "model.safetensors")
    with pytest.raises(ConfigError):
        models.REGISTRY["Koludra"](None, str(tmp_path))


# ---- the oracle's mechanisms against independent statements of the same equations

def test_oracle_gelu_and_softcap():
    z = np.linspace(-4, 4, 81)
    exact = np.array([0.5 * x * (1 + math.erf(x / math.sqrt(2))) for x in z])
    assert np.abs(SO.gelu_tanh(z) - exact).max() < 1e-3 and SO.gelu_tanh(np.zeros(1))[0] == 0
    assert np.allclose(SO.softcap(z, 1e6), z) and abs(SO.softcap(np.array([1e9]), 3.0)[0] - 3.0) < 1e-12


def test_oracle_yarn_keeps_fast_dimensions_and_divides_slow_ones():
    plain, one = SO.rotary_frequencies(V.rotary(64, 10000.0))
    f, mul = SO.rotary_frequencies(V.rotary(64, 10000.0, 4.0, 256, 16.0, 1.0))
    assert one == 1.0 and np.isclose(mul, 0.1 * math.log(4.0) + 1.0)
    turns = 256 * plain / (2 * math.pi)  # turns of a dimension inside the original context
    assert np.allclose(f[turns > 20], plain[turns > 20]) and np.allclose(f[turns < 0.7], plain[turns < 0.7] / 4)
    mid = (turns < 14) & (turns > 1.5)
    assert mid.any() and np.all(f[mid] < plain[mid]) and np.all(f[mid] > plain[mid] / 4)
    # the bounds meet: one step instead of a ramp
    g, _ = SO.rotary_frequencies(V.rotary(8, 10.0, 2.0, 4, 1e6, 1e5))
    assert np.all(np.isfinite(g))


def test_oracle_rotation_is_a_relative_position():
    rng = np.random.default_rng(3)
    q, k = rng.standard_normal((1, 1, 10)), rng.standard_normal((1, 1, 10))
    rot = V.rotary(8, 100.0, 3.0)
    mul = SO.rotary_frequencies(rot)[1]

    def score(i, j):
        return float((SO.rotate(q, np.array([i]), rot) * SO.rotate(k, np.array([j]), rot)).sum())
    assert np.isclose(score(7, 3), score(104, 100)) and not np.isclose(score(7, 3), score(7, 4))
    x = SO.rotate(q, np.array([5]), rot)
    assert np.array_equal(x[..., 8:], q[..., 8:]) and np.isclose((x[..., :8] ** 2).sum(), (q[..., :8] ** 2).sum() * mul ** 2)


def test_oracle_sink_window_and_cap():
    rng = np.random.default_rng(4)
    q, k, v = rng.standard_normal((6, 4)), rng.standard_normal((6, 4)), rng.standard_normal((6, 3))
    # a sink is a key of that score with a zero value
    s = q[5] @ k.T * 0.5
    w = np.exp(np.append(s, 0.7))
    assert np.allclose(SO.attend(q, k, v, 0.5, sink=0.7)[5], (w[:6] @ v) / w.sum())
    assert np.allclose(SO.attend(q, k, v, 0.5, sink=-1e9), SO.attend(q, k, v, 0.5))
    w = np.exp(2.0 * np.tanh(s[4:] / 2.0))
    assert np.allclose(SO.attend(q, k, v, 0.5, window=2, cap=2.0)[5], w @ v[4:] / w.sum())
    assert np.allclose(SO.attend(q, k, v, 0.5, window=1), v)


def test_oracle_linear_attention_closed_form():
    rng = np.random.default_rng(5)
    q, k, v = rng.standard_normal((7, 2, 5)), rng.standard_normal((7, 2, 5)), rng.standard_normal((7, 2, 3))
    decay = np.array([0.5, 0.9])
    o, S = SO.linear_attention(q, k, v, decay)
    i = np.arange(7)
    for h in range(2):
        w = np.tril(decay[h] ** np.maximum(i[:, None] - i[None, :], 0)) * (q[:, h] @ k[:, h].T)
        assert np.allclose(o[:, h], w @ v[:, h])
    head, mid = SO.linear_attention(q[:4], k[:4], v[:4], decay)
    tail, end = SO.linear_attention(q[4:], k[4:], v[4:], decay, mid)
    assert np.allclose(np.concatenate([head, tail]), o) and np.allclose(end, S)


def test_oracle_schedule_of_a_loop():
    cfg = V.config([V.attention()] * 5, loop=(1, 3, 2))
    assert SO.schedule(cfg) == [(0, False), (1, True), (2, False), (1, True), (2, False), (3, False), (4, False)]
    assert SO.schedule(V.config([V.attention()] * 2)) == [(0, False), (1, False)]


def test_oracle_is_causal_and_its_factors_count():
    cfg = V.config([V.parallel(), V.attention(mlp=0), V.parallel(mlp=0)], loop=(1, 2, 3))
    w = V.weights(cfg, 4)
    toks = np.random.default_rng(5).integers(0, cfg["vocab"], 30)
    full = V.oracle_logits(cfg, w, toks)
    assert np.allclose(V.oracle_logits(cfg, w, toks[:17]), full[:17])
    for change in (dict(residual_mult=0.9), dict(logit_softcap=3.0), dict(embedding={"scale": 1.0}), dict(loop=dict(start=1, stop=2, times=2)),
                   dict(norm={"eps": 0.5})):
        assert U.err(V.oracle_logits(dict(cfg, **change), w, toks), full) > 1e-2
    # without mixer output a layer adds its feed-forward of the second norm
    one = V.config([V.attention()], cap=0.0)
    z = V.weights(one, 6, lambda n, a: np.zeros_like(a) if n.endswith("mix.o") else None)
    t = V.oracle_model(one, z)["tensors"]
    x = t["embed"][toks].astype(np.float64) * 3.0
    x = x + 0.45 * SO.dense_ff(HY.rms_norm(x, t["l0.norm2"], 1e-5), lambda n: t["l0.mlp." + n].astype(np.float64))
    assert np.allclose(V.oracle_logits(one, z, toks), HY.rms_norm(x, t["final.norm"], 1e-5) @ t["head"].T.astype(np.float64))
