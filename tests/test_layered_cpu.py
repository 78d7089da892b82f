"""Layered decoders, what needs no GPU: the plain oracle against independent restatements of its mechanisms, the
configuration reader, the registry."""
import copy
import json
import math

import numpy as np
import pytest

from oracle import layered as L


CFG = {"architecture": "Vunolorn", "vocab": 61, "width": 40, "embedding": {"scale": 5.0}, "norm": {"eps": 1e-6}, "layers": [
    {"type": "mamba1", "mixer": {"conv": 3, "dt_rank": 5, "inner": 44, "state": 6}, "mlp": {"kind": "dense", "ff": 28}},
    {"type": "delta", "mixer": {"conv": 2, "dim": 12, "heads": 4, "kv_heads": 2, "vdim": 10}, "mlp": None},
    {"type": "parallel", "mixer": {"left": {"dim": 16, "heads": 4, "kv_heads": 2, "rot": {"base": 100.0, "dims": 8}, "scale": 0.4, "vdim": 12},
                                   "left_scale": 0.7, "right": {"width": 20}, "right_scale": 1.3}, "mlp": None}]}


def test_config_reader_accepts_and_explains(pkg):
    assert pkg.Decoder.check_config(CFG) == ""

    def broken(change):
        c = copy.deepcopy(CFG)
        change(c)
        return pkg.Decoder.check_config(c)

    assert "architecture" in broken(lambda c: c.update(architecture="Other"))
    assert "eps" in broken(lambda c: c["norm"].pop("eps"))
    assert "unknown mixer" in broken(lambda c: c["layers"][0].update(type="mamba9"))
    assert "state" in broken(lambda c: c["layers"][0]["mixer"].update(state=300))
    assert "multiple" in broken(lambda c: c["layers"][1]["mixer"].update(kv_heads=3))
    assert "rot.dims" in broken(lambda c: c["layers"][2]["mixer"]["left"]["rot"].update(dims=18))
    assert "feed-forward" in broken(lambda c: c["layers"][0]["mlp"].update(kind="gated"))
    assert "integer" in broken(lambda c: c.update(width=40.5))
    assert "positive" in broken(lambda c: c.update(vocab=0))
    assert pkg.lib().b200_decoder_check_config(b'{"architecture": "Vunolorn", ', None, 0) == pkg.B200_ERR_SHAPE
    assert pkg.lib().b200_decoder_check_config(b'{"a": "\\u00e9\\ud83d\\ude00\\n", "b": [1, -2.5e3, true, null, {}]}', None, 0) == pkg.B200_ERR_SHAPE


def test_registry_chooses_by_config(pkg, tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(CFG))
    assert pkg.model_class(str(tmp_path)) == (pkg.Decoder, "decoder")
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "GPT2", "num_layers": 2}))
    assert pkg.model_class(str(tmp_path)) == (pkg.GPT2, "gpt2")
    (tmp_path / "config.json").write_text("{}")
    with pytest.raises(pkg.B200Error, match="unknown architecture"):
        pkg.model_class(str(tmp_path))


def test_oracle_recurrences_against_closed_forms():
    rng = np.random.default_rng(0)
    T, n, s = 9, 3, 4
    x, dt = rng.standard_normal((T, n)), rng.uniform(0.01, 1, (T, n))
    A, B, C, D = -rng.uniform(0.1, 2, (n, s)), rng.standard_normal((T, s)), rng.standard_normal((T, s)), rng.standard_normal(n)
    got = L.selective_scan(x, dt, A, B, C, D)
    for t in range(T):  # the sum the recurrence unrolls to
        want = D * x[t]
        for j in range(t + 1):
            decay = np.exp(dt[j + 1:t + 1].sum(0)[:, None] * A)
            want = want + (decay * (dt[j] * x[j])[:, None] * B[j] * C[t]).sum(1)
        assert np.allclose(got[t], want)
    z, u = rng.standard_normal((T, n)), rng.standard_normal((T, n))
    S = L.min_gru(z, u)
    sz, cand = 1 / (1 + np.exp(-z)), np.where(u >= 0, u + 0.5, 1 / (1 + np.exp(-u)))
    for t in range(T):
        assert np.allclose(S[t], sum(np.prod(1 - sz[j + 1:t + 1], axis=0) * sz[j] * cand[j] for j in range(t + 1)))
    # delta rule with g = 1, beta = 1 and a unit key: what was written for a key is what a query equal to it reads
    k = L.unit_norm(rng.standard_normal((T, 1, 5)))
    v = rng.standard_normal((T, 2, 6))
    o = L.gated_delta_rule(k, k, v, np.ones((T, 2)), np.ones((T, 2)))
    assert np.allclose(o, v, atol=1e-5)


def test_oracle_attention_rotation_and_convolution():
    rng = np.random.default_rng(1)
    T = 7
    x = rng.standard_normal((T, 2, 10))
    pos = np.arange(T)
    y = L.rotate_half(x, 6, 50.0, pos)
    assert np.array_equal(y[..., 6:], x[..., 6:]) and np.allclose(y[0], x[0])
    # as complex numbers: u + iv turns by exp(i a)
    for i in range(3):
        a = pos * 50.0 ** (-2 * i / 6)
        z = (x[..., i] + 1j * x[..., i + 3]) * np.exp(1j * a)[:, None]
        assert np.allclose(y[..., i], z.real) and np.allclose(y[..., i + 3], z.imag)
    q, k, v = rng.standard_normal((T, 4, 10)), rng.standard_normal((T, 2, 10)), rng.standard_normal((T, 2, 3))
    got = L.softmax_attention(q, k, v, 0.3)
    for t in range(T):
        for h in range(4):
            e = np.exp(np.array([q[t, h] @ k[j, h // 2] for j in range(t + 1)]) * 0.3)
            assert np.allclose(got[t, h], (e[:, None] * v[:t + 1, h // 2]).sum(0) / e.sum())
    c = rng.standard_normal((T, 3))
    w = rng.standard_normal((3, 4))
    want = sum(np.vstack([np.zeros((j, 3)), c])[:T] * w[:, 3 - j] for j in range(4))
    assert np.allclose(L.short_conv_silu(c, w), want / (1 + np.exp(-want)))
    assert math.isclose(float(L.gelu_erf(np.array([1.0]))[0]), 0.8413447460685429)


def test_oracle_is_causal():
    w = L.as_float64(L.random_weights(CFG, 3))
    tok = np.random.default_rng(4).integers(0, CFG["vocab"], 20)
    full = L.forward(CFG, w, tok)
    assert np.allclose(L.forward(CFG, w, tok[:11]), full[:11])
    other = tok.copy()
    other[3] = (other[3] + 1) % CFG["vocab"]
    assert np.abs(L.forward(CFG, w, other)[19] - full[19]).max() > 1e-6  # and an early token is felt at the end
