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


PUMOTAR = {"architecture": "Pumotar", "vocab": 53, "width": 40, "embedding": {"scale": 0.25}, "norm": {"eps": 1e-6}, "loop": {"start": 0, "stop": 2, "times": 3},
           "layers": [
    {"type": "latent_attention", "mixer": {"heads": 3, "dim": 10, "rot_dim": 4, "vdim": 7, "kv_rank": 9, "scale": 0.4, "rot": {"base": 100.0, "dims": 4}},
     "mlp": {"kind": "moe", "expert": {"ff": 12, "limit": 0.9}, "router": {"experts": 5, "top": 2}, "shared": {"ff": 11, "limit": 1.2}}},
    {"type": "channel_delta", "mixer": {"conv": 3, "dim": 8, "heads": 4, "kv_heads": 2, "vdim": 6}, "mlp": {"kind": "dense", "ff": 20}},
    {"type": "channel_delta", "mixer": {"conv": 2, "dim": 5, "heads": 1, "kv_heads": 1, "vdim": 9}, "mlp": None}]}


def test_config_reader_pumotar(pkg):
    assert pkg.Decoder.check_config(PUMOTAR) == ""

    def broken(change):
        c = copy.deepcopy(PUMOTAR)
        change(c)
        return pkg.Decoder.check_config(c)

    assert broken(lambda c: c.pop("loop")) == "" and broken(lambda c: c.update(loop=None)) == ""
    assert broken(lambda c: c["layers"][0]["mlp"].pop("shared")) == "" and broken(lambda c: c["layers"][0]["mlp"].update(shared=None)) == ""
    for key, value in (("stop", 4), ("start", -1), ("start", 3), ("times", 0)):
        assert "loop" in broken(lambda c: c["loop"].update({key: value}))

    def mixer(i, **change):
        return broken(lambda c: c["layers"][i]["mixer"].update(change))

    assert "rot.dims" in mixer(0, rot={"base": 100.0, "dims": 2})
    assert "rot.dims" in mixer(0, rot_dim=3, rot={"base": 100.0, "dims": 3})
    assert "256" in mixer(0, dim=253)
    assert "kv_rank" in mixer(0, kv_rank=513)
    assert "scale" in broken(lambda c: c["layers"][0]["mixer"].pop("scale"))
    assert "multiple" in mixer(1, kv_heads=3)
    mlp = lambda c: c["layers"][0]["mlp"]
    assert "router.top" in broken(lambda c: mlp(c)["router"].update(top=6))
    assert "limit" in broken(lambda c: mlp(c)["expert"].pop("limit"))
    assert "limit" in broken(lambda c: mlp(c)["shared"].update(limit=0))
    assert "feed-forward" in broken(lambda c: mlp(c).update(kind="switch"))


def test_registry_pumotar(pkg, tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(PUMOTAR))
    assert pkg.model_class(str(tmp_path)) == (pkg.Decoder, "decoder")


def test_oracle_channel_delta_against_closed_forms():
    rng = np.random.default_rng(2)
    T, G, H, D, Dv = 8, 2, 4, 5, 3
    q, k, v = rng.standard_normal((T, G, D)), L.unit_norm(rng.standard_normal((T, G, D))), rng.standard_normal((T, H, Dv))
    g, beta = rng.uniform(0.2, 1, (T, H, D)), rng.uniform(0.1, 0.9, (T, H))
    o = L.channel_delta_rule(q, k, v, g, beta)
    for h in range(H):  # the linear map that a token amounts to, S -> (I - beta k k') diag(g) S + beta k v'
        S = np.zeros((D, Dv))
        for t in range(T):
            kk = k[t, h // 2]
            S = (np.eye(D) - beta[t, h] * np.outer(kk, kk)) @ np.diag(g[t, h]) @ S + beta[t, h] * np.outer(kk, v[t, h])
            assert np.allclose(o[t, h], q[t, h // 2] @ S)
    # one decay for all channels of a head is the other delta rule
    same = rng.uniform(0.2, 1, (T, H))
    assert np.allclose(L.channel_delta_rule(q, k, v, np.repeat(same[:, :, None], D, 2), beta), L.gated_delta_rule(q, k, v, same, beta))


def test_oracle_latent_attention_and_rotation():
    rng = np.random.default_rng(3)
    T = 9
    x = rng.standard_normal((T, 2, 6))
    y = L.rotate_pairs(x, 50.0, np.arange(T))
    for i in range(3):  # as complex numbers
        z = (x[..., 2 * i] + 1j * x[..., 2 * i + 1]) * np.exp(1j * np.arange(T) * 50.0 ** (-2 * i / 6))[:, None]
        assert np.allclose(y[..., 2 * i], z.real) and np.allclose(y[..., 2 * i + 1], z.imag)
    # scores depend on distances only
    a, b = rng.standard_normal((2, 1, 1, 6))
    dots = [float((L.rotate_pairs(a, 7.0, np.array([p + 4])) * L.rotate_pairs(b, 7.0, np.array([p]))).sum()) for p in (0, 3, 11)]
    assert np.allclose(dots, dots[0])
    # queries taken into the latent's space see the same scores and sums
    m = PUMOTAR["layers"][0]["mixer"]
    w = L.as_float64(L.random_weights(PUMOTAR, 1))
    h, p = rng.standard_normal((T, 40)), "l0.mix"
    H, D, Dr, Dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[p + ".q"].T).reshape(T, H, D + Dr)
    qr = L.rotate_pairs(q[..., D:], 100.0, np.arange(T))
    kv = h @ w[p + ".dkv"].T
    c, kr = L.rms_norm(kv[:, :R], 1e-6, w[p + ".dkv.norm"]), L.rotate_pairs(kv[:, None, R:], 100.0, np.arange(T))[:, 0]
    uk, uv = w[p + ".uk"].reshape(H, D, R), w[p + ".uv"].reshape(H, Dv, R)
    out = np.zeros((T, H, Dv))
    for t in range(T):
        for i in range(H):
            s = (c[:t + 1] @ (uk[i].T @ q[t, i, :D]) + kr[:t + 1] @ qr[t, i]) * m["scale"]
            e = np.exp(s - s.max())
            out[t, i] = uv[i] @ (e / e.sum() @ c[:t + 1])
    assert np.allclose(L.mixer_latent_attention(h, w, p, m, 1e-6), out.reshape(T, -1) @ w[p + ".o"].T)


def test_oracle_experts_and_gates():
    assert np.allclose(L.gelu_tanh(np.array([-3.0, 0.0, 1.0])), [-0.00363739, 0.0, 0.84119199])
    g, u = np.array([-9.0, 0.5, 4.0]), np.array([-4.0, 0.25, 4.0])
    want = [min(a, 1.3) / (1 + math.exp(-1.702 * min(a, 1.3))) * (max(-1.3, min(1.3, b)) + 1) for a, b in zip(g, u)]
    assert np.allclose(L.clamped_swish_gate(g, u, 1.3), want)
    m = PUMOTAR["layers"][0]["mlp"]
    w = L.as_float64(L.random_weights(PUMOTAR, 2))
    h, tok = np.random.default_rng(4).standard_normal((6, 40)), [3, 3, 50, 0, 7, 3]
    y = L.table_experts(h, w, "l0.mlp", m, tok)
    for t in range(6):
        parts = [L.clamped_mlp(h[t], w, f"l0.mlp.e{e}", 0.9) for e in w["l0.mlp.table"][tok[t]]]
        gate = 1 / (1 + math.exp(-float((h[t] @ w["l0.mlp.shared.sg"].T)[0])))
        assert np.allclose(y[t], sum(parts) / 2 + gate * L.clamped_mlp(h[t], w, "l0.mlp.shared", 1.2))
    assert all(len(set(r)) == 2 for r in w["l0.mlp.table"].tolist())


def test_oracle_loop_and_causality_pumotar():
    assert L.layer_runs(PUMOTAR) == [0, 1, 0, 1, 0, 1, 2]
    assert L.layer_runs({**PUMOTAR, "loop": None}) == [0, 1, 2]
    w = L.as_float64(L.random_weights(PUMOTAR, 3))
    tok = np.random.default_rng(4).integers(0, 53, 20)
    seen = []
    full = L.forward(PUMOTAR, w, tok, seen)
    assert len(seen) == 7 and np.allclose(L.forward(PUMOTAR, w, tok[:11]), full[:11])
    # a loop is the same layers written out
    flat = {**PUMOTAR, "loop": None, "layers": [PUMOTAR["layers"][i] for i in L.layer_runs(PUMOTAR)]}
    wf = {k: v for k, v in w.items() if not k.startswith("l")}
    for j, i in enumerate(L.layer_runs(PUMOTAR)):
        wf.update({f"l{j}" + k[2:]: v for k, v in w.items() if k.startswith(f"l{i}.")})
    assert np.allclose(L.forward(flat, wf, tok), full)
