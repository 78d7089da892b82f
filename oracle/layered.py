"""Plain numpy restatement of the layered decoders (Vunolorn, Pumotar): one function per mechanism, token by
token, no cache and no batching - a whole sequence in, the logits of every position out.

TEST INFRASTRUCTURE ONLY, like oracle.py: the tests and the smoke check compare the library with
it; the product package never imports it.  Everything is computed in the dtype of the weights that
are passed in (float64 makes it the arbiter).

Shapes: h [T, width]; weights [out, in], applied as h @ W.T; `w` is the dictionary of tensors and
`p` the prefix of the layer ('l3.mix').
"""
from __future__ import annotations

import math

import numpy as np


# ---------------------------------------------------------------- elementwise
def sigmoid(z):
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0) + np.log1p(np.exp(-np.abs(z)))


_erf = np.vectorize(math.erf, otypes=[np.float64])


def gelu_erf(z):
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)).astype(z.dtype))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def clamped_swish_gate(g, u, limit):
    """Gate bounded above, linear part on both sides; the linear part counts from one."""
    g = np.minimum(g, limit)
    u = np.clip(u, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


# ---------------------------------------------------------------- norms
def rms_norm(x, eps, weight=None):
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if weight is None else y * weight


def unit_norm(x, eps=1e-6):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + eps)


# ---------------------------------------------------------------- mechanisms
def short_conv_silu(x, taps, bias=None):
    """Causal depthwise convolution over time, then silu: the last column of `taps` [channels, n]
    meets the current token, tokens before the start count as zero."""
    T, n = x.shape[0], taps.shape[1]
    y = np.zeros_like(x)
    for t in range(T):
        for j in range(n):
            s = t - (n - 1) + j
            if s >= 0:
                y[t] += x[s] * taps[:, j]
    return silu(y if bias is None else y + bias)


def rotate_half(x, dims, base, positions):
    """x [T, heads, dim]: dimensions i and i + dims/2 (i < dims/2) turn by position * base^(-2i/dims)."""
    half = dims // 2
    f = np.asarray(base, np.float64) ** (-2.0 * np.arange(half) / dims)
    a = positions.astype(np.float64)[:, None] * f[None, :]
    c, s = np.cos(a).astype(x.dtype)[:, None, :], np.sin(a).astype(x.dtype)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], axis=-1)


def rotate_pairs(x, base, positions):
    """x [T, heads, dims]: dimensions 2i and 2i + 1 turn by position * base^(-2i/dims)."""
    dims = x.shape[-1]
    y = np.empty_like(x)
    for i in range(dims // 2):
        a = positions.astype(np.float64) * float(base) ** (-2.0 * i / dims)
        c, s = np.cos(a).astype(x.dtype)[:, None], np.sin(a).astype(x.dtype)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = u * c - v * s
        y[..., 2 * i + 1] = v * c + u * s
    return y


def softmax_attention(q, k, v, scale):
    """Causal, grouped: q [T, H, D], k [T, G, D], v [T, G, Dv]; query head h reads key/value head h // (H/G)."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]), q.dtype)
    for h in range(H):
        s = (q[:, h] @ k[:, h // per].T) * scale
        s = np.where(np.tril(np.ones((T, T), bool)), s, -np.inf)
        e = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (e / e.sum(axis=1, keepdims=True)) @ v[:, h // per]
    return out


def selective_scan(x, dt, A, B, C, D):
    """x, dt [T, inner]; A [inner, state]; B, C [T, state]; D [inner]."""
    S = np.zeros(A.shape, x.dtype)
    y = np.zeros_like(x)
    for t in range(x.shape[0]):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y


def gated_delta_rule(q, k, v, g, beta):
    """q, k [T, G, D] (unit vectors, q scaled); v [T, H, Dv]; g, beta [T, H].  The state decays, the
    value it predicts for k is corrected towards v by beta, and q reads it after the write."""
    T, H, Dv = v.shape
    per = H // q.shape[1]
    S = np.zeros((H, q.shape[2], Dv), v.dtype)
    o = np.zeros_like(v)
    for t in range(T):
        for h in range(H):
            kk, qq = k[t, h // per], q[t, h // per]
            S[h] = g[t, h] * S[h]
            u = beta[t, h] * (v[t, h] - kk @ S[h])
            S[h] = S[h] + np.outer(kk, u)
            o[t, h] = qq @ S[h]
    return o


def channel_delta_rule(q, k, v, g, beta):
    """The delta rule with a decay per key channel: q, k [T, G, D]; v [T, H, Dv]; g [T, H, D]; beta [T, H].
    Row d of a head's state is multiplied by g[d] before the token is written."""
    T, H, Dv = v.shape
    per = H // q.shape[1]
    S = np.zeros((H, q.shape[2], Dv), v.dtype)
    o = np.zeros_like(v)
    for t in range(T):
        for h in range(H):
            kk, qq = k[t, h // per], q[t, h // per]
            S[h] = g[t, h][:, None] * S[h]
            u = beta[t, h] * (v[t, h] - S[h].T @ kk)
            S[h] = S[h] + kk[:, None] * u[None, :]
            o[t, h] = S[h].T @ qq
    return o


def min_gru(z_in, x_in):
    """Gated recurrence whose gate z and candidate depend on the current token only."""
    z = sigmoid(z_in)
    cand = np.where(x_in >= 0, x_in + 0.5, sigmoid(x_in))
    S = np.zeros(x_in.shape[1], x_in.dtype)
    out = np.zeros_like(x_in)
    for t in range(x_in.shape[0]):
        S = (1 - z[t]) * S + z[t] * cand[t]
        out[t] = S
    return out


# ---------------------------------------------------------------- mixers
def mixer_mamba1(h, w, p, m, eps):
    inner, rank, state = m["inner"], m["dt_rank"], m["state"]
    xz = h @ w[p + ".in"].T
    x, z = xz[:, :inner], xz[:, inner:]
    x = short_conv_silu(x, w[p + ".conv"], w[p + ".conv.b"])
    dbc = x @ w[p + ".x"].T
    dt = softplus(dbc[:, :rank] @ w[p + ".dt"].T + w[p + ".dt.b"])
    y = selective_scan(x, dt, -np.exp(w[p + ".A_log"]), dbc[:, rank:rank + state], dbc[:, rank + state:], w[p + ".D"])
    return (y * silu(z)) @ w[p + ".o"].T


def mixer_delta(h, w, p, m, eps):
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (short_conv_silu(h @ w[f"{p}.{n}"].T, w[f"{p}.{n}.conv"]) for n in "qkv")
    q = unit_norm(q.reshape(T, G, D)) * D ** -0.5
    k = unit_norm(k.reshape(T, G, D))
    beta = sigmoid(h @ w[p + ".b"].T)
    g = np.exp(-np.exp(w[p + ".A_log"]) * softplus(h @ w[p + ".a"].T + w[p + ".dt_bias"]))
    o = gated_delta_rule(q, k, v.reshape(T, H, Dv), g, beta)
    o = rms_norm(o, eps, w[p + ".norm"]) * silu(h @ w[p + ".g"].T).reshape(T, H, Dv)
    return o.reshape(T, H * Dv) @ w[p + ".o"].T


def mixer_attention(h, w, p, m, eps):
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = np.arange(T)
    q = rms_norm((h @ w[p + ".q"].T).reshape(T, H, D), eps, w[p + ".q.norm"])
    k = rms_norm((h @ w[p + ".k"].T).reshape(T, G, D), eps, w[p + ".k.norm"])
    v = rms_norm((h @ w[p + ".v"].T).reshape(T, G, Dv), eps)
    q = rotate_half(q, m["rot"]["dims"], m["rot"]["base"], pos)
    k = rotate_half(k, m["rot"]["dims"], m["rot"]["base"], pos)
    return softmax_attention(q, k, v, m["scale"]).reshape(T, H * Dv) @ w[p + ".o"].T


def mixer_min_gru(h, w, p, m, eps):
    S = min_gru(h @ w[p + ".z"].T + w[p + ".z.b"], h @ w[p + ".x"].T + w[p + ".x.b"])
    return (S * silu(h @ w[p + ".g"].T)) @ w[p + ".o"].T


def mixer_parallel(h, w, p, m, eps):
    return (m["left_scale"] * mixer_attention(h, w, p + ".left", m["left"], eps)
            + m["right_scale"] * mixer_min_gru(h, w, p + ".right", m["right"], eps))


def mixer_latent_attention(h, w, p, m, eps):
    """Keys and values of all heads come from one low-rank latent per token; the rotated part of the key is
    shared by the heads."""
    T, H, D, Dr, Dv, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos, base = np.arange(T), m["rot"]["base"]
    q = (h @ w[p + ".q"].T).reshape(T, H, D + Dr)
    q = np.concatenate([q[..., :D], rotate_pairs(q[..., D:], base, pos)], axis=-1)
    kv = h @ w[p + ".dkv"].T
    c = rms_norm(kv[:, :R], eps, w[p + ".dkv.norm"])
    k_rot = np.broadcast_to(rotate_pairs(kv[:, None, R:], base, pos), (T, H, Dr))
    k = np.concatenate([(c @ w[p + ".uk"].T).reshape(T, H, D), k_rot], axis=-1)
    v = (c @ w[p + ".uv"].T).reshape(T, H, Dv)
    return softmax_attention(q, k, v, m["scale"]).reshape(T, H * Dv) @ w[p + ".o"].T


def mixer_channel_delta(h, w, p, m, eps):
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (short_conv_silu(h @ w[f"{p}.{n}"].T, w[f"{p}.{n}.conv"]) for n in "qkv")
    q = unit_norm(q.reshape(T, G, D)) * D ** -0.5
    k = unit_norm(k.reshape(T, G, D))
    beta = sigmoid(h @ w[p + ".b"].T)
    a = (h @ w[p + ".a1"].T) @ w[p + ".a2"].T
    g = np.exp(-np.exp(w[p + ".A_log"])[None, :, None] * softplus(a + w[p + ".dt_bias"]).reshape(T, H, D))
    o = channel_delta_rule(q, k, v.reshape(T, H, Dv), g, beta)
    gate = sigmoid((h @ w[p + ".g1"].T) @ w[p + ".g2"].T).reshape(T, H, Dv)
    return (rms_norm(o, eps, w[p + ".norm"]) * gate).reshape(T, H * Dv) @ w[p + ".o"].T


MIXERS = {"mamba1": mixer_mamba1, "delta": mixer_delta, "parallel": mixer_parallel,
          "latent_attention": mixer_latent_attention, "channel_delta": mixer_channel_delta}


# ---------------------------------------------------------------- feed-forward
def dense_mlp(h, w, p):
    return gelu_erf(h @ w[p + ".up"].T) @ w[p + ".down"].T


def gated_mlp(h, w, p):
    return (gelu_tanh(h @ w[p + ".gate"].T) * (h @ w[p + ".up"].T)) @ w[p + ".down"].T


def clamped_mlp(h, w, p, limit):
    return clamped_swish_gate(h @ w[p + ".gate"].T, h @ w[p + ".up"].T, limit) @ w[p + ".down"].T


def table_experts(h, w, p, m, tokens):
    """Every token id has its experts in a table; they count alike.  The shared expert is weighed by a gate."""
    top = m["router"]["top"]
    table = np.asarray(w[p + ".table"]).astype(np.int64)
    y = np.zeros_like(h)
    for t, tok in enumerate(tokens):
        for e in table[tok]:
            y[t] += clamped_mlp(h[t:t + 1], w, f"{p}.e{e}", m["expert"]["limit"])[0] / top
    if m.get("shared"):
        gate = sigmoid(h @ w[p + ".shared.sg"].T)
        y = y + gate * clamped_mlp(h, w, p + ".shared", m["shared"]["limit"])
    return y


# ---------------------------------------------------------------- models
def forward_vunolorn(cfg, w, tokens, layer_outputs=None):
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}"
        y = MIXERS[layer["type"]](rms_norm(x, eps, w[p + ".norm1"]), w, p + ".mix", layer["mixer"], eps)
        x = x + rms_norm(y, eps, w[p + ".norm1b"])
        if layer["mlp"] is not None:
            y = dense_mlp(rms_norm(x, eps, w[p + ".norm2"]), w, p + ".mlp")
            x = x + rms_norm(y, eps, w[p + ".norm2b"])
        if layer_outputs is not None:
            layer_outputs.append(x.copy())
    return rms_norm(x, eps, w["final.norm"]) @ w["head"].T


def layer_runs(cfg):
    """The order in which the layers run: those of the loop several times over."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    body = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + body * loop["times"] + list(range(loop["stop"], n))


def forward_pumotar(cfg, w, tokens, layer_outputs=None):
    eps, tokens = cfg["norm"]["eps"], np.asarray(tokens)
    x = w["embed"][tokens] * cfg["embedding"]["scale"]
    for i in layer_runs(cfg):
        p, layer = f"l{i}", cfg["layers"][i]
        x = x + MIXERS[layer["type"]](rms_norm(x, eps, 1 + w[p + ".norm1"]), w, p + ".mix", layer["mixer"], eps)
        mlp = layer["mlp"]
        if mlp is not None:
            h = rms_norm(x, eps, 1 + w[p + ".norm2"])
            x = x + (gated_mlp(h, w, p + ".mlp") if mlp["kind"] == "dense" else table_experts(h, w, p + ".mlp", mlp, tokens))
        if layer_outputs is not None:
            layer_outputs.append(x.copy())
    return rms_norm(x, eps, 1 + w["final.norm"]) @ w["embed"].T


DESIGNS = {"Vunolorn": forward_vunolorn, "Pumotar": forward_pumotar}


def forward(cfg, w, tokens, layer_outputs=None):
    """Logits [T, vocab] of a whole sequence; the residual stream after every layer run is appended to
    layer_outputs if a list is given."""
    return DESIGNS[cfg["architecture"]](cfg, w, tokens, layer_outputs)


# ---------------------------------------------------------------- random models
def tensor_shapes(cfg):
    """name -> shape of every tensor of the model."""
    C, V = cfg["width"], cfg["vocab"]
    post_norm = own_head = cfg["architecture"] == "Vunolorn"
    s = {"embed": (V, C)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}", layer["mixer"]
        s[p + ".norm1"] = (C,)
        if post_norm:
            s[p + ".norm1b"] = (C,)
        if layer["type"] == "mamba1":
            n, r, st = m["inner"], m["dt_rank"], m["state"]
            s.update({p + ".mix.in": (2 * n, C), p + ".mix.conv": (n, m["conv"]), p + ".mix.conv.b": (n,),
                      p + ".mix.x": (r + 2 * st, n), p + ".mix.dt": (n, r), p + ".mix.dt.b": (n,),
                      p + ".mix.A_log": (n, st), p + ".mix.D": (n,), p + ".mix.o": (C, n)})
        elif layer["type"] == "delta":
            H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for n, rows in (("q", G * D), ("k", G * D), ("v", H * Dv)):
                s[f"{p}.mix.{n}"] = (rows, C)
                s[f"{p}.mix.{n}.conv"] = (rows, m["conv"])
            s.update({p + ".mix.b": (H, C), p + ".mix.A_log": (H,), p + ".mix.norm": (Dv,), p + ".mix.a": (H, C),
                      p + ".mix.dt_bias": (H,), p + ".mix.g": (H * Dv, C), p + ".mix.o": (C, H * Dv)})
        elif layer["type"] == "channel_delta":
            H, G, D, Dv, x = m["heads"], m["kv_heads"], m["dim"], m["vdim"], p + ".mix"
            ra, rg = low_ranks(layer)
            for n, rows in (("q", G * D), ("k", G * D), ("v", H * Dv)):
                s[f"{x}.{n}"] = (rows, C)
                s[f"{x}.{n}.conv"] = (rows, m["conv"])
            s.update({x + ".b": (H, C), x + ".A_log": (H,), x + ".norm": (Dv,), x + ".a1": (ra, C), x + ".a2": (H * D, ra),
                      x + ".dt_bias": (H * D,), x + ".g1": (rg, C), x + ".g2": (H * Dv, rg), x + ".o": (C, H * Dv)})
        elif layer["type"] == "latent_attention":
            H, D, Dr, Dv, R, x = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], p + ".mix"
            s.update({x + ".q": (H * (D + Dr), C), x + ".dkv": (R + Dr, C), x + ".dkv.norm": (R,), x + ".uk": (H * D, R),
                      x + ".uv": (H * Dv, R), x + ".o": (C, H * Dv)})
        else:
            l, r = m["left"], m["right"]
            a, b = p + ".mix.left", p + ".mix.right"
            s.update({a + ".q": (l["heads"] * l["dim"], C), a + ".k": (l["kv_heads"] * l["dim"], C),
                      a + ".v": (l["kv_heads"] * l["vdim"], C), a + ".q.norm": (l["dim"],), a + ".k.norm": (l["dim"],),
                      a + ".o": (C, l["heads"] * l["vdim"])})
            W = r["width"]
            s.update({b + ".z": (W, C), b + ".z.b": (W,), b + ".x": (W, C), b + ".x.b": (W,), b + ".g": (W, C), b + ".o": (C, W)})
        mlp = layer["mlp"]
        if mlp is None:
            continue
        s[p + ".norm2"] = (C,)
        gated = lambda q, F: {q + ".gate": (F, C), q + ".up": (F, C), q + ".down": (C, F)}
        if post_norm:
            F = mlp["ff"]
            s.update({p + ".norm2b": (C,), p + ".mlp.up": (F, C), p + ".mlp.down": (C, F)})
        elif mlp["kind"] == "dense":
            s.update(gated(p + ".mlp", mlp["ff"]))
        else:
            for e in range(mlp["router"]["experts"]):
                s.update(gated(f"{p}.mlp.e{e}", mlp["expert"]["ff"]))
            s[p + ".mlp.table"] = (V, mlp["router"]["top"])
            if mlp.get("shared"):
                s.update(gated(p + ".mlp.shared", mlp["shared"]["ff"]))
                s[p + ".mlp.shared.sg"] = (1, C)
    s["final.norm"] = (C,)
    if own_head:
        s["head"] = (V, C)
    return s


def low_ranks(layer):
    """Ranks of the low-rank decay and output gate, which only the tensors' shapes give: picked here from the sizes."""
    m = layer["mixer"]
    return m.get("ranks", (m["dim"] // 3 + 1, m["vdim"] // 2 + 3))


def to_bf16(a):
    """Nearest bf16 value (ties to even) of every element, as float32."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return (((u.astype(np.uint64) + 0x7FFF + ((u >> 16) & 1)) >> 16 << 16).astype(np.uint32)).view(np.float32)


def random_weights(cfg, seed):
    """Weights (float32, every value exact in bf16) whose activations stay of order one and whose
    decays cover slow and fast channels."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf == "table":  # the entries of a row differ
            i = int(name[1:].split(".")[0])
            experts = cfg["layers"][i]["mlp"]["router"]["experts"]
            w[name] = np.stack([rng.permutation(experts)[:shape[1]] for _ in range(shape[0])]).astype(np.int32)
            continue
        if name == "final.norm" or leaf in ("norm1", "norm2"):
            a = (0.0 if cfg["architecture"] == "Pumotar" else 1.0) + 0.3 * rng.standard_normal(shape)
        elif "norm" in leaf:
            a = 1.0 + 0.3 * rng.standard_normal(shape)
        elif leaf == "A_log":
            a = rng.uniform(-2.0, 1.5, shape)
        elif leaf == "D":
            a = 1.0 + 0.3 * rng.standard_normal(shape)
        elif leaf == "dt_bias" or name.endswith(".dt.b"):
            a = rng.uniform(-5.0, -0.5, shape)
        elif leaf == "b" and len(shape) == 1:
            a = 0.5 * rng.standard_normal(shape)
        elif leaf == "conv":
            a = rng.standard_normal(shape) / math.sqrt(shape[1])
        elif name == "embed":
            a = rng.standard_normal(shape) / cfg["embedding"]["scale"]
            if cfg["architecture"] == "Pumotar":  # (the layers' part of the residual stream is to outweigh the token's own embedding)
                a *= 0.2
        else:
            a = rng.standard_normal(shape) / math.sqrt(shape[1])
        w[name] = to_bf16(a)
    return w


def as_float64(w):
    return {k: v if v.dtype == np.int32 else v.astype(np.float64) for k, v in w.items()}


def as_bits(w):
    """The weights as the library takes them: bf16 bits, int32 tables."""
    return {k: v if v.dtype == np.int32 else (v.view(np.uint32) >> 16).astype(np.uint16) for k, v in w.items()}


def save_safetensors(path, w):
    """Writes the weights as bf16 (their values must be exact in bf16), tables as int32."""
    import json
    import struct
    head, off, blobs = {}, 0, []
    for name, a in w.items():
        table = a.dtype == np.int32
        b = a.astype("<i4").tobytes() if table else (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype(np.uint16).tobytes()
        head[name] = {"dtype": "I32" if table else "BF16", "shape": list(a.shape), "data_offsets": [off, off + len(b)]}
        off += len(b)
        blobs.append(b)
    h = json.dumps(head).encode()
    h += b" " * (-len(h) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(h)))
        f.write(h)
        for b in blobs:
            f.write(b)
