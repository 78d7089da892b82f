"""Pumotar (latent attention, delta rule with a decay per key channel, gated feed-forwards, table-routed experts, looped
layers) on the GPU against the plain oracle (oracle/layered.py, float64).  Errors and tolerances as in
test_layered_gpu.py.  A prompt's portion is expanded (keys and values of all heads are formed) from some twenty tokens on; shorter
ones, and decoding, attend to the latents themselves: the portions below reach both."""
import json
import os
import subprocess

import numpy as np
import pytest

from oracle import layered as L
from test_layered_gpu import ROOT, TOL, check, delta as head_delta, run, tokens

pytestmark = pytest.mark.gpu
DTYPES = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts=5, top=2, ff=36, limit=0.8, shared=44, shared_limit=1.1):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared, "limit": shared_limit}
    return m


def latent(heads=4, dim=32, rot_dim=16, vdim=24, kv_rank=40, base=1000.0, scale=0.3, mlp=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                                                  "rot": {"base": base, "dims": rot_dim}}, "mlp": mlp}


def channel(heads=4, kv_heads=2, dim=32, vdim=24, conv=4, ranks=None, mlp=None):
    m = {"conv": conv, "dim": dim, "heads": heads, "kv_heads": kv_heads, "vdim": vdim}
    if ranks:
        m["ranks"] = ranks
    return {"type": "channel_delta", "mixer": m, "mlp": mlp}


def config(layers, width=96, vocab=211, eps=1e-5, scale=3.0, loop=None):
    c = {"architecture": "Pumotar", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps}, "layers": layers}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def model(pkg, ctx, cfg, dtype, seed=1, tweak=None, **kw):
    w = L.random_weights(cfg, seed)
    if tweak:
        tweak(w)
    kw.setdefault("max_slots", 4)
    kw.setdefault("max_seq", 640)
    m = pkg.Decoder(ctx, cfg, dtype=dtype, **kw)
    m.load_tensors(L.as_bits(w))
    return m, L.as_float64(w)


LAYERS = {
    "latent": [latent()],
    "latent_one": [latent(heads=1, dim=1, rot_dim=2, vdim=1, kv_rank=1)],
    "latent_odd": [latent(heads=3, dim=23, rot_dim=6, vdim=21, kv_rank=37)],
    "latent_17": [latent(heads=17, dim=16, rot_dim=8, vdim=12, kv_rank=130)],
    "latent_40": [latent(heads=40, dim=20, rot_dim=4, vdim=8, kv_rank=64)],
    "latent_256": [latent(heads=6, dim=64, rot_dim=32, vdim=64, kv_rank=256, scale=0.15)],
    "latent_512": [latent(heads=2, dim=128, rot_dim=64, vdim=128, kv_rank=512, scale=0.1)],
    "latent_640": [latent(heads=20, dim=24, rot_dim=128, vdim=16, kv_rank=512, scale=0.1)],
    "latent_v128": [latent(heads=3, dim=40, rot_dim=24, vdim=128, kv_rank=72)],
    "latent_v200": [latent(heads=2, dim=100, rot_dim=100, vdim=200, kv_rank=90, scale=0.15)],
    "channel": [channel()],
    "channel_one": [channel(heads=1, kv_heads=1, dim=1, vdim=1, conv=1, ranks=(1, 1))],
    "channel_two": [channel(heads=1, kv_heads=1, dim=2, vdim=3, conv=1, ranks=(1, 1))],
    "channel_odd": [channel(heads=6, kv_heads=2, dim=23, vdim=21, conv=3, ranks=(5, 13))],
    "channel_wide": [channel(heads=2, kv_heads=1, dim=128, vdim=160, conv=2, ranks=(70, 9))],
    "channel_80": [channel(heads=4, kv_heads=4, dim=80, vdim=40, conv=6, ranks=(8, 130))],
    "channel_200": [channel(heads=2, kv_heads=2, dim=200, vdim=36, ranks=(33, 64))],
    "channel_64": [channel(heads=3, kv_heads=1, dim=64, vdim=64, conv=5)],
    "head_decay": [head_delta()],
    "dense": [latent(mlp=dense(50))],
    "dense_one": [channel(mlp=dense(1))],
    "dense_128": [channel(mlp=dense(128))],
    "moe": [latent(mlp=moe())],
    "moe_top1": [channel(mlp=moe(experts=7, top=1, ff=64, shared=33, shared_limit=0.4))],
    "moe_all": [channel(mlp=moe(experts=3, top=3, ff=20, limit=2.5, shared=100))],
    "moe_alone": [latent(mlp=moe(experts=20, top=4, ff=9, shared=None))],
    "moe_one": [channel(mlp=moe(experts=1, top=1, ff=1, shared=1))],
    "moe_many": [channel(mlp=moe(experts=70, top=6, ff=40))],
}


@DTYPES
@pytest.mark.parametrize("name", sorted(LAYERS))
def test_each_mechanism(pkg, ctx, name, dtype):
    """One layer at several sizes: whole, token by token from the start, prompt then decoding, portions."""
    if name in ("channel_one", "channel_two") and dtype == "bfloat16":
        pytest.skip("an output of one or two channels may be nearly nothing before its norm: 16-bit rounding of the inputs decides it")
    cfg = config(LAYERS[name])
    m, w = model(pkg, ctx, cfg, dtype)
    tok = tokens(cfg, 75)
    want = L.forward(cfg, w, tok)
    for portions in ([75], [1], [41, 1], [2, 3, 1, 17, 2], [33, 31, 2]):
        check(run(m, tok, portions), want, TOL[dtype], f"{name} {dtype} {portions}")
    m.close()


STACK = [channel(mlp=dense(60)), latent(mlp=moe()), channel(heads=2, kv_heads=2, dim=64, vdim=32, mlp=moe(experts=6, top=1, ff=70, shared=20)),
         latent(heads=6, dim=48, rot_dim=32, vdim=40, kv_rank=70), channel(heads=3, kv_heads=1, conv=2, mlp=moe(experts=4, top=3, shared=None))]


@DTYPES
@pytest.mark.parametrize("width,vocab,eps,scale,loop", [(96, 211, 1e-5, 3.0, None), (50, 77, 1e-3, 1.0, (1, 4, 2)), (264, 1030, 1e-6, 16.0, (0, 2, 3)),
                                                        (72, 90, 1e-5, 0.5, (3, 5, 2)), (40, 60, 1e-5, 2.0, (0, 5, 1)), (40, 60, 1e-5, 2.0, (2, 2, 4))])
def test_stack_of_layers(pkg, ctx, dtype, width, vocab, eps, scale, loop):
    """Layers of every kind, some of them run several times with a state of their own each time."""
    cfg = config(STACK, width, vocab, eps, scale, loop)
    m, w = model(pkg, ctx, cfg, dtype, seed=2)
    tok = tokens(cfg, 330, seed=width)
    want = L.forward(cfg, w, tok)
    for portions in ([330], [129, 128, 1, 1, 2, 7, 2], [64], [300, 1]):
        check(run(m, tok, portions), want, TOL[dtype] * (2 if dtype == "bfloat16" else 1), f"{dtype} {portions}")
    m.close()


def test_mixers_are_shared_between_designs(pkg, ctx):
    """A mixer of one design in a model of the other."""
    cfg = dict(config([latent(), channel()]), architecture="Vunolorn")
    m, w = model(pkg, ctx, cfg, "float32", seed=3)
    tok = tokens(cfg, 60)
    check(run(m, tok, [50, 1]), L.forward(cfg, w, tok), TOL["float32"])
    m.close()


@DTYPES
def test_first_tokens(pkg, ctx, dtype):
    cfg = config(STACK, loop=(1, 3, 2))
    m, w = model(pkg, ctx, cfg, dtype, seed=3)
    tok = tokens(cfg, 9)
    want = L.forward(cfg, w, tok)
    for n in range(1, 10):
        check(run(m, tok[:n], [n]), want[:n], TOL[dtype] * 2, f"prompt of {n}")
        check(run(m, tok[:n], [max(1, n - 3), 1]), want[:n], TOL[dtype] * 2, f"prompt of {n}, decoded")
    m.close()


@DTYPES
@pytest.mark.parametrize("rank,heads,vdim", [(64, 2, 64), (128, 2, 128), (64, 20, 16), (192, 1, 40)])
def test_far_keys_and_tile_borders(pkg, ctx, dtype, rank, heads, vdim):
    """Each of the queries below finds one key, far away or just across a border of the kernels' tiles: unrotated keys are the latents
    themselves, the query projection is the latents' behind a rotation of the width by one (and nothing in the rotated part), and
    the token at place a is embedded as the rotated embedding of the token at place b, so that b's score for a stands out."""
    T, width = 600, 192
    cfg = config([latent(heads=heads, dim=rank, rot_dim=2, vdim=vdim, kv_rank=rank, scale=0.5)], width=width, vocab=700)
    tok = (np.arange(T) * 11 + 3) % 700  # all different
    pairs = ((0, 599), (511, 598), (5, 513), (300, 512), (256, 511), (383, 384), (255, 257), (128, 256), (127, 129), (1, 128), (64, 127), (63, 64), (31, 32))

    def paired(w):
        w["l0.norm1"].fill(0.0)
        w["l0.mix.dkv.norm"].fill(1.0)
        q = np.roll(w["l0.mix.dkv"][:rank], -1, axis=1)
        w["l0.mix.q"] = np.concatenate([q, np.zeros((2, width), np.float32)] * heads)
        w["l0.mix.uk"] = np.concatenate([np.eye(rank, dtype=np.float32)] * heads)
        for a, b in pairs:
            w["embed"][tok[a]] = np.roll(w["embed"][tok[b]], 1)
    m, w = model(pkg, ctx, cfg, dtype, seed=4, tweak=paired)
    want = L.forward(cfg, w, tok)
    for a, b in pairs[:3]:  # without its far key a query's logits are others altogether
        lost = tok.copy()
        lost[a] = (T * 11 + 3) % 700
        assert np.sqrt(((L.forward(cfg, w, lost)[b] - want[b]) ** 2).mean() / (want ** 2).mean()) > 0.1
    for portions in ([600], [1, 127, 129, 2, 300, 1], [126, 1, 1, 1, 1, 124, 1, 1, 1, 2, 250, 1], [511, 1], [7]):
        check(run(m, tok, portions), want, TOL[dtype], f"{rank} {portions}")
    m.close()


@DTYPES
def test_rotation_decides(pkg, ctx, dtype):
    """Scores from the rotated part alone, sharp: every query falls on the one key whose distance turns its pairs into line."""
    cfg = config([latent(heads=2, dim=8, rot_dim=32, vdim=40, kv_rank=48, base=50.0, scale=2.0)], width=64, vocab=300)

    def rotated_only(w):
        w["l0.mix.uk"].fill(0.0)
    m, w = model(pkg, ctx, cfg, dtype, seed=5, tweak=rotated_only)
    tok = tokens(cfg, 200)
    want = L.forward(cfg, w, tok)
    for portions in ([200], [1], [100, 3]):
        check(run(m, tok, portions), want, TOL[dtype] * 2, str(portions))
    m.close()


@DTYPES
def test_long_memory_and_strong_decays(pkg, ctx, dtype):
    """Channels that forget slowly - the first tokens are still felt hundreds of tokens later - beside channels that forget at once."""
    cfg = config([channel(heads=2, kv_heads=1, dim=64, vdim=32), channel(heads=4, kv_heads=4, dim=48, vdim=64, conv=3)])

    def decays(w):
        for l in (0, 1):
            w[f"l{l}.mix.A_log"][:] = -4.0
            w[f"l{l}.mix.dt_bias"][:] = -4.0
            w[f"l{l}.mix.b"][:] *= 0.5
        w["l0.mix.A_log"][1] = 4.0
        w["l0.mix.dt_bias"][100:] = 6.0   # exp(-54 * 6) is nothing
        w["l1.mix.dt_bias"][::3] = 3.0
    m, w = model(pkg, ctx, cfg, dtype, seed=6, tweak=decays)
    tok = tokens(cfg, 420)
    want = L.forward(cfg, w, tok)
    cut = np.sqrt(((L.forward(cfg, w, tok[200:])[-1] - want[-1]) ** 2).mean()) / np.sqrt((want ** 2).mean())
    assert cut > 3 * TOL["bfloat16"], cut
    for portions in ([420], [5, 1], [150, 2, 33, 1, 64, 3], [128, 128, 128, 1]):
        check(run(m, tok, portions), want, TOL[dtype], str(portions))
    m.close()


@DTYPES
def test_batches_of_unequal_requests(pkg, ctx, dtype):
    """Ragged steps - prompts, portions and single tokens of several requests together - against each request alone."""
    cfg = config(STACK, loop=(1, 3, 2))
    m, w = model(pkg, ctx, cfg, dtype, seed=7, max_slots=20, max_seq=320, max_rows=400)
    lens = [1, 2, 300, 17, 128, 129, 45, 64, 3, 255, 31]
    toks = [tokens(cfg, n, seed=100 + i) for i, n in enumerate(lens)]
    want = [L.forward(cfg, w, t) for t in toks]
    rng = np.random.default_rng(8)
    slots, at = [m.open() for _ in lens], [0] * len(lens)
    got = [[] for _ in lens]
    step = 0
    while any(a < n for a, n in zip(at, lens)):
        live = [i for i in range(len(lens)) if at[i] < lens[i] and (step % 3 == 2 or rng.random() < 0.7)]
        if not live:
            continue
        # every third step is one token for each live request (the decode path), the others portions
        counts = {i: 1 if step % 3 == 2 else int(min(lens[i] - at[i], rng.integers(1, 60))) for i in live}
        total = sum(counts.values())
        lg = m.step([(slots[i], toks[i][at[i]:at[i] + counts[i]]) for i in live], want=range(total))
        r = 0
        for i in live:
            got[i].append(lg[r:r + counts[i]])
            at[i] += counts[i]
            r += counts[i]
        step += 1
    for i in range(len(lens)):
        check(np.concatenate(got[i]), want[i], TOL[dtype] * 2, f"request {i} of {lens[i]} tokens")
    m.close()


@pytest.mark.parametrize("B", [1, 2, 3, 4, 5, 8, 9, 16])
def test_decode_batch_sizes(pkg, ctx, B):
    """The decode path at every padding of the batch, sequences at different positions, graph replays included; the
    last steps bring the same token everywhere, so that all rows share their experts."""
    cfg = config(STACK, loop=(0, 2, 2))
    m, w = model(pkg, ctx, cfg, "bfloat16", seed=9, max_slots=16, max_seq=160)
    toks = [tokens(cfg, 30 + 7 * i, seed=i) for i in range(B)]
    for t in toks:
        t[-2:] = 5
    want = [L.forward(cfg, w, t) for t in toks]
    slots = [m.open() for _ in range(B)]
    for i in range(B):
        m.step([(slots[i], toks[i][:-6])])
    for k in range(6):
        lg = m.step([(slots[i], toks[i][len(toks[i]) - 6 + k:][:1]) for i in range(B)])
        for i in range(B):
            check(lg[i:i + 1], want[i][len(toks[i]) - 6 + k:][:1], TOL["bfloat16"] * 2, f"sequence {i}, step {k}")
    m.close()


@pytest.mark.parametrize("mlp", [moe(experts=64, top=16, ff=33, shared=200), moe(experts=2, top=1, ff=300, shared=20), moe(experts=9, top=2, ff=520, shared=None)])
def test_decode_with_many_experts(pkg, ctx, mlp):
    """Up to 256 (row, expert) pairs in a decode step; experts wider and narrower than the shared one."""
    cfg = config([channel(mlp=mlp), latent(mlp=mlp)], width=136)
    m, w = model(pkg, ctx, cfg, "bfloat16", seed=10, max_slots=16, max_seq=64)
    toks = [tokens(cfg, 8, seed=i) for i in range(16)]
    slots = [m.open() for _ in toks]
    got = np.stack([m.step([(s, t[k:k + 1]) for s, t in zip(slots, toks)]) for k in range(8)], axis=1)
    for g, t in zip(got, toks):
        check(g, L.forward(cfg, w, t), TOL["bfloat16"] * 1.5)
    m.close()


@DTYPES
def test_slots_are_reused(pkg, ctx, dtype):
    """A slot that held a longer sequence serves the next one as a fresh one would: bit for bit."""
    cfg = config(STACK, loop=(1, 4, 2))
    fresh, _ = model(pkg, ctx, cfg, dtype, seed=10, max_slots=1)
    t1, t2 = tokens(cfg, 400, seed=1), tokens(cfg, 90, seed=2)
    portions = [50, 1, 1, 5, 1]
    want = run(fresh, t2, portions)
    fresh.close()
    m, _ = model(pkg, ctx, cfg, dtype, seed=10, max_slots=1)
    for _ in range(2):
        run(m, t1, [300, 1, 40])
        assert np.array_equal(run(m, t2, portions), want)
    m.close()


@pytest.mark.parametrize("layer,width", [
    (latent(heads=12, dim=64, rot_dim=32, vdim=64, kv_rank=256, scale=0.1, mlp=moe(experts=4, top=1, ff=300, shared=260)), 128),
    (latent(heads=14, dim=96, rot_dim=32, vdim=128, kv_rank=192, scale=0.1, mlp=dense(2600)), 128),
    (channel(heads=12, kv_heads=6, dim=64, vdim=128, mlp=moe(experts=2, top=2, ff=1024, shared=None)), 256),
    (channel(heads=24, kv_heads=24, dim=64, vdim=128, mlp=moe(experts=3, top=1, ff=1500, shared=700)), 512),
    (channel(heads=16, kv_heads=4, dim=128, vdim=128, mlp=moe(experts=40, top=2, ff=96, shared=100)), 128)])
def test_large_steps_equal_small_ones(pkg, ctx, layer, width):
    """Steps of thousands of rows - persistent kernels with several items per CTA, paired-CTA products with gated and with grouped
    tiles, runs of 256 rows, the delta rule's wider column groups - against each sequence alone."""
    cfg = config([layer], width=width, vocab=300)
    n = 12
    m, _ = model(pkg, ctx, cfg, "bfloat16", seed=16, max_slots=n, max_seq=384, max_rows=4096)
    toks = [tokens(cfg, 200 + 13 * i, seed=i) for i in range(n)]
    slots = [m.open() for _ in range(n)]
    first = [len(t) // 3 + i for i, t in enumerate(toks)]
    m.step([(s, t[:k]) for s, t, k in zip(slots, toks, first)])
    rest = [t[k:] for t, k in zip(toks, first)]
    together = m.step(list(zip(slots, rest)), want=range(sum(map(len, rest))))
    for s in slots:
        m.close_slot(s)
    slots = [m.open() for _ in range(n)]  # all of them once more, in one step from their start
    whole = m.step(list(zip(slots, toks)), want=range(sum(map(len, toks))))
    for s in slots:
        m.close_slot(s)
    r = w = 0
    for i, t in enumerate(toks):
        alone = run(m, t, [64])
        check(together[r:r + len(rest[i])], alone[first[i]:], TOL["bfloat16"], f"sequence {i}, continued")
        check(whole[w:w + len(t)], alone, TOL["bfloat16"], f"sequence {i}, whole")
        r += len(rest[i])
        w += len(t)
    m.close()


def test_long_decoding(pkg, ctx):
    cfg = config([channel(mlp=moe()), latent(mlp=dense(40))], loop=(0, 2, 2))
    m, w = model(pkg, ctx, cfg, "bfloat16", seed=11, max_seq=600)
    tok = tokens(cfg, 560)
    check(run(m, tok, [3, 1]), L.forward(cfg, w, tok), TOL["bfloat16"] * 1.5, "557 tokens decoded one by one")
    m.close()


@DTYPES
def test_steps_beyond_the_activation_buffers(pkg, ctx, dtype):
    """max_rows smaller than the step: it is cut, and the wanted rows come back in the order asked for."""
    cfg = config(STACK, loop=(1, 2, 3))
    m, w = model(pkg, ctx, cfg, dtype, seed=12, max_slots=3, max_seq=200, max_rows=48)
    toks = [tokens(cfg, n, seed=n) for n in (150, 20, 70)]
    want = np.concatenate([L.forward(cfg, w, t) for t in toks])
    slots = [m.open() for _ in toks]
    rows = np.random.default_rng(0).permutation(240)[:40]
    check(m.step(list(zip(slots, toks)), want=rows), want[rows], TOL[dtype] * 2)
    m.close()


@DTYPES
def test_greedy_generation(pkg, ctx, dtype):
    """More requests than slots, unequal prompts, prompts longer than max_rows, through the scheduler: every generated
    token is the oracle's arg-max after the tokens before it (up to a near-tie)."""
    cfg = config(STACK, loop=(1, 3, 2))
    m, w = model(pkg, ctx, cfg, dtype, seed=13, max_slots=3, max_seq=128, max_rows=40)
    prompts = [tokens(cfg, n, seed=n) for n in (1, 33, 90, 2, 57, 40, 8)]
    n_new = 14
    out = m.generate(prompts, n_new)
    assert out.shape == (len(prompts), n_new)
    for p, o in zip(prompts, out):
        lg = L.forward(cfg, w, np.concatenate([p, o[:-1]]))[len(p) - 1:]
        gap = lg.max(1) - lg[np.arange(n_new), o]
        assert gap.max() <= 4 * TOL[dtype] * np.sqrt((lg ** 2).mean()), gap
    assert all(m.length(s) == -1 for s in range(3))  # every slot was given back
    alone = np.concatenate([m.generate([p], n_new) for p in prompts])
    if dtype == "float32":
        assert np.array_equal(alone, out)
    else:  # a near-tie that falls the other way changes all that follows it
        assert (alone[:, :3] == out[:, :3]).mean() > 0.8
    m.close()


def test_sampled_generation(pkg, ctx):
    cfg = config([channel(mlp=moe()), latent(mlp=dense(40))])
    m, _ = model(pkg, ctx, cfg, "bfloat16", seed=14, max_slots=2, max_seq=64)
    prompts = [tokens(cfg, n, seed=n) for n in (5, 9, 3)]
    a = m.generate(prompts, 12, temperature=0.9, seed=7)
    assert np.array_equal(a, m.generate(prompts, 12, temperature=0.9, seed=7))
    assert not np.array_equal(a, m.generate(prompts, 12, temperature=0.9, seed=8))
    assert np.array_equal(m.generate(prompts, 12), m.generate(prompts, 12, temperature=0.5, top_k=1, seed=3))
    m.close()


def test_preconditions(pkg, ctx):
    cfg = config([latent(mlp=moe()), channel()])
    w = L.as_bits(L.random_weights(cfg, 1))

    def refused(match, **change):
        m = pkg.Decoder(ctx, cfg, max_slots=2, max_seq=32)
        with pytest.raises(pkg.B200Error, match=match):
            m.load_tensors({k: v for k, v in {**w, **change}.items() if v is not None})
        m.close()

    table = w["l0.mlp.table"]
    bad = table.copy()
    bad[3, 1] = 5
    refused("expert that is not there", **{"l0.mlp.table": bad})
    bad = table.copy()
    bad[4, 1] = bad[4, 0]
    refused("twice", **{"l0.mlp.table": bad})
    refused("int32", **{"l0.mlp.table": table.astype(np.float32)})
    refused("bf16 or fp32", **{"l0.norm1": np.zeros(96, np.int32)})
    refused("l1.mix.a1", **{"l1.mix.a1": None})
    refused("shape", **{"l1.mix.a2": w["l1.mix.a2"][:, :-1]})
    refused("l0.mlp.e4.down", **{"l0.mlp.e4.down": None})


def test_commands(pkg, tmp_path):
    """bin/trace_run and bin/generate on a folder with config.json and model.safetensors."""
    cfg = config([channel(mlp=dense(30)), latent(mlp=moe())], loop=(1, 2, 2))
    w = L.random_weights(cfg, 15)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    L.save_safetensors(tmp_path / "model.safetensors", w)
    ta, tb = tokens(cfg, 40, seed=1), tokens(cfg, 25, seed=2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ta[:30].tolist(), "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": tb[:20].tolist(), "want": []}, {"id": "a", "tokens": ta[30:39].tolist(), "want": [8, 3]}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": ta[39:].tolist(), "want": [0]}, {"id": "b", "tokens": tb[20:21].tolist(), "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": tb[21:].tolist(), "want": [0, 1, 2, 3]}], "end": ["b"]}]
    wf = L.as_float64(w)
    A, B = L.forward(cfg, wf, ta), L.forward(cfg, wf, tb)
    want = {0: A[[0, 29]], 1: A[[38, 33]], 2: np.stack([A[39], B[20]]), 3: B[21:25]}
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(out), "--max-tokens", "70"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
        assert r.returncode == 0, r.stderr
        assert r.stdout.split("\n")[:4] == ["done 0", "done 1", "done 2", "done 3"]
        for k, v in want.items():
            check(np.fromfile(out / f"{k}.f32", "<f4").reshape(-1, cfg["vocab"]), v, TOL[dtype] * 1.5, f"step {k}")
    r = subprocess.run([os.path.join(ROOT, "bin", "generate"), "--model", str(tmp_path), "--dtype", "float32", "--new", "5", "--prompt", "1,2,3", "--prompt", "9"],
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    rows = [[int(t) for t in line.split(",")] for line in r.stdout.split()]
    for p, o in zip(([1, 2, 3], [9]), rows):
        assert o == [int(np.argmax(L.forward(cfg, wf, p + o[:i])[-1])) for i in range(5)]
