"""Layered decoders on the GPU against the plain oracle (oracle/layered.py, float64).

Logit errors are root mean squares over the vocabulary, relative to the root mean square of the logits.
TOL["float32"] is fp32 rounding; TOL["bfloat16"] what 8-bit significands of weights' products leave on models of
a few layers.  Attention tests use a `scale` that makes the softmax fall on one or a few keys, so that a key that is
missed, seen too early or mixed up changes the logits by far more than either."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import layered as L

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 3e-5, "bfloat16": 3e-2}


def mamba(inner=72, state=16, dt_rank=7, conv=4, ff=None):
    return {"type": "mamba1", "mixer": {"conv": conv, "dt_rank": dt_rank, "inner": inner, "state": state}, "mlp": ff and {"kind": "dense", "ff": ff}}


def delta(heads=4, kv_heads=2, dim=32, vdim=24, conv=4, ff=None):
    return {"type": "delta", "mixer": {"conv": conv, "dim": dim, "heads": heads, "kv_heads": kv_heads, "vdim": vdim}, "mlp": ff and {"kind": "dense", "ff": ff}}


def parallel(heads=4, kv_heads=2, dim=64, vdim=64, rot=32, base=1000.0, scale=0.4, width=56, ls=0.8, rs=1.2, ff=None):
    return {"type": "parallel", "mixer": {"left": {"dim": dim, "heads": heads, "kv_heads": kv_heads, "rot": {"base": base, "dims": rot}, "scale": scale,
                                                   "vdim": vdim}, "left_scale": ls, "right": {"width": width}, "right_scale": rs},
            "mlp": ff and {"kind": "dense", "ff": ff}}


def config(layers, width=96, vocab=211, eps=1e-5, scale=3.0):
    return {"architecture": "Vunolorn", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps}, "layers": layers}


def model(pkg, ctx, cfg, dtype, seed=1, tweak=None, **kw):
    w = L.random_weights(cfg, seed)
    if tweak:
        tweak(w)
    kw.setdefault("max_slots", 4)
    kw.setdefault("max_seq", 640)
    m = pkg.Decoder(ctx, cfg, dtype=dtype, **kw)
    m.load_tensors({k: (v.view(np.uint32) >> 16).astype(np.uint16) for k, v in w.items()})
    return m, L.as_float64(w)


def tokens(cfg, n, seed=5):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n)


def run(m, tok, portions):
    """Logits of every position of a sequence fed in the given portions (the last one repeats)."""
    slot = m.open()
    out, i, k = [], 0, 0
    while i < len(tok):
        n = min(portions[min(k, len(portions) - 1)], len(tok) - i)
        out.append(m.step([(slot, tok[i:i + n])], want=range(n)))
        i += n
        k += 1
    m.close_slot(slot)
    return np.concatenate(out)


def check(got, want, tol, what=""):
    e = np.sqrt(((got - want) ** 2).mean(1)) / np.sqrt((want ** 2).mean())
    # (where rounding meets a steep place - a sharp softmax, a small norm - a position may stray a little)
    bad = np.nonzero(e > tol)[0]
    assert bad.size <= 0.02 * len(e) and e.max() <= 2 * tol, f"{what}: {bad.size} of {len(e)} positions, first {bad[:8]}, worst {e.max():.2e} (limit {tol})"


MIXERS = {
    "mamba": [mamba()],
    "mamba_mlp": [mamba(inner=64, state=8, dt_rank=16, conv=3, ff=50)],
    "mamba_odd": [mamba(inner=52, state=5, dt_rank=3, conv=2, ff=33)],
    "mamba_one": [mamba(inner=33, state=1, dt_rank=1, conv=1)],
    "mamba_33": [mamba(inner=130, state=33, dt_rank=65, conv=5)],
    "mamba_100": [mamba(inner=40, state=100, dt_rank=4, conv=7)],
    "mamba_200": [mamba(inner=40, state=200, dt_rank=4)],
    "delta": [delta()],
    "delta_mlp": [delta(heads=3, kv_heads=3, dim=64, vdim=64, conv=2, ff=40)],
    "delta_odd": [delta(heads=6, kv_heads=2, dim=23, vdim=21, conv=3)],
    "delta_one": [delta(heads=1, kv_heads=1, dim=1, vdim=1, conv=1)],
    "delta_wide": [delta(heads=2, kv_heads=1, dim=128, vdim=160)],
    "delta_80": [delta(heads=4, kv_heads=4, dim=80, vdim=40, conv=6)],
    "delta_200": [delta(heads=2, kv_heads=1, dim=200, vdim=36)],
    "attention": [parallel(rs=0.0)],
    "min_gru": [parallel(ls=0.0)],
    "parallel_mlp": [parallel(ff=70)],
    "parallel_mqa": [parallel(heads=8, kv_heads=1, dim=32, vdim=48, rot=32, width=33)],
    "parallel_mha": [parallel(heads=3, kv_heads=3, dim=80, vdim=64, rot=20, width=100)],
    "parallel_128": [parallel(heads=4, kv_heads=1, dim=128, vdim=128, rot=64, scale=0.25)],
    "parallel_v128": [parallel(heads=2, kv_heads=1, dim=64, vdim=100, rot=0)],
    "parallel_256": [parallel(heads=2, kv_heads=1, dim=192, vdim=256, rot=192, scale=0.2)],
    "parallel_groups": [parallel(heads=12, kv_heads=2, dim=48, vdim=20, rot=2)],
    "parallel_10": [parallel(heads=10, kv_heads=1, dim=36, vdim=30, rot=36)],
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(MIXERS))
def test_each_mixer(pkg, ctx, name, dtype):
    """One layer of each mixer at several sizes: whole, token by token from the start, prompt then decoding, portions."""
    cfg = config(MIXERS[name])
    m, w = model(pkg, ctx, cfg, dtype)
    tok = tokens(cfg, 75)
    want = L.forward(cfg, w, tok)
    for portions in ([75], [1], [41, 1], [2, 3, 1, 17, 2], [33, 31, 2]):
        check(run(m, tok, portions), want, TOL[dtype], f"{name} {dtype} {portions}")
    m.close()


STACK = [mamba(ff=60), delta(), parallel(ff=48), delta(heads=2, kv_heads=2, dim=64, vdim=32, ff=36), parallel(heads=6, kv_heads=2, dim=48, vdim=40, rot=48),
         mamba(inner=100, state=32, dt_rank=12)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width,vocab,eps,scale", [(96, 211, 1e-5, 3.0), (50, 77, 1e-3, 1.0), (1, 3, 1e-6, 0.5), (264, 1030, 1e-6, 16.0)])
def test_stack_of_layers(pkg, ctx, dtype, width, vocab, eps, scale):
    """Every mixer in one model; portions of changing size down to two tokens; residual rows of several lengths."""
    cfg = config(STACK, width, vocab, eps, scale)
    m, w = model(pkg, ctx, cfg, dtype, seed=2)
    tok = tokens(cfg, 330, seed=width)
    want = L.forward(cfg, w, tok)
    tol = TOL[dtype] * (1.5 if dtype == "bfloat16" else 1)
    if width == 1:  # a row of one element is its own norm: signs, which 16-bit rounding may flip
        if dtype == "bfloat16":
            m.close()
            pytest.skip("rows of one element in 16-bit arithmetic")
        tol = 1e-3
    for portions in ([330], [129, 128, 1, 1, 2, 7, 2], [64], [300, 1]):
        check(run(m, tok, portions), want, tol, f"{dtype} {portions}")
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_first_tokens(pkg, ctx, dtype):
    cfg = config(STACK)
    m, w = model(pkg, ctx, cfg, dtype, seed=3)
    tok = tokens(cfg, 9)
    want = L.forward(cfg, w, tok)
    for n in range(1, 10):
        check(run(m, tok[:n], [n]), want[:n], TOL[dtype] * 1.5, f"prompt of {n}")
        check(run(m, tok[:n], [max(1, n - 3), 1]), want[:n], TOL[dtype] * 1.5, f"prompt of {n}, decoded")
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dims", [(64, 64), (128, 128), (64, 128), (160, 64)])
def test_far_keys_and_tile_borders(pkg, ctx, dtype, dims):
    """Each of the queries below finds one key, far away or just across a border of the kernels' 32-, 64-, 128- and
    256-key tiles: the query projection is the key projection behind a rotation of the width by one, and the token at
    place a is embedded as the rotated embedding of the token at place b, so that b's score for a stands out from
    hundreds.  In a prompt, in portions and decoded."""
    D, Dv = dims
    cfg = config([parallel(heads=2, kv_heads=1, dim=D, vdim=Dv, rot=0, scale=0.5, rs=0.0)], width=128, vocab=700)
    T = 600
    tok = (np.arange(T) * 11 + 3) % 700  # all different
    pairs = ((0, 599), (511, 598), (5, 513), (300, 512), (256, 511), (383, 384), (255, 257), (128, 256), (127, 129), (1, 128), (64, 127), (63, 64), (31, 32))

    def paired(w):
        w["l0.norm1"].fill(1.0)
        w["l0.mix.left.q"] = np.concatenate([np.roll(w["l0.mix.left.k"], -1, axis=1)] * 2)
        w["l0.mix.left.q.norm"].fill(1.0)
        w["l0.mix.left.k.norm"].fill(1.0)
        for a, b in pairs:
            w["embed"][tok[a]] = np.roll(w["embed"][tok[b]], 1)
    m, w = model(pkg, ctx, cfg, dtype, seed=4, tweak=paired)
    want = L.forward(cfg, w, tok)
    # the test is worth something: without its far key a query's logits are others altogether
    for a, b in pairs[:3]:
        lost = tok.copy()
        lost[a] = (T * 11 + 3) % 700
        assert np.sqrt(((L.forward(cfg, w, lost)[b] - want[b]) ** 2).mean() / (want ** 2).mean()) > 0.3
    for portions in ([600], [1, 127, 129, 2, 300, 1], [126, 1, 1, 1, 1, 124, 1, 1, 1, 2, 250, 1], [511, 1]):
        check(run(m, tok, portions), want, TOL[dtype], f"{dims} {portions}")
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_memory(pkg, ctx, dtype):
    """Slow decays and nearly closed gates: the state of the first tokens is still felt hundreds of tokens later, so
    a state that is lost, doubled or mixed up between portions shows at the end."""
    cfg = config([mamba(inner=64, state=16), delta(heads=2, kv_heads=1, dim=64, vdim=32), parallel(ls=0.0, width=64)])

    def slow(w):
        w["l0.mix.A_log"][:] = L.to_bf16(np.full_like(w["l0.mix.A_log"], -3.0))
        w["l0.mix.dt.b"][:] = -3.0
        w["l1.mix.A_log"][:] = -3.0
        w["l1.mix.dt_bias"][:] = -3.0
        w["l2.mix.right.z.b"][:] = -5.0
    m, w = model(pkg, ctx, cfg, dtype, seed=6, tweak=slow)
    tok = tokens(cfg, 420)
    want = L.forward(cfg, w, tok)
    cut = np.sqrt(((L.forward(cfg, w, tok[200:])[-1] - want[-1]) ** 2).mean()) / np.sqrt((want ** 2).mean())
    assert cut > 3 * TOL["bfloat16"], cut
    for portions in ([420], [5, 1], [150, 2, 33, 1, 64, 3], [128, 128, 128, 1]):
        check(run(m, tok, portions), want, TOL[dtype], str(portions))
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batches_of_unequal_requests(pkg, ctx, dtype):
    """Ragged steps - prompts, portions and single tokens of several requests together - against each request alone."""
    cfg = config(STACK)
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
        check(np.concatenate(got[i]), want[i], TOL[dtype] * 1.5, f"request {i} of {lens[i]} tokens")
    m.close()


@pytest.mark.parametrize("B", [1, 2, 3, 4, 5, 8, 9, 16])
def test_decode_batch_sizes(pkg, ctx, B):
    """The decode path at every padding of the batch, sequences at different positions, graph replays included."""
    cfg = config(STACK)
    m, w = model(pkg, ctx, cfg, "bfloat16", seed=9, max_slots=16, max_seq=160)
    toks = [tokens(cfg, 30 + 7 * i, seed=i) for i in range(B)]
    want = [L.forward(cfg, w, t) for t in toks]
    slots = [m.open() for _ in range(B)]
    for i in range(B):
        if len(toks[i]) > 6:
            m.step([(slots[i], toks[i][:-6])])
    for k in range(6):
        lg = m.step([(slots[i], toks[i][len(toks[i]) - 6 + k:][:1]) for i in range(B)])
        for i in range(B):
            check(lg[i:i + 1], want[i][len(toks[i]) - 6 + k:][:1], TOL["bfloat16"] * 1.5, f"sequence {i}, step {k}")
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_slots_are_reused(pkg, ctx, dtype):
    """A slot that held a longer sequence serves the next one as a fresh one would: bit for bit."""
    cfg = config(STACK)
    fresh, _ = model(pkg, ctx, cfg, dtype, seed=10, max_slots=1)
    t1, t2 = tokens(cfg, 400, seed=1), tokens(cfg, 90, seed=2)
    want = run(fresh, t2, [50, 1, 1, 5, 1])
    fresh.close()
    m, _ = model(pkg, ctx, cfg, dtype, seed=10, max_slots=1)
    for _ in range(2):
        run(m, t1, [300, 1, 40])
        assert np.array_equal(run(m, t2, [50, 1, 1, 5, 1]), want)
    with pytest.raises(pkg.B200Error, match="no free slot"):
        m.open(), m.open()
    m.close()


@pytest.mark.parametrize("layer,width", [
    (parallel(heads=12, kv_heads=3, dim=64, vdim=64, rot=64), 128),
    (parallel(heads=14, kv_heads=2, dim=128, vdim=128, rot=64, scale=0.2), 128),
    (delta(heads=12, kv_heads=6, dim=64, vdim=128), 128),
    (delta(heads=24, kv_heads=24, dim=64, vdim=128), 128),
    (delta(heads=16, kv_heads=4, dim=128, vdim=128), 128),
    (delta(heads=40, kv_heads=20, dim=32, vdim=128), 128),
    (mamba(inner=1300, state=16, ff=2600), 96)])
def test_large_steps_equal_small_ones(pkg, ctx, layer, width):
    """Steps of thousands of rows - persistent kernels with several items per CTA, paired-CTA products with the exact
    gelu in their epilogue, the delta rule's wider column groups - against each sequence alone."""
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
    # all of them once more, in one step from their start
    slots = [m.open() for _ in range(n)]
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
    cfg = config([delta(), parallel(), mamba(ff=40)])
    m, w = model(pkg, ctx, cfg, "bfloat16", seed=11, max_seq=600)
    tok = tokens(cfg, 560)
    check(run(m, tok, [3, 1]), L.forward(cfg, w, tok), TOL["bfloat16"], "557 tokens decoded one by one")
    m.close()


def test_steps_beyond_the_activation_buffers(pkg, ctx):
    """max_rows smaller than the step: it is cut, and the wanted rows come back in the order asked for."""
    cfg = config(STACK)
    m, w = model(pkg, ctx, cfg, "float32", seed=12, max_slots=3, max_seq=200, max_rows=48)
    toks = [tokens(cfg, n, seed=n) for n in (150, 20, 70)]
    want = np.concatenate([L.forward(cfg, w, t) for t in toks])
    slots = [m.open() for _ in toks]
    rows = np.random.default_rng(0).permutation(240)[:40]
    check(m.step(list(zip(slots, toks)), want=rows), want[rows], TOL["float32"])
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation(pkg, ctx, dtype):
    """More requests than slots, unequal prompts, prompts longer than max_rows, through the scheduler: every generated
    token is the oracle's arg-max after the tokens before it (up to a near-tie)."""
    cfg = config(STACK)
    m, w = model(pkg, ctx, cfg, dtype, seed=13, max_slots=3, max_seq=128, max_rows=40)
    prompts = [tokens(cfg, n, seed=n) for n in (1, 33, 90, 2, 57, 40, 8)]
    n_new = 14
    out = m.generate(prompts, n_new)
    assert out.shape == (len(prompts), n_new)
    for p, o in zip(prompts, out):
        lg = L.forward(cfg, w, np.concatenate([p, o[:-1]]))[len(p) - 1:]
        gap = lg.max(1) - lg[np.arange(n_new), o]
        assert gap.max() <= 3 * TOL[dtype] * np.sqrt((lg ** 2).mean()), gap
    assert all(m.length(s) == -1 for s in range(3))  # every slot was given back
    # and alone each request gets the same continuation (up to such near-ties in 16-bit arithmetic)
    alone = np.concatenate([m.generate([p], n_new) for p in prompts])
    if dtype == "float32":
        assert np.array_equal(alone, out)
    else:
        assert (alone == out).mean() > 0.8
    m.close()


def test_sampled_generation(pkg, ctx):
    cfg = config([delta(), parallel(ff=40)])
    m, _ = model(pkg, ctx, cfg, "float32", seed=14, max_slots=2, max_seq=64)
    prompts = [tokens(cfg, n, seed=n) for n in (5, 9, 3)]
    a = m.generate(prompts, 12, temperature=0.9, seed=7)
    assert np.array_equal(a, m.generate(prompts, 12, temperature=0.9, seed=7))
    assert not np.array_equal(a, m.generate(prompts, 12, temperature=0.9, seed=8))
    assert np.array_equal(a[0], m.generate(prompts[:1], 12, temperature=0.9, seed=7)[0])  # whatever else is active
    assert np.array_equal(m.generate(prompts, 12), m.generate(prompts, 12, temperature=0.5, top_k=1, seed=3))
    m.close()


def test_preconditions(pkg, ctx):
    cfg = config([mamba()])
    m = pkg.Decoder(ctx, cfg, max_slots=2, max_seq=32)
    w = {k: (v.view(np.uint32) >> 16).astype(np.uint16) for k, v in L.random_weights(cfg, 1).items()}
    with pytest.raises(pkg.B200Error, match="set up"):
        m.step([(0, [1])])
    with pytest.raises(pkg.B200Error, match="l0.mix.D"):
        m.load_tensors({k: v for k, v in w.items() if k != "l0.mix.D"})
    m.close()
    m = pkg.Decoder(ctx, cfg, max_slots=2, max_seq=32)
    with pytest.raises(pkg.B200Error, match="shape"):
        m.load_tensors({**w, "l0.mix.D": np.zeros(5, np.uint16)})
    m.close()
    with pytest.raises(pkg.B200Error, match="unknown mixer"):
        pkg.Decoder(ctx, config([dict(mamba(), type="x")]))
    m, _ = model(pkg, ctx, cfg, "bfloat16", max_slots=2, max_seq=32)
    s = m.open()
    for entries, what in (([(s, [1]), (s, [2])], "twice"), ([(1, [1])], "not open"), ([(s, [cfg["vocab"]])], "vocabulary"), ([(s, [-1, 2])], "vocabulary"),
                          ([(s, [1] * 33)], "max_seq"), ([(s, [])], "without tokens")):
        with pytest.raises(pkg.B200Error, match=what):
            m.step(entries)
    with pytest.raises(pkg.B200Error, match="wanted row"):
        m.step([(s, [1, 2])], want=[2])
    assert m.length(s) == 0
    assert m.step([(s, [1, 2])], want=[]).shape == (0, cfg["vocab"]) and m.length(s) == 2
    m.close()


def test_commands(pkg, tmp_path):
    """bin/trace_run and bin/generate on a folder with config.json and model.safetensors; bin/generate on a GPT-2 folder."""
    cfg = config([delta(), mamba(ff=20), parallel()])
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
            check(np.fromfile(out / f"{k}.f32", "<f4").reshape(-1, cfg["vocab"]), v, TOL[dtype], f"step {k}")
    r = subprocess.run([os.path.join(ROOT, "bin", "generate"), "--model", str(tmp_path), "--dtype", "float32", "--new", "5", "--prompt", "1,2,3", "--prompt", "9"],
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    rows = [[int(t) for t in line.split(",")] for line in r.stdout.split()]
    for p, o in zip(([1, 2, 3], [9]), rows):
        assert o == [int(np.argmax(L.forward(cfg, wf, p + o[:i])[-1])) for i in range(5)]
    g = tmp_path / "gpt2"
    g.mkdir()
    c = dict(architecture="GPT2", max_seq_len=128, vocab_size=500, padded_vocab_size=512, num_layers=1, num_heads=2, channels=128)
    (g / "config.json").write_text(json.dumps(c))
    n = pkg.param_offsets(pkg.GPT2Config(**{k: v for k, v in c.items() if k != "architecture"}))[16]
    (0.02 * np.random.default_rng(0).standard_normal(n)).astype(np.float32).tofile(g / "model.bin")
    r = subprocess.run([os.path.join(ROOT, "bin", "generate"), "--model", str(g), "--new", "6", "--prompt", "1,2,3"], capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    assert len(r.stdout.strip().split(",")) == 6
