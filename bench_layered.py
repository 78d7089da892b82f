"""bench.py --layered: prefill and decode throughput of the layered decoders: Vunolorn beside GPT-2, Pumotar beside Vunolorn, at
equal width and depth.

Random weights at sizes that resemble real layers (no checkpoint exists).  Prefill is 8 sequences of 1024 tokens in
one step (the GPT-2 benchmark's batch), logits of every position; decode is one token per sequence behind 1024 cached
ones, replayed as a CUDA graph.  Times are CUDA events on the launching stream after warm-up; activations and weights
are far beyond L2, so nothing is flushed.  Per operator: event time per launch and the fraction of its roofline, the
larger of bytes / HBM bandwidth and operations / peak of the unit that has to do them.
"""
from __future__ import annotations

import json

FP32_FMA = 148 * 128 * 2 * 1.965e9   # nominal fp32 operations per second
SFU = 148 * 16 * 1.965e9             # nominal special-function results per second
B, T = 8, 1024
VOCAB = 50304

SIZES = {
    # width, heads, kv_heads, ff, mamba inner, dt_rank, state, delta heads, delta kv_heads, delta dim, delta vdim, layers
    "768": dict(width=768, heads=12, kv=4, ff=3072, inner=1536, rank=48, state=16, dh=12, dkv=6, dd=64, dv=128, layers=12),
    "1600": dict(width=1600, heads=25, kv=5, ff=6400, inner=3200, rank=100, state=16, dh=25, dkv=25, dd=128, dv=128, layers=8),
}
PUMOTAR = {
    # ... experts, of which each token uses top, and the shared one; the channel delta rule as Vunolorn's delta rule
    "768": dict(width=768, heads=12, dim=64, rot=32, vdim=64, rank=256, ff=3072, experts=16, top=2, eff=768, sff=1536, dh=12, dkv=6, dd=64, dv=128, layers=12),
    "1600": dict(width=1600, heads=25, dim=64, rot=64, vdim=64, rank=512, ff=6400, experts=16, top=2, eff=1600, sff=3200, dh=25, dkv=25, dd=128, dv=128,
                 layers=8),
}


def make_pumotar(s):
    lat = {"heads": s["heads"], "dim": s["dim"], "rot_dim": s["rot"], "vdim": s["vdim"], "kv_rank": s["rank"], "scale": (s["dim"] + s["rot"]) ** -0.5,
           "rot": {"base": 10000.0, "dims": s["rot"]}}
    cd = {"conv": 4, "dim": s["dd"], "heads": s["dh"], "kv_heads": s["dkv"], "vdim": s["dv"], "ranks": [s["dd"], s["dv"]]}
    moe = {"kind": "moe", "expert": {"ff": s["eff"], "limit": 7.0}, "router": {"experts": s["experts"], "top": s["top"]},
           "shared": {"ff": s["sff"], "limit": 7.0}}
    layers = [{"type": "latent_attention" if i % 4 == 3 else "channel_delta", "mixer": lat if i % 4 == 3 else cd,
               "mlp": moe if i else {"kind": "dense", "ff": s["ff"]}} for i in range(s["layers"])]
    return {"architecture": "Pumotar", "vocab": VOCAB, "width": s["width"], "embedding": {"scale": 1.0}, "norm": {"eps": 1e-5}, "layers": layers}


def make_config(s):
    att = {"dim": 64, "heads": s["heads"], "kv_heads": s["kv"], "rot": {"base": 10000.0, "dims": 64}, "scale": 0.125, "vdim": 64}
    period = [{"type": "parallel", "mixer": {"left": att, "left_scale": 1.0, "right": {"width": s["width"]}, "right_scale": 1.0},
               "mlp": {"kind": "dense", "ff": s["ff"]}}]
    period += [{"type": "mamba1", "mixer": {"conv": 4, "dt_rank": s["rank"], "inner": s["inner"], "state": s["state"]}, "mlp": None}] * 2
    period += [{"type": "delta", "mixer": {"conv": 4, "dim": s["dd"], "heads": s["dh"], "kv_heads": s["dkv"], "vdim": s["dv"]}, "mlp": None}]
    return {"architecture": "Vunolorn", "vocab": VOCAB, "width": s["width"], "embedding": {"scale": 1.0}, "norm": {"eps": 1e-5},
            "layers": (period * ((s["layers"] + 3) // 4))[:s["layers"]]}


def random_tensors(torch, np, cfg):
    from oracle import layered
    g = torch.Generator(device="cuda").manual_seed(1)
    out = {}
    for name, shape in layered.tensor_shapes(cfg).items():
        if name.endswith(".table"):
            experts = cfg["layers"][int(name[1:].split(".")[0])]["mlp"]["router"]["experts"]
            t = torch.rand((shape[0], experts), device="cuda", generator=g).argsort(dim=1)[:, :shape[1]]
            out[name] = np.ascontiguousarray(t.to(torch.int32).cpu().numpy())
            continue
        t = torch.empty(shape, device="cuda").normal_(0.0, 1.0, generator=g)
        leaf = name.rsplit(".", 1)[-1]
        if "norm" in leaf or leaf == "D":
            t = 1.0 + 0.1 * t
        elif leaf == "A_log":
            t = t.abs()
        elif leaf == "dt_bias" or name.endswith(".dt.b"):
            t = t - 4.0
        elif len(shape) == 2:
            t = t / shape[1] ** 0.5
        out[name] = t.to(torch.bfloat16).view(torch.int16).cpu().numpy().view(np.uint16)
    return out


def operator_costs(cfg, M):
    """operator -> (bytes, tensor-core flop, fp32 operations, special-function results) of one launch with M rows of 8 sequences."""
    C = cfg["width"]
    P = lambda n: max(64, (n + 7) // 8 * 8)
    c = {}

    def gemm(name, K, N, out_bytes=4, rows=M):
        c[name] = (2.0 * rows * K + 2.0 * N * K + out_bytes * rows * N, 2.0 * rows * K * N, 0.0, 0.0)
    c["embed norm"] = (M * C * (2 + 4 + 2.0), 0, 0, 0)
    c["residual norms"] = (M * C * (4 + 4 + 4 + 2.0), 0, 0, 0)
    c["final norm"] = (M * C * (4 + 4 + 2.0), 0, 0, 0)
    gemm("gemm head", C, cfg["vocab"])
    for l in cfg["layers"]:
        m = l["mixer"]
        if l["type"] == "mamba1":
            n, r, s = m["inner"], m["dt_rank"], m["state"]
            gemm("gemm mamba1 in", C, 2 * n)
            c["conv mamba1"] = (M * n * (4 + 2.0), 0, M * n * 2.0 * m["conv"], M * n * 2.0)
            gemm("gemm mamba1 x", n, P(r) + 2 * s)
            c["slice"] = (M * r * 6.0, 0, 0, 0)
            gemm("gemm mamba1 dt", P(r), n)
            gemm("gemm mamba1 o", n, C)
            c["selective scan"] = (M * n * (2 + 4 + 4 + 2.0) + M * 8.0 * s, 0, M * n * s * 6.0, M * n * (s + 4.0))
        elif l["type"] == "latent_attention":
            H, D, Dr, Dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            gemm("gemm latent in", C, H * (D + Dr) + R + Dr)
            c["latent prep"] = (M * (H * (D + Dr) * 6.0 + (R + Dr) * 8.0), 0, 0, 0)
            gemm("gemm latent kv", R, H * (D + Dv), 2)
            c["attention"] = (M * H * (2 * (D + Dr) + 2 * Dv) * 2.0, 2.0 * H * (D + Dr + Dv) * M * (T + 1) / 2, 0, H * M * (T + 1) / 2.0)
            gemm("gemm latent o", H * Dv, C)
        elif l["type"] == "channel_delta":
            H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            ra, rg = m["ranks"]
            nc = 2 * G * D + H * Dv
            gemm("gemm delta in", C, nc + ra + rg + H)
            c["slice"] = (M * (ra + rg) * 6.0, 0, 0, 0)
            c["gemm delta low rank"] = (2.0 * M * (ra + rg) + 2.0 * H * (D * ra + Dv * rg) + 4.0 * M * H * (D + Dv), 2.0 * M * H * (D * ra + Dv * rg), 0, 0)
            c["conv delta v"] = (M * H * Dv * 8.0, 0, M * H * Dv * 2.0 * m["conv"], M * H * Dv * 2.0)
            c["delta prep"] = (M * 2 * G * D * 8.0 + M * H * (4 + 16.0) + M * H * D * 8.0, 0, M * 2 * G * D * (2.0 * m["conv"] + 5), M * (2 * G * D * 2.0 + H * D * 3.0))
            c["delta scan"] = (M * (nc + H * D + H * Dv + 4 * H) * 4.0, 0, M * H * D * Dv * 7.0, 0)
            c["head norm"] = (M * H * Dv * (4 + 4 + 2.0), 0, 0, M * H * Dv * 2.0)
            gemm("gemm delta o", H * Dv, C)
        elif l["type"] == "delta":
            H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            nc = 2 * G * D + H * Dv
            gemm("gemm delta in", C, P(nc + H * Dv + 2 * H))
            c["conv delta v"] = (M * H * Dv * 8.0, 0, M * H * Dv * 2.0 * m["conv"], M * H * Dv * 2.0)
            c["delta prep"] = (M * 2 * G * D * 8.0 + M * H * (8 + 16.0), 0, M * 2 * G * D * (2.0 * m["conv"] + 5), M * 2 * G * D * 2.0)
            c["delta scan"] = (M * (nc + H * Dv + 4 * H) * 4.0, 0, M * H * D * Dv * 6.0, 0)
            c["head norm"] = (M * H * Dv * (4 + 4 + 2.0), 0, 0, M * H * Dv * 2.0)
            gemm("gemm delta o", H * Dv, C)
        else:
            a, W = m["left"], m["right"]["width"]
            H, G, D, Dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            gemm("gemm parallel in", C, H * D + G * (D + Dv) + 3 * W)
            c["attention prep"] = (M * (H * D + G * (D + Dv)) * 6.0, 0, 0, 0)
            c["attention"] = (M * (H * (D + Dv) + G * (D + Dv)) * 2.0, 2.0 * H * (D + Dv) * M * (T + 1) / 2, 0, H * M * (T + 1) / 2.0)
            c["min gru"] = (M * W * 14.0, 0, 0, M * W * 6.0)
            gemm("gemm parallel o", H * Dv + W, C)
        f = l["mlp"]
        if f and f["kind"] == "moe":
            E, top, F, S = f["router"]["experts"], f["router"]["top"], f["expert"]["ff"], f["shared"]["ff"]
            c["residual norms experts"] = (M * C * (4 + 4 + 4 + 2.0 + 2 * top), 0, 0, 0)
            c["residual norms parts"] = (M * C * (4 + 4 + 4 * top + 4 + 2.0), 0, 0, 0)
            c["gemm experts up"] = (M * top * (2.0 * C + 2.0 * F) + 4.0 * E * F * C, 4.0 * M * top * C * F, 0, M * top * F * 2.0)
            c["gemm experts down"] = (M * top * (2.0 * F + 4.0 * C) + 2.0 * E * F * C, 2.0 * M * top * C * F, 0, 0)
            c["gemm shared up"] = (M * (2.0 * C + 2.0 * S) + 4.0 * S * C, 4.0 * M * C * S, 0, M * S * 2.0)
            c["gemm shared down"] = (M * (2.0 * S + 4.0 * C) + 2.0 * S * C, 2.0 * M * C * S, 0, 0)
            c["expert routes"] = (M * top * 8.0, 0, 0, 0)
        elif f:
            gates = 2 if cfg["architecture"] == "Pumotar" else 1
            c["gemm mlp up"] = (2.0 * M * C + 2.0 * gates * f["ff"] * C + 2.0 * M * f["ff"], 2.0 * gates * M * C * f["ff"], 0, 0)
            gemm("gemm mlp down", f["ff"], C)
    return c


def gpt2_costs(C, NH, M, V, vp):
    g = lambda K, N, o: (4.0 * M * K + 4.0 * N * K + o * M * N, 3 * 2.0 * M * K * N, 0, 0)  # split-bf16: three products
    return {"encoder": (M * C * 8.0, 0, 0, 0), "layernorm": (M * C * 8.0, 0, 0, 0), "gemm_qkv": g(C, 3 * C, 4), "gemm_attproj": g(C, C, 8),
            "gemm_fc": g(C, 4 * C, 4), "gemm_fcproj": g(4 * C, C, 8), "gemm_lmhead": g(C, vp, 4),
            "attention": (M * C * (2 * 2 + 4 + 4.0), 2.0 * C * M * (T + 1) / 2 * 3, 0, NH * M * (T + 1) / 2.0)}


def roofline(costs, prof, peaks):
    rows = {}
    for name, (ms, n) in prof.items():
        if n == 0:
            continue
        us = ms * 1e3 / n
        row = {"us": round(us, 1), "launches": n}
        if name in costs:
            by, mma, fma, sfu = costs[name]
            limits = {"hbm": by / (peaks["hbm_gbs"] * 1e9), "tensor": mma / (peaks["bf16_burst"] * 1e12), "fp32": fma / FP32_FMA, "sfu": sfu / SFU}
            bound = max(limits, key=limits.get)
            row.update(bound=bound, roofline_us=round(limits[bound] * 1e6, 1), fraction=round(limits[bound] * 1e6 / us, 3))
        rows[name] = row
    return rows


def run(args, load_package, peaks, sampler):
    import numpy as np
    import torch
    pkg = load_package()
    torch.cuda.set_device(0)
    stream = torch.cuda.Stream()
    ctx = pkg.Context(0, stream)
    rng = np.random.default_rng(0)

    def timed(fn, steps, warmup):
        for _ in range(warmup):
            fn()
        ctx.sync_check()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record(stream)
        for _ in range(steps):
            fn()
        e1.record(stream)
        ctx.sync_check()
        return e0.elapsed_time(e1) / steps

    def measure(cfg, label):
        M = B * T
        m = pkg.Decoder(ctx, cfg, "bfloat16", max_slots=16, max_seq=T + 256, max_rows=M)
        m.load_tensors(random_tensors(torch, np, cfg))
        toks = [rng.integers(0, VOCAB, T).astype(np.int32) for _ in range(B)]
        want = np.arange(M, dtype=np.int32)

        def prefill(w=want, keep=False, n=B):
            slots = [m.open() for _ in range(n)]
            m.prefill_device([(slots[i], toks[i % B]) for i in range(n)], w)
            if not keep:
                for x in slots:
                    m.close_slot(x)
            return slots
        pre_ms = timed(prefill, args.steps, args.warmup)
        m.set_profile(True)
        prefill()
        ctx.sync_check()
        m.read_profile()
        for _ in range(3):
            prefill()
        prof = m.read_profile()
        m.set_profile(False)
        out = {"model": label, "data": "synthetic", "dtype": "bf16",
               "prefill": {"batch": B, "seq_len": T, "ms": round(pre_ms, 3), "tokens_per_s": round(M / pre_ms * 1e3), "logits": "every position"},
               "decode": {}}
        one = timed(lambda: prefill(np.arange(B) * T + T - 1), args.steps, args.warmup)
        out["prefill_last_logits_only"] = {"ms": round(one, 3), "tokens_per_s": round(M / one * 1e3)}
        single = timed(lambda: prefill(np.array([T - 1]), n=1), args.steps, args.warmup)
        out["prefill_one_sequence"] = {"ms": round(single, 3), "tokens_per_s": round(T / single * 1e3)}
        for b in (1, 8, 16):
            slots = []
            for first in range(0, b, B):
                n = min(B, b - first)
                slots += prefill(np.arange(n) * T + T - 1, keep=True, n=n)
            if cfg["architecture"] == "Pumotar":  # ids of the device's token buffer choose the experts: unequal ones
                m.step([(x, [int(t)]) for x, t in zip(slots, rng.integers(0, VOCAB, b))])
            ms = timed(lambda: m.decode_device(slots), 64, 8)
            out["decode"][b] = {"us_per_step": round(ms * 1e3, 1), "tokens_per_s": round(b / ms * 1e3)}
            for x in slots:
                m.close_slot(x)
        out["operators"] = roofline(operator_costs(cfg, M), prof, peaks)
        m.close()
        return out, toks

    names = list(SIZES) + ["pumotar-" + n for n in PUMOTAR] if args.layered == "all" else args.layered.split(",")
    for name in names:
        M = B * T
        sampler.start()
        size = name.split("-")[-1]
        if name.startswith("pumotar"):
            s = PUMOTAR[size]
            out, _ = measure(make_pumotar(s), f"Pumotar {s['layers']} layers, width {s['width']}")
            s = SIZES[size]
            out["closest_model"], _ = measure(make_config(s), f"Vunolorn {s['layers']} layers, width {s['width']}")
            out["clocks"] = sampler.stop()
            out["peaks"] = peaks
            print(json.dumps(out), flush=True)
            continue
        s = SIZES[name]
        out, toks = measure(make_config(s), f"Vunolorn {s['layers']} layers, width {s['width']}")
        # GPT-2 of the same width and depth in the framework's default arithmetic
        gc = pkg.GPT2Config(num_layers=s["layers"], num_heads=s["width"] // 64, channels=s["width"])
        g2 = pkg.GPT2(ctx, gc, B, T)
        gp = torch.Generator(device="cuda").manual_seed(2)
        g2.params_tensor().normal_(0.0, 0.02, generator=gp)
        torch.cuda.synchronize()
        tok = torch.from_numpy(np.stack(toks)).cuda() % gc.vocab_size
        torch.cuda.synchronize()
        ref = {}
        ms = timed(lambda: g2.forward(tok, B, T), args.steps, args.warmup)
        ref["prefill"] = {"ms": round(ms, 3), "tokens_per_s": round(M / ms * 1e3)}
        g2.set_profile(True)
        g2.forward(tok, B, T)
        g2.read_profile()
        for _ in range(3):
            g2.forward(tok, B, T)
        gprof = g2.read_profile()
        g2.set_profile(False)
        g2.set_options(use_graph=1)
        g2.enable_kv_cache()
        g2.prefill(tok, B, T)
        ref["decode"] = {}
        for b in (1, 8):
            col = tok[:b, 0].contiguous()
            torch.cuda.synchronize()
            ms = timed(lambda: g2.decode_step(col, b, T - 1), 64, 8)
            ref["decode"][b] = {"us_per_step": round(ms * 1e3, 1), "tokens_per_s": round(b / ms * 1e3)}
        ref["operators"] = roofline(gpt2_costs(s["width"], s["width"] // 64, M, gc.vocab_size, gc.padded_vocab_size), gprof, peaks)
        g2.close()
        out["gpt2_same_width_and_depth"] = ref
        out["clocks"] = sampler.stop()
        out["peaks"] = peaks
        print(json.dumps(out), flush=True)
    ctx.close()
    return 0
