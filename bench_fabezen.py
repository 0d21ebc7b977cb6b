"""Throughput of Fabezen decoders (gated delta rules, latent attention in a window, gated GELU feed-forward) at sizes that resemble a
real model's layers, random weights, beside the closest existing model (the hybrid decoder of retention and differential attention)
at equal size: `python bench.py --workload fabezen`.  Prints one JSON line.  Timing and rooflines as in bench_hybrid.py."""
import json

import bench_hybrid as B

SIZES = {str(w): dict(width=w, vocab=32768, heads=w // 128, kv=w // 256, dim=128, vdim=128, conv=4, rank=128, lheads=w // 128, ldim=128, rot=64, lvdim=128,
                      kv_rank=512, q_rank=min(1536, 3 * w // 4), window=4096, ff=3 * w) for w in (1024, 2048, 4096)}
LAYERS = 8


def fabezen_config(s, layers=LAYERS):
    """channel_delta, delta, channel_delta, latent_attention, each with a feed-forward, repeated."""
    mlp = {"kind": "dense", "ff": s["ff"]}
    d = lambda kind, kv: {"type": kind, "mixer": {"heads": s["heads"], "kv_heads": kv, "dim": s["dim"], "vdim": s["vdim"], "conv": s["conv"]}, "mlp": mlp}  # noqa: E731
    lat = {"type": "latent_attention", "mlp": mlp, "mixer": {
        "heads": s["lheads"], "dim": s["ldim"], "rot_dim": s["rot"], "vdim": s["lvdim"], "kv_rank": s["kv_rank"], "q_rank": s["q_rank"],
        "scale": (s["ldim"] + s["rot"]) ** -0.5, "mask": {"size": s["window"]}, "rot": {"base": 1e5, "dims": s["rot"]}}}
    return {"architecture": "Fabezen", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-5}, "residual_mult": 0.7,
            "embedding": {"scale": 8.0, "bigram": {"buckets": 8191, "mul_prev": 31, "mul_cur": 7}},
            "layers": [d("channel_delta", s["heads"]), d("delta", s["kv"]), d("channel_delta", s["heads"]), lat] * (layers // 4)}


def like_config(s, layers=LAYERS):
    """The closest existing model: retention and differential attention of the same heads, each with a feed-forward of the same width
    (scans have no counterpart here)."""
    mlp = {"kind": "dense", "ff": s["ff"]}
    h = s["heads"]
    ret = {"type": "retention", "mlp": mlp, "mixer": {"heads": h, "dim": s["dim"], "vdim": s["vdim"], "rot": {"base": 10000.0, "dims": s["dim"]},
                                                      "decay": [1 - 2.0 ** (-5 - 7 * i / h) for i in range(h)]}}
    att = {"type": "attention", "mlp": mlp, "mixer": {"heads": h, "kv_heads": s["kv"], "dim": 64, "vdim": 128, "scale": 0.125, "diff": 0.5}}
    return {"architecture": "Sebesun", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-5}, "layers": [ret, ret, ret, att] * (layers // 4)}


def kernels(pkg, torch, pk, s, T=2048, ctx=8192, only=""):
    X, HM = pkg.sc_mixers, pkg.host_model
    W, BF, F32 = s["width"], torch.bfloat16, torch.float32
    t = B.Timer(torch, pk)
    rnd = lambda *sh, dtype=BF: (torch.randn(*sh, device="cuda") * 0.5).to(dtype)          # noqa: E731
    H, d, dv, ra, ff = s["heads"], s["dim"], s["vdim"], s["rank"], s["ff"]
    lh, ld, r, lv, R, Q, win = s["lheads"], s["ldim"], s["rot"], s["lvdim"], s["kv_rank"], s["q_rank"], s["window"]

    def kernel(name, *a, **k):
        if only in name:
            t.kernel(name, *a, **k)

    def gemm(name, n, k, out=BF, act=None):
        def make(i):
            lin, x = X.Linear(rnd(n, k)), rnd(T, k)
            return lambda: lin(x, out, act=act)
        nout = n // 2 if act is not None else n
        kernel(name, make, 2 * (T * k + n * k) + T * nout * (4 if out == F32 else 2), 2.0 * T * n * k)

    gemm("prefill gemm channel in", 3 * H * d + 2 * ra + H, W)
    gemm("prefill gemm channel decays", H * d, ra, F32)
    gemm("prefill gemm channel gates", H * dv, ra)
    gemm("prefill gemm delta in", 2 * s["kv"] * d + 2 * H * dv + 2 * H, W)
    gemm("prefill gemm latent in", Q + R + r, W)
    gemm("prefill gemm latent queries", lh * (ld + r), Q)
    gemm("prefill gemm latent keys values", lh * (ld + lv), R)
    gemm("prefill gemm o", W, H * dv, F32)
    gemm("prefill gemm gate|up gelu", 2 * ff, W, act=X.GatedGELU())
    gemm("prefill gemm down", W, ff, F32)

    def embed(i):
        table, pairs, ids = rnd(s["vocab"], W), rnd(8192, W), torch.randint(0, s["vocab"], (T,), device="cuda")
        x, prev = torch.empty(T, W, device="cuda"), torch.full((1,), -1, dtype=torch.long, device="cuda")
        return lambda: X.embed_pair(ids, table, x, 2.0, pairs, (8191, 31, 7), prev)
    kernel("prefill embedding", embed, 8 * T * W)

    C = 2 * H * d + H * dv

    def conv(i):
        x, w, tail = rnd(T, C), rnd(C, s["conv"], dtype=F32), torch.zeros(C, s["conv"] - 1, device="cuda")
        return lambda: X.conv_silu(x, w, None, tail)
    kernel("prefill conv", conv, 4 * T * C)

    def delta(channel, G):
        def make(i):
            q, k, v = rnd(T, 2 * G * d + H * dv).split([G * d, G * d, H * dv], 1)
            b, a = rnd(T, H), rnd(T, H * d, dtype=F32) if channel else rnd(T, H)
            nA, dtb, st = -torch.rand(H, device="cuda"), rnd(a.shape[1], dtype=F32), torch.zeros(H, d, dv, device="cuda")
            return lambda: X.delta(q, k, v, b, a, channel, nA, dtb, st)
        return make
    chunk = 64        # within a chunk: two score products, inverse applied to keys and values, weighted corrections; across: three products with the state
    flops = 2.0 * T * H * (chunk / 2 * (3 * d + 2 * dv) + 3 * d * dv)
    kernel("prefill delta per channel", delta(True, H), T * H * (2 * (2 * d + dv) + 4 * d + 4 * dv), flops)
    kernel("prefill delta per head", delta(False, s["kv"]), T * (4 * s["kv"] * d + H * dv * 6), flops)

    def gate(i):
        o, g, w = rnd(T, H, dv, dtype=F32), rnd(T, H * dv), rnd(dv, dtype=F32)
        return lambda: X.head_norm_gate(o, g, 1e-5, w, 1)
    kernel("prefill head norm gate", gate, 8 * T * H * dv)

    def addnorm(n):
        def make(i):
            y, x, w, h = rnd(n, W, dtype=F32), rnd(n, W, dtype=F32), rnd(W, dtype=F32), torch.empty(n, W, dtype=BF if n > 1 else F32, device="cuda")
            return lambda: X.add_norm(y, x, w, 0.7, 1e-5, h)
        return make
    kernel("prefill residual + norm", addnorm(T), T * W * 14)

    def latent_cache(n, full=True):
        c = HM.LatentCache(R, r, n, "cuda", BF)
        if full:
            c.c.normal_()
        return c

    def append(i):
        y, c = rnd(T, Q + R + r), latent_cache(T, False)
        qw, cw, cs = rnd(Q, dtype=F32), rnd(R, dtype=F32), X.rotary_table(1e5, r, T, "cuda")
        return lambda: X.latent_append(y, Q, R, r, qw, cw, cs, 1e-5, c, BF)
    kernel("prefill latent append", append, 4 * T * (Q + R + r))
    cs = X.rotary_table(1e5, r, ctx, "cuda")

    def prompt(i):       # W_uk, W_uv apart: rotation and attention alone, on products made before
        c, q, kv = latent_cache(T), rnd(T, lh * (ld + r)), rnd(T, lh * (ld + lv))
        return lambda: X.latent_prompt(q, lambda rows: kv, cs, c, lh, ld, r, lv, R, win, (ld + r) ** -0.5)
    pairs = sum(min(i + 1, win) for i in range(T))
    kernel("prefill latent rotate + attention", prompt, 2 * T * (lh * (2 * ld + r + 2 * lv) + r), 2.0 * pairs * lh * (ld + r + lv))

    # ---- decode
    def gemv(name, n, k, act=None):
        def make(i):
            lin, x, o = X.Linear(rnd(n, k)), rnd(k, dtype=F32), torch.empty(n, device="cuda")
            return lambda: lin.vec(x, act=act, out=o)
        kernel(name, make, 2 * n * k + 4 * (n + k))
    gemv("decode gemv channel in", 3 * H * d + 2 * ra + H, W)
    gemv("decode gemv delta in", 2 * s["kv"] * d + 2 * H * dv + 2 * H, W)
    gemv("decode gemv latent in", Q + R + r, W)
    gemv("decode gemv latent queries", lh * (ld + r), Q)
    gemv("decode gemv o", W, H * dv)
    gemv("decode gemv gate|up gelu", 2 * ff, W, X.GatedGELU())
    gemv("decode gemv down", W, ff)
    gemv("decode gemv head", s["vocab"], W)

    def step(channel, G):
        def make(i):
            st, y, w = torch.zeros(H, d, dv, device="cuda"), torch.empty(H * dv, device="cuda"), rnd(dv, dtype=F32)
            q, k, v, b = rnd(G * d, dtype=F32), rnd(G * d, dtype=F32), rnd(H * dv, dtype=F32), rnd(H, dtype=F32)
            a, g = (rnd(ra, dtype=F32), rnd(ra, dtype=F32)) if channel else (rnd(H, dtype=F32), rnd(H * dv, dtype=F32))
            wa, wg = (X.Linear(rnd(H * d, ra)), X.Linear(rnd(H * dv, ra))) if channel else (None, None)
            nA, dtb = -torch.rand(H, device="cuda"), rnd(H * d if channel else H, dtype=F32)
            return lambda: X.delta_step(q, k, v, b, a, g, wa, wg, nA, dtb, w, 1e-5, st, y)
        return make
    kernel("decode delta step per channel", step(True, H), 8 * H * d * dv + 2 * ra * H * (d + dv))
    kernel("decode delta step per head", step(False, s["kv"]), 8 * H * d * dv)

    def append1(i):
        y, c, qw, cw = rnd(1, Q + R + r, dtype=F32), latent_cache(64), rnd(Q, dtype=F32), rnd(R, dtype=F32)
        return lambda: X.latent_append(y, Q, R, r, qw, cw, cs, 1e-5, c, F32)
    kernel("decode latent append", append1, 8 * (Q + R + r))
    for n in (1024, ctx):
        def rows(i):
            c, q, w = latent_cache(n), rnd(1, lh * (ld + r), dtype=F32), X.Linear(rnd(lh * (ld + lv), R))
            uk, uv = w.rows(0, lh * ld), w.rows(lh * ld, lh * (ld + lv))
            c.offset = n - 1
            return lambda: X.latent_rows(q, uk, uv, cs, c, lh, ld, r, lv, win, (ld + r) ** -0.5, F32)
        kernel(f"decode latent attention (3 kernels) ctx {n}", rows, 2 * (min(n, win) * (R + r) + lh * (ld + lv) * R))
    kernel("decode residual + norm", addnorm(1), W * 4 * 5)
    return t.rows


def run(pkg, torch, pk, sampler, sizes=None):
    torch.manual_seed(0)
    torch.cuda.set_device(0)
    out = {"workload": "fabezen", "layers": LAYERS, "data": "synthetic weights and token ids", "peaks": pk,
           "timing": "CUDA graph over copies of each call on different buffers, larger than L2 together", "sizes": {}}
    with sampler as clk:
        for name in sizes or SIZES:
            s = SIZES[name]
            models = {"fabezen": B.measure_hybrid(pkg, torch, pk, fabezen_config(s), rank=s["rank"]), "hybrid": B.measure_hybrid(pkg, torch, pk, like_config(s))}
            out["sizes"][name] = {"config": s, "models": models, "kernels": {"fabezen": kernels(pkg, torch, pk, s),
                                                                            "hybrid": B.hybrid_kernels(pkg, torch, pk, {**B.SIZES[name], "rvdim": s["vdim"]})}}
    out["clocks"] = clk.summary()
    pkg._lib.check_mixer_status()
    print(json.dumps(out))
