"""Throughput of hybrid decoders (selective scan, retention, differential attention) at sizes that resemble a real model's
layers, random weights, beside the closest existing model (the Qwen3-style W4A8 decoder) at equal size: `python bench.py
--workload hybrid`.  Prints one JSON line.

Every kernel is timed from a CUDA graph that runs copies of the call on different buffers (together larger than L2), and set
against its roofline: algorithmic bytes over the measured copy bandwidth, operations over the measured bf16 rate (INT8: twice
that), for the scan also exponentials over the special-function rate.  `frac` = roofline time / measured time."""
import json

import numpy as np

SIZES = {
    "1024": dict(width=1024, vocab=32768, inner=2048, state=16, rank=64, conv=4, rheads=8, rdim=128, rvdim=256, heads=8, kv=4, dim=64, vdim=128, ff=3072),
    "2048": dict(width=2048, vocab=32768, inner=4096, state=16, rank=128, conv=4, rheads=16, rdim=128, rvdim=256, heads=16, kv=8, dim=64, vdim=128, ff=6144),
    "4096": dict(width=4096, vocab=32768, inner=8192, state=16, rank=256, conv=4, rheads=32, rdim=128, rvdim=256, heads=32, kv=8, dim=64, vdim=128, ff=12288),
}
LAYERS = 8


def hybrid_config(s, layers=LAYERS):
    """mamba1, retention, mamba1, attention + feed-forward, repeated."""
    mam = {"type": "mamba1", "mixer": {"inner": s["inner"], "state": s["state"], "dt_rank": s["rank"], "conv": s["conv"]}, "mlp": None}
    ret = {"type": "retention", "mixer": {"heads": s["rheads"], "dim": s["rdim"], "vdim": s["rvdim"], "rot": {"base": 10000.0, "dims": s["rdim"]},
                                          "decay": [1 - 2.0 ** (-5 - 7 * h / s["rheads"]) for h in range(s["rheads"])]}, "mlp": None}
    att = {"type": "attention", "mixer": {"heads": s["heads"], "kv_heads": s["kv"], "dim": s["dim"], "vdim": s["vdim"], "scale": s["dim"] ** -0.5,
                                          "diff": 0.5}, "mlp": {"kind": "dense", "ff": s["ff"]}}
    return {"architecture": "Sebesun", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-5}, "layers": [mam, ret, mam, att] * (layers // 4)}


class Timer:
    def __init__(self, torch, pk):
        self.torch, self.pk, self.rows = torch, pk, {}

    def graph(self, fns):
        torch = self.torch
        s = torch.cuda.Stream()
        s.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(s), torch.no_grad():
            for f in fns:
                f()
            torch.cuda.synchronize()
            g = torch.cuda.CUDAGraph()
            with torch.cuda.graph(g, stream=s):
                for f in fns:
                    f()
        torch.cuda.current_stream().wait_stream(s)
        return g

    def replay_ms(self, g, reps=7):
        torch = self.torch
        ts = []
        for i in range(3 + reps):
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            g.replay()
            e1.record()
            torch.cuda.synchronize()
            if i >= 3:
                ts.append(e0.elapsed_time(e1))
        return float(np.median(ts))

    def kernel(self, name, make, nbytes, flops=0.0, int8=False, sfu=0.0, foot=None):
        """make(i) -> closure on its own buffers; foot: bytes one closure touches (for the number of copies)."""
        copies = int(max(2, min(24, 4e8 // max(foot or nbytes, 1) + 1)))
        fns = [make(i) for i in range(copies)]
        g = self.graph(fns)
        ms = self.replay_ms(g) / copies
        bound = max(nbytes / (self.pk["hbm_gbs"] * 1e9), flops / (self.pk["bf16_tflops"] * 1e12 * (2 if int8 else 1)), sfu / (148 * 16 * 1.965e9)) * 1e3
        self.rows[name] = dict(us=round(ms * 1e3, 2), roofline_us=round(bound * 1e3, 2), frac=round(bound / ms, 3))
        if flops:
            self.rows[name]["tflops"] = round(flops / ms / 1e9, 1)
        else:
            self.rows[name]["gbs"] = round(nbytes / ms / 1e6, 1)
        del g, fns
        self.torch.cuda.empty_cache()


def bench_kernels(pkg, torch, pk, s):
    """Kernels of the hybrid model and the like kernels of the closest model at the same sizes."""
    return dict(hybrid=hybrid_kernels(pkg, torch, pk, s), qwen3_style=qwen3_kernels(pkg, torch, pk, s))


def hybrid_kernels(pkg, torch, pk, s, T=2048, ctx=8192):
    X, HM = pkg.sc_mixers, pkg.host_model
    W, C, N, R, BF, F32 = s["width"], s["inner"], s["state"], s["rank"], torch.bfloat16, torch.float32
    t = Timer(torch, pk)
    rnd = lambda *sh, dtype=BF: (torch.randn(*sh, device="cuda") * 0.5).to(dtype)          # noqa: E731
    half = 2

    def gemm(name, n, k, out=BF, act=None):
        def make(i):
            lin, x = X.Linear(rnd(n, k)), rnd(T, k)
            return lambda: lin(x, out, act=act)
        t.kernel(name, make, half * (T * k + n * k) + T * n * (4 if out == F32 else 2), 2.0 * T * n * k)

    H, G_, d, dv, ff = s["heads"], s["kv"], s["dim"], s["vdim"], s["ff"]
    rh, rd, rv = s["rheads"], s["rdim"], s["rvdim"]
    act = X.XIELU(torch.tensor([0.3, -0.2]))
    gemm("prefill gemm mamba in", 2 * C, W)
    gemm("prefill gemm mamba x", R + 2 * N, C)
    gemm("prefill gemm mamba dt", C, R, F32)
    gemm("prefill gemm mamba o", W, C, F32)
    gemm("prefill gemm retention qkvg", 2 * rh * (rd + rv), W)
    gemm("prefill gemm retention o", W, rh * rv, F32)
    gemm("prefill gemm attention qkv", 2 * (H + G_) * d + G_ * dv, W)
    gemm("prefill gemm up xielu", ff, W, act=act)
    gemm("prefill gemm down", W, ff, F32)

    def conv(i):
        x, w, b, tail = rnd(T, 2 * C), rnd(C, s["conv"], dtype=F32), rnd(C, dtype=F32), torch.zeros(C, s["conv"] - 1, device="cuda")
        return lambda: X.conv_silu(x[:, :C], w, b, tail)
    t.kernel("prefill conv", conv, 4 * T * C, foot=6 * T * C)

    def scan(i):
        x, z, bc, dtp = rnd(T, C), rnd(T, C), rnd(T, 2 * N), rnd(T, C, dtype=F32)
        b, A2, D, st = rnd(C, dtype=F32), -torch.rand(C, N, device="cuda") * 3, rnd(C, dtype=F32), torch.zeros(C, N, device="cuda")
        return lambda: X.selective_scan(x, dtp, bc, z, b, A2, D, st)
    t.kernel("prefill scan", scan, T * C * 10 + T * 4 * N, sfu=float(T) * C * N)

    def reten(i):
        qkv, st = rnd(T, 2 * rh * rd + rh * rv), torch.zeros(rh, rd, rv, device="cuda")
        q, k, v = qkv.split([rh * rd, rh * rd, rh * rv], 1)
        cs, dec = X.rotary_table(1e4, rd, T, "cuda"), torch.full((rh,), 0.99, device="cuda")
        return lambda: X.retention(q, k, v, cs, rd, rd ** -0.5, dec, st)
    chunk = 256      # within a chunk: scores and weighted values; across chunks: state update and state product
    t.kernel("prefill retention", reten, 2 * T * rh * (2 * rd + rv) + 4 * T * rh * rv, 2.0 * T * rh * (chunk / 2 * (rd + rv) + 2 * rd * rv))

    def gate(i):
        o, g = rnd(T, rh, rv, dtype=F32), rnd(T, rh * rv)
        return lambda: X.head_norm_gate(o, g, 1e-5)
    t.kernel("prefill head norm gate", gate, 8 * T * rh * rv)

    def prep(i):
        q, k, v = rnd(T, 2 * (H + G_) * d + G_ * dv).split([2 * H * d, 2 * G_ * d, G_ * dv], 1)
        c, w = HM.KVCache(2 * G_, d, T, "cuda", BF, G_, dv), rnd(d, dtype=F32)
        return lambda: X.qk_norm_append(q, k, v, H, G_, w, w, 1e-5, c, BF)
    t.kernel("prefill qk norm append", prep, 4 * T * (2 * (H + G_) * d + G_ * dv))

    def attn(i):
        c, q = HM.KVCache(2 * G_, d, T, "cuda", BF, G_, dv), rnd(2 * H, T, d)
        c.k.normal_(), c.v.normal_()
        return lambda: X.diff_attention(q, c, H, G_, d ** -0.5, 0.4, 0.5, 1e-5)
    t.kernel("prefill diff attention", attn, 2 * T * (2 * (H + G_) * d + (G_ + H) * dv), 2.0 * T * T * H * (d + dv))

    def resnorm(n):
        def make(i):
            y, x, w = rnd(T, W, dtype=F32), rnd(T, W, dtype=F32), rnd(W, dtype=F32)
            xs, dwa, h = (rnd(n, T, W, dtype=F32), rnd(n, dtype=F32), torch.empty(T, W, dtype=BF, device="cuda")) if n else (None, None, torch.empty(T, W, dtype=BF, device="cuda"))
            return lambda: X.res_norm(y, x, w, 1e-5, x, h, (xs, dwa, True) if n else None)
        return make
    t.kernel("prefill residual norm", resnorm(0), T * W * 14)
    t.kernel("prefill residual norm + average of 6", resnorm(6), T * W * (14 + 4 * 6))

    # ---- decode
    def gemv(name, n, k):
        def make(i):
            lin, x, o = X.Linear(rnd(n, k)), rnd(k, dtype=F32), torch.empty(n, device="cuda")
            return lambda: lin.vec(x, out=o)
        t.kernel(name, make, 2 * n * k + 4 * (n + k))
    gemv("decode gemv mamba in", 2 * C, W)
    gemv("decode gemv mamba x", R + 2 * N, C)
    gemv("decode gemv mamba o", W, C)
    gemv("decode gemv retention qkvg", 2 * rh * (rd + rv), W)
    gemv("decode gemv attention qkv", 2 * (H + G_) * d + G_ * dv, W)
    gemv("decode gemv up", ff, W)
    gemv("decode gemv down", W, ff)
    gemv("decode gemv head", s["vocab"], W)

    def sstep(i):
        x, z, dbc, w = rnd(C, dtype=F32), rnd(C, dtype=F32), rnd(R + 2 * N, dtype=F32), X.Linear(rnd(C, R))
        b, A2, D, st, y = rnd(C, dtype=F32), -torch.rand(C, N, device="cuda"), rnd(C, dtype=F32), torch.zeros(C, N, device="cuda"), torch.empty(C, device="cuda")
        return lambda: X.scan_step(x, z, dbc, w, b, A2, D, st, y)
    t.kernel("decode scan step", sstep, C * (12 * N + 2 * R + 20))

    def rstep(i):
        st, y = torch.zeros(rh, rd, rv, device="cuda"), torch.empty(rh * rv, device="cuda")
        q, k, v, g = rnd(rh * rd, dtype=F32), rnd(rh * rd, dtype=F32), rnd(rh * rv, dtype=F32), rnd(rh * rv, dtype=F32)
        cs, dec = X.rotary_table(1e4, rd, 1024, "cuda"), torch.full((rh,), 0.99, device="cuda")
        return lambda: X.retention_step(q, k, v, g, cs, rd, rd ** -0.5, dec, 1e-5, st, y, pos=77)
    t.kernel("decode retention step", rstep, 8 * rh * rd * rv)

    for n in (1024, ctx):
        def adec(i):
            c, q, o = HM.KVCache(2 * G_, d, n, "cuda", BF, G_, dv), rnd(2 * H, d, dtype=F32), torch.empty(H * dv, device="cuda")
            c.k.normal_(), c.v.normal_()
            at = X.DiffDecodeAttention(H, G_, d, dv, "cuda")
            return lambda: at(q, c, d ** -0.5, 0.4, 0.5, 1e-5, o, n_pos=n)
        t.kernel(f"decode diff attention ctx {n}", adec, 2 * n * G_ * (2 * d + dv))

    def rn1(i):
        y, x, w, xs, dwa = rnd(1, W, dtype=F32), rnd(1, W, dtype=F32), rnd(W, dtype=F32), rnd(6, 1, W, dtype=F32), rnd(6, dtype=F32)
        return lambda: X.res_norm(y, x, w, 1e-5, x, None, (xs, dwa, True))
    t.kernel("decode residual norm + average of 6", rn1, W * 4 * 9)
    return t.rows


def qwen3_kernels(pkg, torch, pk, s, T=2048, ctx=8192):
    S, G, HM, F = pkg.sc_kernels, pkg.sc_decode, pkg.host_model, pkg.sc_format
    W, H, G_, ff, BF = s["width"], s["heads"], s["kv"], s["ff"], torch.bfloat16
    t = Timer(torch, pk)
    rnd = lambda *sh, dtype=BF: (torch.randn(*sh, device="cuda") * 0.5).to(dtype)          # noqa: E731

    def igemm(name, n, k, epi):
        def make(i):
            xq = torch.randint(-127, 128, (T, k), dtype=torch.int8, device="cuda")
            wq = torch.randint(-96, 97, (n, k), dtype=torch.int8, device="cuda")
            xs, ws = torch.full((T,), 1e-2, device="cuda"), torch.full((n,), 2.0 ** -9, device="cuda")
            res = rnd(T, n) if epi == 2 else None
            return lambda: S.mm_epi(xq, wq, xs, ws, epi, res=res)
        t.kernel(name, make, T * k + n * k + 2 * T * n, 2.0 * T * n * k, int8=True)
    qd = 128
    igemm("prefill gemm qkv", (H + 2 * G_) * qd, W, 1)
    igemm("prefill gemm o", W, H * qd, 2)
    igemm("prefill gemm gate|up", 2 * ff, W, 3)
    igemm("prefill gemm down", W, ff, 2)

    def sdpa(i):
        q, k, v = rnd(H, T, qd), rnd(G_, T, qd), rnd(G_, T, qd)
        return lambda: HM.sdpa(q, k, v, qd ** -0.5, True)
    t.kernel("prefill attention", sdpa, 2 * T * 2 * (H + G_) * qd, 2.0 * T * T * H * qd)

    def rmsq(i):
        x, w = rnd(T, W), rnd(W)
        return lambda: S.rmsnorm_quant(x, w, 1e-6, T)
    t.kernel("prefill rmsnorm quant", rmsq, 3 * T * W)

    def qgemv(name, n, k):
        c, b, ws, _, _ = F.quantize_device(torch.randn(n, k, device="cuda") * 0.02, want_qw=False)

        def make(i):
            cc, bb, w2, xq, xs = c.clone(), b.clone(), ws.clone(), torch.randint(-127, 128, (k,), dtype=torch.int8, device="cuda"), torch.ones(1, device="cuda")
            return lambda: G.gemv(xq, cc, bb, xs, w2, n, 1)
        t.kernel(name, make, n * k // 2 + n * k // 128 + 6 * n + k)
    qgemv("decode gemv qkv", (H + 2 * G_) * qd, W)
    qgemv("decode gemv o", W, H * qd)
    qgemv("decode gemv gate|up", 2 * ff, W)
    qgemv("decode gemv down", W, ff)
    if S.DecodeAttention.supports(H, G_, qd):
        for n in (1024, ctx):
            def qdec(i):
                c, q = HM.KVCache(G_, qd, n), rnd(H, qd)
                c.k.normal_(), c.v.normal_()
                at = S.DecodeAttention(H, G_, qd)
                return lambda: at(q, c, qd ** -0.5, n_pos=n)
            t.kernel(f"decode attention ctx {n}", qdec, 4 * n * G_ * qd)

    def rq1(i):
        x, w = rnd(1, W), rnd(W)
        return lambda: S.rmsnorm_quant(x, w, 1e-6, 1)
    t.kernel("decode rmsnorm quant", rq1, 5 * W)
    return t.rows


def measure_model(torch, pk, fused, dec, vocab, lengths=(512, 2048), n_tok=64):
    """Prompt tokens/s (graph replay, last position's logits included) and greedy tokens/s after a 512-token prompt."""
    t = Timer(torch, pk)
    ids = torch.randint(0, vocab, (1, max(lengths) + n_tok), device="cuda")
    cache, res = fused.make_cache(max(lengths) + n_tok + 8), {}

    def prefill(n):
        for c in cache:
            c.offset = 0
        return fused.logits(fused.hidden(ids[:, :n], cache)[:, -1:])
    for n in lengths:
        ms = t.replay_ms(t.graph([lambda: prefill(n)]))
        res[f"prefill_{n}_tok_s"] = round(n / ms * 1e3)
        res[f"prefill_{n}_ms"] = round(ms, 3)
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    with torch.no_grad():
        for _ in range(3):                                  # the first pass captures the step
            prefill(512)
            e0.record()
            dec.generate(ids[:, 512:513], cache, n_tok)
            e1.record()
            torch.cuda.synchronize()
    res["decode_tok_s"] = round(n_tok / e0.elapsed_time(e1) * 1e3, 1)
    return res


def measure_hybrid(pkg, torch, pk, cfg, **init):
    """A hybrid decoder of a configuration, random weights."""
    model = pkg.host_model.HybridLM(pkg.host_model.HybridArgs.from_config(cfg)).init_random(0, **init)
    fused = pkg.fused_hybrid.FusedHybrid(model)
    out = measure_model(torch, pk, fused, pkg.decode.DecodeHybrid(fused), cfg["vocab"])
    out["weight_gb"] = round(sum(w.numel() * 2 for w in model.w.values()) / 1e9, 3)
    del model, fused
    torch.cuda.empty_cache()
    return out


def bench_model(pkg, torch, pk, s):
    """Whole models of LAYERS layers."""
    HM, FQ, DEC = pkg.host_model, pkg.fused_qwen3, pkg.decode
    out = {"hybrid": measure_hybrid(pkg, torch, pk, hybrid_config(s))}
    a = HM.ModelArgs(s["width"], s["ff"], LAYERS, s["heads"], s["kv"], 128, 1e-6, 1e6, s["vocab"], False)
    with torch.device("cuda"):
        model = HM.CausalLM(a)
    model.init_random(0)
    fused = FQ.FusedQwen3(model, FQ.pack_model(model, on_device=True))
    out["qwen3_style"] = measure_model(torch, pk, fused, DEC.DecodeQwen3(fused), s["vocab"])
    out["qwen3_style"]["weight_gb"] = round(fused.weight_bytes() / 1e9, 3)
    del model, fused
    torch.cuda.empty_cache()
    return out


def run(pkg, torch, pk, sampler, sizes=None):
    torch.manual_seed(0)
    torch.cuda.set_device(0)
    out = {"workload": "hybrid", "layers": LAYERS, "data": "synthetic weights and token ids", "peaks": pk,
           "timing": "CUDA graph over copies of each call on different buffers, larger than L2 together", "sizes": {}}
    with sampler as clk:
        for name in sizes or SIZES:
            s = SIZES[name]
            out["sizes"][name] = {"config": s, "models": bench_model(pkg, torch, pk, s), "kernels": bench_kernels(pkg, torch, pk, s)}
    out["clocks"] = clk.summary()
    pkg._lib.check_status()
    print(json.dumps(out))
