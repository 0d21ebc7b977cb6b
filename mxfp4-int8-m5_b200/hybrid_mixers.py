"""Sequence mixers of the hybrid decoders, one class per type of host_model.MIXERS: a layer's weights prepared for the kernels
(projections of the same input concatenated, small vectors float32) and the mixer's two paths,

    prefill(f, h, c)          a portion h [T, W] -> the input of the output projection [T, K]; cache c is read from c.offset on
    step(f, x, c, b, pos)     one float32 row in the buffers b = buffers(dev); `pos` (int32 on the device) replaces c.offset

The caller applies w_o and advances the cache.  `f` is the fused_hybrid.FusedHybrid, which holds the rotation tables.

    mamba1            xz = W_in h; xc = silu(conv(x)); dbc = W_x xc; step = W_dt dbc; y = scan(xc, step, B, C) silu(z)
    retention         q|k|v|g = W h (one GEMM); o = retention(rotated q, k, v); o / rms(o) silu(g)
    attention         q|k|v = W h; q, k normalized, k and v appended to the cache; differential attention
    delta             q|k|v|g|b|a = W h; q|k|v through convolution + SiLU; gated delta rule; o / rms(o) w silu(g)
    channel_delta     q|k|v|a1|g1|b = W h; decays W_a2 a1 per key channel; gate sigmoid(W_g2 g1); otherwise as delta
    latent_attention  query latent|latent|key part = W h; norms, rotation, cache; queries W_uq; attention over the window"""
import torch

from . import sc_mixers as X


class Mixer:
    rot = None               # (base, dims) of the rotation table it needs

    def __init__(self, m, w, p, dev, eps):
        self.eps = eps
        self.f32 = lambda n: w[p + n].float().contiguous()
        self.lin = lambda *n: X.Linear(torch.cat([w[p + k] for k in n]))
        self.setup(m, w, p, dev)
        self.w_o = self.lin("o")
        del self.f32, self.lin

    def buffers(self, dev):
        """Float32 vectors of one step, written before they are read."""
        return {"in": torch.empty(self.w_in.N, dtype=torch.float32, device=dev), "o": torch.empty(self.w_o.K, dtype=torch.float32, device=dev)}


class Mamba1(Mixer):
    def setup(self, m, w, p, dev):
        self.C, self.N, self.R = m["inner"], m["state"], m["dt_rank"]
        self.w_in, self.w_x, self.w_dt = self.lin("in"), self.lin("x"), self.lin("dt")
        self.conv_w, self.conv_b, self.dt_b, self.D = self.f32("conv"), self.f32("conv.b"), self.f32("dt.b"), self.f32("D")
        self.A2 = (-torch.exp(w[p + "A_log"].double()) * X.LOG2E).float().contiguous()

    def prefill(self, f, h, c):
        xz = self.w_in(h)
        z = xz[:, self.C:]
        xc = X.conv_silu(xz[:, :self.C], self.conv_w, self.conv_b, c.tail)
        dbc = self.w_x(xc)
        step = self.w_dt(dbc[:, :self.R], torch.float32)
        return X.selective_scan(xc, step, dbc[:, self.R:], z, self.dt_b, self.A2, self.D, c.ssm)

    def buffers(self, dev):
        return {**super().buffers(dev), "dbc": torch.empty(self.w_x.N, dtype=torch.float32, device=dev)}

    def step(self, f, x, c, b, pos):
        xz = self.w_in.vec(x, conv=(self.conv_w, self.conv_b, c.tail), out=b["in"])
        dbc = self.w_x.vec(xz[:self.C], out=b["dbc"])
        return X.scan_step(xz, xz[self.C:], dbc, self.w_dt, self.dt_b, self.A2, self.D, c.ssm, b["o"])


class Retention(Mixer):
    def setup(self, m, w, p, dev):
        self.H, self.d, self.dv = m["heads"], m["dim"], m["vdim"]
        rot = m.get("rot") or {"base": 1.0, "dims": 0}
        self.rot, self.dims, self.kscale = (float(rot["base"]), int(rot["dims"])), int(rot["dims"]), self.d ** -0.5
        self.w_in = self.lin("q", "k", "v", "g")
        self.sizes = [self.H * self.d] * 2 + [self.H * self.dv] * 2
        self.decay = torch.tensor(m["decay"], dtype=torch.float32, device=dev)
        self.form = 0 if min(m["decay"]) > 0 else 1          # the chunked form works with logarithms of the decays

    def prefill(self, f, h, c):
        q, k, v, g = self.w_in(h).split(self.sizes, 1)
        o = X.retention(q, k, v, f.table(self.rot)[c.offset:], self.dims, self.kscale, self.decay, c.kv, self.form)
        return X.head_norm_gate(o, g, self.eps)

    def step(self, f, x, c, b, pos):
        q, k, v, g = self.w_in.vec(x, out=b["in"]).split(self.sizes)
        return X.retention_step(q, k, v, g, f.table(self.rot), self.dims, self.kscale, self.decay, self.eps, c.kv, b["o"], c.offset, pos)


class DiffAttention(Mixer):
    def setup(self, m, w, p, dev):
        self.H, self.G, self.d, self.dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        self.scale, self.diff = float(m["scale"]), float(m["diff"])
        self.w_in = self.lin("q", "k", "v")
        self.sizes = [2 * self.H * self.d, 2 * self.G * self.d, self.G * self.dv]
        self.q_norm, self.k_norm = self.f32("q.norm"), self.f32("k.norm")
        l1, l2 = ((w[f"{p}lq{j}"].double() * w[f"{p}lk{j}"].double()).sum().exp().item() for j in (1, 2))
        self.lam = l1 - l2 + self.diff

    def prefill(self, f, h, c):
        q, k, v = self.w_in(h).split(self.sizes, 1)
        q = X.qk_norm_append(q, k, v, self.H, self.G, self.q_norm, self.k_norm, self.eps, c, h.dtype)
        return X.diff_attention(q, c, self.H, self.G, self.scale, self.lam, self.diff, self.eps)

    def buffers(self, dev):
        return {**super().buffers(dev), "attn": X.DiffDecodeAttention(self.H, self.G, self.d, self.dv, dev)}

    def step(self, f, x, c, b, pos):
        q, k, v = self.w_in.vec(x, out=b["in"])[None].split(self.sizes, 1)
        q = X.qk_norm_append(q, k, v, self.H, self.G, self.q_norm, self.k_norm, self.eps, c, torch.float32, pos)
        return b["attn"](q, c, self.scale, self.lam, self.diff, self.eps, b["o"], n_pos=c.offset + 1, pos_dev=pos)


class Delta(Mixer):
    channel = False

    def setup(self, m, w, p, dev):
        self.H, self.G, self.d, self.dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        self.qkv = [self.G * self.d] * 2 + [self.H * self.dv]
        self.C = sum(self.qkv)
        self.conv_w = torch.cat([self.f32(n + ".conv") for n in "qkv"]).contiguous()
        self.nA = (-torch.exp(w[p + "A_log"].double())).float().contiguous()
        self.dt_b, self.norm = self.f32("dt_bias"), self.f32("norm")
        self.w_a = self.w_g = None
        if self.channel:
            self.w_in, self.w_a, self.w_g = self.lin("q", "k", "v", "a1", "g1", "b"), self.lin("a2"), self.lin("g2")
            self.sizes = [self.C, self.w_a.K, self.w_g.K, self.H]
        else:
            self.w_in = self.lin("q", "k", "v", "g", "a", "b")
            self.sizes = [self.C, self.H * self.dv, self.H, self.H]

    def prefill(self, f, h, c):
        x, *rest = self.w_in(h).split(self.sizes, 1)
        q, k, v = X.conv_silu(x, self.conv_w, None, c.tail).split(self.qkv, 1)
        if self.channel:
            a, g, b = rest
            a, g = self.w_a(a, torch.float32), self.w_g(g)
        else:
            g, a, b = rest
        o = X.delta(q, k, v, b, a, self.channel, self.nA, self.dt_b, c.kv)
        return X.head_norm_gate(o, g, self.eps, self.norm, int(self.channel))

    def step(self, f, x, c, b, pos):
        x, *rest = self.w_in.vec(x, conv=(self.conv_w, None, c.tail), out=b["in"]).split(self.sizes)
        q, k, v = x.split(self.qkv)
        a, g, beta = rest if self.channel else (rest[1], rest[0], rest[2])
        return X.delta_step(q, k, v, beta, a, g, self.w_a, self.w_g, self.nA, self.dt_b, self.norm, self.eps, c.kv, b["o"])


class ChannelDelta(Delta):
    channel = True


class LatentAttention(Mixer):
    def setup(self, m, w, p, dev):
        self.H, self.d, self.r, self.dv, self.R, self.Q = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
        self.rot = (float(m["rot"]["base"]), self.r) if self.r else (1.0, 0)
        self.scale, self.window = float(m["scale"]), int((m.get("mask") or {}).get("size") or 0)
        self.w_in, self.w_uq, self.w_ukv = self.lin("dq", "dkv"), self.lin("uq"), self.lin("uk", "uv")
        self.w_uk, self.w_uv = self.w_ukv.rows(0, self.H * self.d), self.w_ukv.rows(self.H * self.d, self.H * (self.d + self.dv))
        self.q_norm, self.kv_norm = self.f32("dq.norm"), self.f32("dkv.norm")

    def _queries(self, f, y, c, dtype, pos):
        cs = f.table(self.rot)
        return X.latent_append(y, self.Q, self.R, self.r, self.q_norm, self.kv_norm, cs, self.eps, c, dtype, pos), cs

    def _rows(self, q, cs, c, dtype, pos=None):
        return X.latent_rows(q, self.w_uk, self.w_uv, cs, c, self.H, self.d, self.r, self.dv, self.window, self.scale, dtype, pos)

    def prefill(self, f, h, c):
        cq, cs = self._queries(f, self.w_in(h), c, h.dtype, None)
        q = self.w_uq(cq)
        if h.shape[0] < X.LATENT_TC_MIN or not X.latent_prompt_supported(q, self.d, self.r, self.dv, self.scale):
            return self._rows(q, cs, c, h.dtype)
        return X.latent_prompt(q, self.w_ukv, cs, c, self.H, self.d, self.r, self.dv, self.R, self.window, self.scale)

    def buffers(self, dev):
        return {**super().buffers(dev), "q": torch.empty(self.w_uq.N, dtype=torch.float32, device=dev)}

    def step(self, f, x, c, b, pos):
        cq, cs = self._queries(f, self.w_in.vec(x, out=b["in"])[None], c, torch.float32, pos)
        return self._rows(self.w_uq.vec(cq[0], out=b["q"])[None], cs, c, torch.float32, pos)[0]


CLASSES = {"mamba1": Mamba1, "retention": Retention, "attention": DiffAttention, "delta": Delta, "channel_delta": ChannelDelta,
           "latent_attention": LatentAttention}
