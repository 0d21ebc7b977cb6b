"""Prefill of hybrid decoders (host_model.HybridLM): every layer names its mixer - selective scan, retention or differential
attention - and may have a feed-forward.  Per sublayer x <- x + norm(sublayer(x)), and after every layer x becomes a weighted
sum of the embedding output and all layers' results:

    mamba1      xz = W_in h; xc = silu(conv(x)); dbc = W_x xc; step = W_dt dbc; y = scan(xc, step, B, C) silu(z); W_o y
    retention   q|k|v|g = W h (one GEMM); o = retention(rotated q, k, v); W_o (o / rms(o) silu(g))
    attention   q|k|v = W h (one GEMM); q, k normalized, k and v appended to the cache; differential attention; W_o
    feed-forward W_down xielu(W_up h), the activation in the GEMM's epilogue

The residual stream, norms, scores and states are float32; matrix products and their activations are in the weights' type.
A portion continues from the cache, so a prompt may be cut anywhere; long prompts are cut into `portion` tokens here, which
bounds the store of the layers' results."""
import torch

from . import host_model as HM
from . import sc_mixers as X


class HybridLayer:
    """A layer's weights prepared for the kernels: projections of the same input concatenated, small vectors float32."""

    def __init__(self, args, w, p, dev):
        m, f32 = args.mixer, lambda n: w[p + n].float().contiguous()
        self.type = args.type
        mix = lambda *n: X.Linear(torch.cat([w[f"{p}mix.{k}"] for k in n]))           # noqa: E731
        if self.type == "mamba1":
            self.C, self.N, self.R = m["inner"], m["state"], m["dt_rank"]
            self.w_in, self.w_x, self.w_dt = mix("in"), mix("x"), mix("dt")
            self.conv_w, self.conv_b, self.dt_b, self.D = f32("mix.conv"), f32("mix.conv.b"), f32("mix.dt.b"), f32("mix.D")
            self.A2 = (-torch.exp(w[p + "mix.A_log"].double()) * X.LOG2E).float().contiguous()
        elif self.type == "retention":
            self.H, self.d, self.dv = m["heads"], m["dim"], m["vdim"]
            rot = m.get("rot") or {"base": 1.0, "dims": 0}
            self.rot, self.dims, self.kscale = (float(rot["base"]), int(rot["dims"])), int(rot["dims"]), self.d ** -0.5
            self.w_in = mix("q", "k", "v", "g")
            self.sizes = [self.H * self.d] * 2 + [self.H * self.dv] * 2
            self.decay = torch.tensor(m["decay"], dtype=torch.float32, device=dev)
            self.form = 0 if min(m["decay"]) > 0 else 1          # the chunked form works with logarithms of the decays
        else:
            self.H, self.G, self.d, self.dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            self.scale, self.diff = float(m["scale"]), float(m["diff"])
            self.w_in = mix("q", "k", "v")
            self.sizes = [2 * self.H * self.d, 2 * self.G * self.d, self.G * self.dv]
            self.q_norm, self.k_norm = f32("mix.q.norm"), f32("mix.k.norm")
            l1, l2 = ((w[f"{p}mix.lq{j}"].double() * w[f"{p}mix.lk{j}"].double()).sum().exp().item() for j in (1, 2))
            self.lam = l1 - l2 + self.diff
        self.w_o = mix("o")
        self.norm1, self.dwa = f32("norm1"), f32("dwa")
        self.w_up = self.w_down = None
        if args.mlp is not None:
            self.norm2 = f32("norm2")
            self.w_up, self.w_down, self.act = X.Linear(w[p + "mlp.up"]), X.Linear(w[p + "mlp.down"]), X.XIELU(w[p + "mlp.act"])


class FusedHybrid:
    def __init__(self, model, portion=4096):
        """model: host_model.HybridLM with weights."""
        self.model, self.args, self.eps, self.portion = model, model.args, model.args.rms_norm_eps, portion
        w = model.w
        self.embed, self.head, self.final_norm = w["embed"], X.Linear(w["head"]), w["final.norm"].float().contiguous()
        self.layers = [HybridLayer(e, w, f"l{i}.", model.device) for i, e in enumerate(model.args.layers)]
        self._tables, self._retired = {}, []
        self.trace = None            # a list: receives the residual stream after every layer of the next portions
        self.ensure_positions(1)

    # ---- rotary tables -------------------------------------------------------------------------------------------------
    def ensure_positions(self, n):
        """Tables of at least n positions.  A table that a captured graph may have read is kept when a longer one replaces it."""
        for key in {ly.rot for ly in self.layers if ly.type == "retention"}:
            old = self._tables.get(key)
            if old is None or old.shape[0] < n:
                if old is not None:
                    self._retired.append(old)
                rows = 1 << max(10, (n - 1).bit_length())
                self._tables[key] = X.rotary_table(key[0], key[1], rows, self.model.device)

    def table(self, ly):
        return self._tables[ly.rot]

    # ---- mixers --------------------------------------------------------------------------------------------------------
    def _mamba1(self, ly, h, c):
        xz = ly.w_in(h)
        z = xz[:, ly.C:]
        xc = X.conv_silu(xz[:, :ly.C], ly.conv_w, ly.conv_b, c.tail)
        dbc = ly.w_x(xc)
        step = ly.w_dt(dbc[:, :ly.R], torch.float32)
        return X.selective_scan(xc, step, dbc[:, ly.R:], z, ly.dt_b, ly.A2, ly.D, c.ssm)

    def _retention(self, ly, h, c):
        q, k, v, g = ly.w_in(h).split(ly.sizes, 1)
        o = X.retention(q, k, v, self.table(ly)[c.offset:], ly.dims, ly.kscale, ly.decay, c.kv, ly.form)
        return X.head_norm_gate(o, g, self.eps)

    def _attention(self, ly, h, c):
        q, k, v = ly.w_in(h).split(ly.sizes, 1)
        q = X.qk_norm_append(q, k, v, ly.H, ly.G, ly.q_norm, ly.k_norm, self.eps, c, h.dtype)
        return X.diff_attention(q, c, ly.H, ly.G, ly.scale, ly.lam, ly.diff, self.eps)

    # ---- one portion ---------------------------------------------------------------------------------------------------
    def _portion(self, ids, cache):
        """ids int64 [T] -> residual stream [T, W] float32 after the last layer; the cache advances by T positions."""
        T, W, dev, dt = ids.numel(), self.args.hidden_size, self.model.device, self.model.dtype
        assert cache[0].offset + T <= cache[0].capacity, "KV cache capacity exceeded"
        self.ensure_positions(cache[0].offset + T)
        nl = len(self.layers)
        xs = torch.empty((nl + 1, T, W), dtype=torch.float32, device=dev)
        x = torch.empty((T, W), dtype=torch.float32, device=dev)
        h = torch.empty((T, W), dtype=dt, device=dev)
        X.embed(ids, self.embed, xs[0], h)
        cur = xs[0]
        for i, (ly, c) in enumerate(zip(self.layers, cache)):
            y = ly.w_o(getattr(self, "_" + ly.type)(ly, h, c), torch.float32)
            norm = ly.norm1
            if ly.w_up is not None:
                X.res_norm(y, cur, norm, self.eps, x, h)
                cur, norm = x, ly.norm2
                y = ly.w_down(ly.w_up(h, act=ly.act), torch.float32)
            X.res_norm(y, cur, norm, self.eps, x, h if i + 1 < nl else None, (xs, ly.dwa, i + 1 < nl))
            cur = x
            if self.trace is not None:
                self.trace.append(x.clone())
            c.offset += T
        return x

    @torch.no_grad()
    def hidden(self, ids, cache):
        """Final normed hidden states [1, L, W] for ids [1, L] (prefill into a fresh or offset cache)."""
        parts = [X.norm_rows(self._portion(t, cache), self.final_norm, self.eps, self.model.dtype)
                 for t in ids.reshape(-1).contiguous().split(self.portion)]
        return (parts[0] if len(parts) == 1 else torch.cat(parts))[None]

    def make_cache(self, capacity=4096):
        return HM.make_prompt_cache(self.model, capacity)

    def logits(self, h):
        """h [1, L, W] -> float32 [1, L, V]."""
        return self.head(h[0], torch.float32)[None]

    def __call__(self, ids, cache=None):
        """Logits for every position."""
        cache = cache if cache is not None else self.make_cache(max(ids.shape[1], 1))
        return self.logits(self.hidden(ids, cache))
