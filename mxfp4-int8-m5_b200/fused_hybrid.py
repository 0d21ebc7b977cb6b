"""Prefill of hybrid decoders (host_model.HybridLM): every layer names its mixer (hybrid_mixers.py) and may have a feed-forward.

Around the mixers (host_model.Design) either, per sublayer, x <- x + norm(sublayer(x)), and after every layer x becomes a weighted
sum of the embedding output and all layers' results; or x <- x + m sublayer(norm(x)), where the sum and the next sublayer's norm
are one kernel.  The feed-forward is W_down act(..), the activation in the first GEMM's epilogue.

The residual stream, norms, scores and states are float32; matrix products and their activations are in the weights' type.
A portion continues from the cache, so a prompt may be cut anywhere; long prompts are cut into `portion` tokens here, which
bounds the store of the layers' results."""
import torch

from . import host_model as HM
from . import hybrid_mixers as MX
from . import sc_mixers as X


class HybridLayer:
    """A layer's mixer, norms and feed-forward weights prepared for the kernels."""

    def __init__(self, args, design, w, p, dev, eps):
        f32 = lambda n: w[p + n].float().contiguous()       # noqa: E731
        self.mixer = MX.CLASSES[args.type](args.mixer, w, p + "mix.", dev, eps)
        self.norm1 = f32("norm1")
        self.dwa = None if design.prenorm else f32("dwa")
        self.w_up = self.w_down = None
        if args.mlp is not None:
            self.norm2, self.w_down = f32("norm2"), X.Linear(w[p + "mlp.down"])
            if design.act == "xielu":
                self.w_up, self.act = X.Linear(w[p + "mlp.up"]), X.XIELU(w[p + "mlp.act"])
            else:
                self.w_up, self.act = X.Linear(X.GatedGELU.weight(w[p + "mlp.gate"], w[p + "mlp.up"])), X.GatedGELU()

    def feed_forward(self, h):
        return self.w_down(self.w_up(h, act=self.act)[:, :self.w_down.K], torch.float32)

    def feed_forward_vec(self, x, u, y):
        return self.w_down.vec(self.w_up.vec(x, act=self.act, out=u)[:self.w_down.K], out=y)


class FusedHybrid:
    def __init__(self, model, portion=4096):
        """model: host_model.HybridLM with weights."""
        self.model, self.args, self.eps, self.portion = model, model.args, model.args.rms_norm_eps, portion
        w, a, dev = model.w, model.args, model.device
        self.embed_table, self.final_norm = w["embed"], w["final.norm"].float().contiguous()
        self.head = X.Linear(w["embed"] if a.design.tied else w["head"])
        own = {i: HybridLayer(e, a.design, w, f"l{i}.", dev, self.eps) for i, e in enumerate(a.layers) if e.weights_of is None}
        self.layers = [own[a.source(i)] for i in range(len(a.layers))]
        self._tables, self._retired = {}, []
        self.trace = None            # a list: receives the residual stream after every layer of the next portions
        self.ensure_positions(1)

    # ---- rotary tables -------------------------------------------------------------------------------------------------
    def ensure_positions(self, n):
        """Tables of at least n positions.  A table that a captured graph may have read is kept when a longer one replaces it."""
        for key in {ly.mixer.rot for ly in self.layers if ly.mixer.rot is not None}:
            old = self._tables.get(key)
            if old is None or old.shape[0] < n:
                if old is not None:
                    self._retired.append(old)
                rows = 1 << max(10, (n - 1).bit_length())
                self._tables[key] = X.rotary_table(key[0], key[1], rows, self.model.device)

    def table(self, rot):
        return self._tables[rot]

    # ---- one portion ---------------------------------------------------------------------------------------------------
    def embed(self, ids, cache, x, h=None):
        """x float32 <- embedding of ids [T]; h: the same in the weights' type where the first mixer reads it unnormalized."""
        a = self.args
        if a.design.prenorm:
            b = a.bigram
            X.embed_pair(ids, self.embed_table, x, a.embed_scale, *((self.model.w["bigram"], (b["buckets"], b["mul_prev"], b["mul_cur"]), cache[-1].prev) if b else ()))
        else:
            X.embed(ids, self.embed_table, x, h)

    def _portion(self, ids, cache):
        """ids int64 [T] -> final normed hidden states [T, W]; the cache advances by T positions."""
        T, W, dev, dt = ids.numel(), self.args.hidden_size, self.model.device, self.model.dtype
        assert cache[0].offset + T <= cache[0].capacity, "KV cache capacity exceeded"
        self.ensure_positions(cache[0].offset + T)
        out = (self._prenorm if self.args.design.prenorm else self._postnorm)(ids, cache, T, W, dev, dt)
        for c in cache:
            c.offset += T
        return out

    def _prenorm(self, ids, cache, T, W, dev, dt):
        x = torch.empty((T, W), dtype=torch.float32, device=dev)
        h = torch.empty((T, W), dtype=dt, device=dev)
        mult, nl = self.args.residual_mult, len(self.layers)
        self.embed(ids, cache, x)
        X.add_norm(None, x, self.layers[0].norm1 if nl else self.final_norm, mult, self.eps, h)
        for i, (ly, c) in enumerate(zip(self.layers, cache)):
            after = self.layers[i + 1].norm1 if i + 1 < nl else self.final_norm
            y = ly.mixer.w_o(ly.mixer.prefill(self, h, c), torch.float32)
            X.add_norm(y, x, after if ly.w_up is None else ly.norm2, mult, self.eps, h)
            if ly.w_up is not None:
                X.add_norm(ly.feed_forward(h), x, after, mult, self.eps, h)
            if self.trace is not None:
                self.trace.append(x.clone())
        return h

    def _postnorm(self, ids, cache, T, W, dev, dt):
        nl = len(self.layers)
        xs = torch.empty((nl + 1, T, W), dtype=torch.float32, device=dev)
        x = torch.empty((T, W), dtype=torch.float32, device=dev)
        h = torch.empty((T, W), dtype=dt, device=dev)
        self.embed(ids, cache, xs[0], h)
        cur = xs[0]
        for i, (ly, c) in enumerate(zip(self.layers, cache)):
            y = ly.mixer.w_o(ly.mixer.prefill(self, h, c), torch.float32)
            norm = ly.norm1
            if ly.w_up is not None:
                X.res_norm(y, cur, norm, self.eps, x, h)
                cur, norm = x, ly.norm2
                y = ly.feed_forward(h)
            X.res_norm(y, cur, norm, self.eps, x, h if i + 1 < nl else None, (xs, ly.dwa, i + 1 < nl))
            cur = x
            if self.trace is not None:
                self.trace.append(x.clone())
        return X.norm_rows(x, self.final_norm, self.eps, dt)

    @torch.no_grad()
    def hidden(self, ids, cache):
        """Final normed hidden states [1, L, W] for ids [1, L] (prefill into a fresh or offset cache)."""
        parts = [self._portion(t, cache) for t in ids.reshape(-1).contiguous().split(self.portion)]
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
