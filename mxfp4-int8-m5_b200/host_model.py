"""Torch containers for the decoder checkpoints the fused W4A8 paths wrap, with the attribute layout of the mlx_lm models
the reference wires into (model.model.layers[i].self_attn.q_proj, .mlp.gate_proj / .mlp.switch_mlp, ...; see
e2e/fused_qwen3.py:82-118 and e2e/fused_olmoe.py:132-176), plus what surrounds the W4A8 linears in a block: RMSNorm in
MLX's rounding order, half-split rotary embedding, a preallocated KV cache and scaled-dot-product attention (torch's).

`CausalLM.forward` is the unfused path: every linear is whatever module sits in the tree (a bf16 torch Linear, or a
W4A8Linear after apply_w4a8), as in e2e/w4a8_mlx.py:197-207.
"""
from dataclasses import dataclass

import torch
import torch.nn.functional as TF

from . import sc_kernels as S


@dataclass
class ModelArgs:
    hidden_size: int
    intermediate_size: int
    num_hidden_layers: int
    num_attention_heads: int
    num_key_value_heads: int
    head_dim: int
    rms_norm_eps: float = 1e-6
    rope_theta: float = 1e6
    vocab_size: int = 32000
    tie_word_embeddings: bool = True
    num_experts: int = 0
    num_experts_per_tok: int = 0
    norm_topk_prob: bool = False
    model_type: str = "qwen3"


QWEN3_1_7B = ModelArgs(2048, 6144, 28, 16, 8, 128, 1e-6, 1e6, 151936, True)
OLMOE_1B_7B = ModelArgs(2048, 1024, 16, 16, 16, 128, 1e-5, 1e4, 50304, False, 64, 8, False, "olmoe")

LINEARS = ["self_attn.q_proj", "self_attn.k_proj", "self_attn.v_proj", "self_attn.o_proj",
           "mlp.gate_proj", "mlp.up_proj", "mlp.down_proj"]


class RMSNorm(torch.nn.Module):
    """w * T(x * rsqrt(mean(x^2) + eps)): the product x * inv is rounded to the activation type before the weight
    multiplies it, the order of MLX's rms_norm that the fused row kernels replicate."""

    def __init__(self, dims, eps):
        super().__init__()
        self.weight = torch.nn.Parameter(torch.ones(dims, dtype=torch.bfloat16), requires_grad=False)
        self.eps = eps

    def forward(self, x):
        xf = x.float()
        inv = torch.rsqrt(xf.double().pow(2).mean(-1, keepdim=True).float() + self.eps)
        return self.weight * (xf * inv).to(x.dtype)


def rope(x, inv_freq, offset=0):
    """Half-split rotary embedding of x [..., L, d] at positions offset.. (mlx.nn.RoPE(traditional=False))."""
    L, d = x.shape[-2], x.shape[-1]
    ang = torch.arange(offset, offset + L, device=x.device, dtype=torch.float32)[:, None] * inv_freq[None, :]
    c, s = torch.cos(ang.double()).float(), torch.sin(ang.double()).float()
    x1, x2 = x[..., :d // 2].float(), x[..., d // 2:].float()
    return torch.cat([x1 * c - x2 * s, x1 * s + x2 * c], -1).to(x.dtype)


class KVCache:
    """Keys and values of one layer in preallocated [heads, capacity, d] tensors; `offset` positions are filled.  Values may have
    their own head count and size."""

    def __init__(self, heads, d, capacity, device="cuda", dtype=torch.bfloat16, v_heads=None, v_d=None):
        self.k = torch.empty((heads, capacity, d), dtype=dtype, device=device)
        self.v = torch.empty((v_heads or heads, capacity, v_d or d), dtype=dtype, device=device)
        self.offset, self.capacity = 0, capacity

    def reset(self):
        """Forget the sequence; rows past `offset` are never read."""
        self.offset = 0

    def carried(self):
        """Tensors that a step changes in place and whose old content it reads (none: a row is only overwritten)."""
        return []

    def update_and_fetch(self, k, v):
        L = k.shape[-2]
        assert self.offset + L <= self.k.shape[1], "KV cache capacity exceeded"
        self.k[:, self.offset:self.offset + L] = k.reshape(self.k.shape[0], L, -1)
        self.v[:, self.offset:self.offset + L] = v.reshape(self.k.shape[0], L, -1)
        self.offset += L
        return self.k[:, :self.offset], self.v[:, :self.offset]


class StateCache:
    """Recurrent state of one layer: float32 tensors of fixed size that every token updates in place, zero at the start of a
    sequence.  `offset` and `capacity` count positions as in KVCache, so that both kinds sit in one list."""

    def __init__(self, shapes, capacity, device="cuda"):
        self.state = {n: torch.zeros(s, dtype=torch.float32, device=device) for n, s in shapes.items()}
        self.offset, self.capacity = 0, capacity

    def __getattr__(self, name):
        try:
            return self.__dict__["state"][name]
        except KeyError:
            raise AttributeError(name) from None

    def reset(self):
        self.offset = 0
        for t in self.state.values():
            t.zero_()

    def carried(self):
        return list(self.state.values())


class LatentCache:
    """Latents of one layer's attention: rows of [latent, rotated key part], each part zero padded to a multiple of 8 values."""

    def __init__(self, latent, rot, capacity, device="cuda", dtype=torch.bfloat16):
        up8 = lambda n: (n + 7) // 8 * 8      # noqa: E731
        self.c = torch.zeros((capacity, up8(latent) + up8(rot)), dtype=dtype, device=device)
        self.offset, self.capacity = 0, capacity

    def reset(self):
        """Forget the sequence; rows past `offset` are never read."""
        self.offset = 0

    def carried(self):
        return []


class TokenCache:
    """The token before the next one, where the embedding depends on it; negative at the start of a sequence."""

    def __init__(self, capacity, device="cuda"):
        self.prev = torch.full((1,), -1, dtype=torch.long, device=device)
        self.offset, self.capacity = 0, capacity

    def reset(self):
        self.offset = 0
        self.prev.fill_(-1)

    def carried(self):
        return [self.prev]


def sdpa(q, k, v, scale, causal):
    """q [hq, L, d], k / v [hk, T, d] (T >= L: the last L keys are the queries' own positions) -> [L, hq * d]."""
    hq, L, d = q.shape
    hk, T = k.shape[0], k.shape[1]
    mask = None
    is_causal = bool(causal and L > 1 and T == L)
    if causal and L > 1 and T != L:
        mask = torch.ones(L, T, dtype=torch.bool, device=q.device).tril(T - L)
    o = TF.scaled_dot_product_attention(q[None], k[None], v[None], attn_mask=mask, is_causal=is_causal, scale=scale,
                                        enable_gqa=hq != hk)
    return o[0].transpose(0, 1).reshape(L, hq * d)


def sdpa_f64(q, k, v, scale, causal):
    """The same attention in float64 with a single rounding at the output: a slow, kernel-independent form for checks."""
    hq, L, d = q.shape
    hk, T = k.shape[0], k.shape[1]
    kk, vv = (t.double().repeat_interleave(hq // hk, 0) for t in (k, v))
    s = torch.einsum("hld,htd->hlt", q.double(), kk) * scale
    if causal:
        s.masked_fill_(~torch.ones(L, T, dtype=torch.bool, device=q.device).tril(T - L), float("-inf"))
    o = torch.einsum("hlt,htd->hld", torch.softmax(s, -1), vv)
    return o.transpose(0, 1).reshape(L, hq * d).to(q.dtype)


def _linear(i, o):
    lin = torch.nn.Linear(i, o, bias=False, dtype=torch.bfloat16)
    lin.weight.requires_grad_(False)
    return lin


class Attention(torch.nn.Module):
    def __init__(self, a):
        super().__init__()
        D, hq, hk, d = a.hidden_size, a.num_attention_heads, a.num_key_value_heads, a.head_dim
        self.hq, self.hk, self.d, self.scale = hq, hk, d, d ** -0.5
        self.full_norm = a.model_type == "olmoe"
        self.q_proj, self.k_proj, self.v_proj, self.o_proj = _linear(D, hq * d), _linear(D, hk * d), _linear(D, hk * d), _linear(hq * d, D)
        self.q_norm = RMSNorm(hq * d if self.full_norm else d, a.rms_norm_eps)
        self.k_norm = RMSNorm(hk * d if self.full_norm else d, a.rms_norm_eps)
        self.register_buffer("inv_freq", S.rope_inv_freq(d, a.rope_theta, None), persistent=False)

    def forward(self, x, cache):
        L = x.shape[0]
        q, k, v = self.q_proj(x), self.k_proj(x), self.v_proj(x)
        if self.full_norm:
            q, k = self.q_norm(q), self.k_norm(k)
        q = q.reshape(L, self.hq, self.d).transpose(0, 1)
        k = k.reshape(L, self.hk, self.d).transpose(0, 1)
        v = v.reshape(L, self.hk, self.d).transpose(0, 1)
        if not self.full_norm:
            q, k = self.q_norm(q), self.k_norm(k)
        q, k = rope(q, self.inv_freq, cache.offset), rope(k, self.inv_freq, cache.offset)
        k, v = cache.update_and_fetch(k, v)
        return self.o_proj(sdpa(q, k, v, self.scale, True))


class MLP(torch.nn.Module):
    def __init__(self, a):
        super().__init__()
        D, F = a.hidden_size, a.intermediate_size
        self.gate_proj, self.up_proj, self.down_proj = _linear(D, F), _linear(D, F), _linear(F, D)

    def forward(self, x):
        return self.down_proj(TF.silu(self.gate_proj(x)) * self.up_proj(x))


class _Stacked(torch.nn.Module):
    def __init__(self, E, o, i):
        super().__init__()
        self.weight = torch.nn.Parameter(torch.empty((E, o, i), dtype=torch.bfloat16), requires_grad=False)


class SwitchMLP(torch.nn.Module):
    """Expert weights stacked [E, out, in] per projection (mlx_lm's switch_mlp layout)."""

    def __init__(self, a):
        super().__init__()
        E, D, F = a.num_experts, a.hidden_size, a.intermediate_size
        self.gate_proj, self.up_proj, self.down_proj = _Stacked(E, F, D), _Stacked(E, F, D), _Stacked(E, D, F)


class MoeMLP(torch.nn.Module):
    def __init__(self, a):
        super().__init__()
        self.k, self.norm_topk = a.num_experts_per_tok, a.norm_topk_prob
        self.gate = _linear(a.hidden_size, a.num_experts)
        self.switch_mlp = SwitchMLP(a)

    def forward(self, x):
        rw = torch.softmax(self.gate(x).float(), dim=1).to(x.dtype)
        scores, inds = torch.topk(rw, self.k, dim=-1)
        if self.norm_topk:
            scores = scores / scores.sum(-1, keepdim=True)
        sw, out = self.switch_mlp, torch.zeros_like(x)
        for e in inds.unique().tolist():
            t, j = (inds == e).nonzero(as_tuple=True)
            xe = x[t]
            ye = (TF.silu(xe @ sw.gate_proj.weight[e].T) * (xe @ sw.up_proj.weight[e].T)) @ sw.down_proj.weight[e].T
            out.index_add_(0, t, ye * scores[t, j][:, None])
        return out


class Layer(torch.nn.Module):
    def __init__(self, a):
        super().__init__()
        self.self_attn = Attention(a)
        self.mlp = MoeMLP(a) if a.num_experts else MLP(a)
        self.input_layernorm = RMSNorm(a.hidden_size, a.rms_norm_eps)
        self.post_attention_layernorm = RMSNorm(a.hidden_size, a.rms_norm_eps)

    def forward(self, h, cache):
        h = h + self.self_attn(self.input_layernorm(h), cache)
        return h + self.mlp(self.post_attention_layernorm(h))


class Inner(torch.nn.Module):
    def __init__(self, a):
        super().__init__()
        self.embed_tokens = torch.nn.Embedding(a.vocab_size, a.hidden_size, dtype=torch.bfloat16)
        self.embed_tokens.weight.requires_grad_(False)
        self.layers = torch.nn.ModuleList(Layer(a) for _ in range(a.num_hidden_layers))
        self.norm = RMSNorm(a.hidden_size, a.rms_norm_eps)


class CausalLM(torch.nn.Module):
    """Qwen3-style dense or OLMoE-style mixture-of-experts decoder (args.num_experts > 0)."""

    def __init__(self, args):
        super().__init__()
        self.args = args
        self.model = Inner(args)
        self.lm_head = None if args.tie_word_embeddings else _linear(args.hidden_size, args.vocab_size)

    def head(self, h):
        return TF.linear(h, self.model.embed_tokens.weight) if self.lm_head is None else self.lm_head(h)

    def forward(self, ids, cache=None):
        """ids int [1, L] -> logits [1, L, V]; prefill into a fresh or offset cache."""
        cache = cache if cache is not None else make_prompt_cache(self, ids.shape[1])
        h = self.model.embed_tokens(ids)[0]
        for layer, c in zip(self.model.layers, cache):
            h = layer(h, c)
        return self.head(self.model.norm(h)[None])

    @torch.no_grad()
    def init_random(self, seed=0, scale=0.02):
        """Seeded synthetic weights of the architecture (no checkpoint is read), generated on the parameters' device."""
        dev = self.model.embed_tokens.weight.device
        g = torch.Generator(device=dev).manual_seed(seed)
        for name, p in self.named_parameters():
            r = torch.randn(p.shape, generator=g, device=dev, dtype=torch.float32)
            if name.endswith("norm.weight") or "layernorm" in name:
                p.copy_((1.0 + 0.1 * r).to(p.dtype))
            else:
                p.copy_((scale * r).to(p.dtype))
        return self

    @torch.no_grad()
    def load_hf_state_dict(self, sd):
        """Hugging Face key names (model.layers.{i}.mlp.experts.{e}.gate_proj.weight are stacked into switch_mlp)."""
        own = dict(self.named_parameters())
        for k, p in own.items():
            if ".switch_mlp." in k:
                pre, proj = k.split(".switch_mlp.")
                proj = proj[:-len(".weight")]
                p.copy_(torch.stack([sd[f"{pre}.experts.{e}.{proj}.weight"] for e in range(p.shape[0])]).to(p.dtype))
            else:
                p.copy_(sd[k].to(p.dtype))
        return self


# ---- hybrid decoders: every layer names its own mixer -------------------------------------------------------------------------

@dataclass
class LayerArgs:
    """One entry of a hybrid model's layer list: the mixer's type and sizes, its feed-forward (None: no second sublayer), and the
    layer whose tensors it uses (None: its own)."""
    type: str
    mixer: dict
    mlp: dict = None
    weights_of: int = None


@dataclass(frozen=True)
class Design:
    """What the decoders of one architecture have around their mixers.  prenorm: x <- x + m sublayer(norm(x)); otherwise
    x <- x + norm(sublayer(x)) and a weighted sum of all layers' results after every layer.  act: the feed-forward's activation,
    "xielu" (two parameters) or "gated_gelu" (a gate projection)."""
    prenorm: bool
    act: str
    tied: bool


DESIGNS = {"sebesun": Design(False, "xielu", False), "fabezen": Design(True, "gated_gelu", True)}


@dataclass
class HybridArgs:
    vocab_size: int
    hidden_size: int
    rms_norm_eps: float
    layers: list
    model_type: str = "sebesun"
    residual_mult: float = 1.0
    embed_scale: float = 1.0
    bigram: dict = None          # buckets, mul_prev, mul_cur of the table added per pair of neighbouring tokens

    @property
    def design(self):
        return DESIGNS[self.model_type]

    def source(self, i):
        """The layer whose tensors layer i uses."""
        seen = set()
        while self.layers[i].weights_of is not None:
            if i in seen:
                raise ValueError(f"layer {i}: its weights are its own through weights_of")
            seen.add(i)
            i = self.layers[i].weights_of
        return i

    @classmethod
    def from_config(cls, cfg):
        """cfg: the dictionary of a config.json with 'vocab', 'width', 'norm' and 'layers'."""
        layers = [LayerArgs(e["type"], dict(e["mixer"]), dict(e["mlp"]) if e.get("mlp") else None, e.get("weights_of")) for e in cfg["layers"]]
        for i, e in enumerate(layers):
            if e.type not in MIXERS:
                raise ValueError(f"layer {i}: mixer {e.type!r} is not one of {sorted(MIXERS)}")
            if e.mlp is not None and e.mlp.get("kind") != "dense":
                raise ValueError(f"layer {i}: feed-forward kind {e.mlp.get('kind')!r} (only 'dense')")
            m = e.mixer
            if "kv_heads" in m and m["heads"] % m["kv_heads"]:
                raise ValueError(f"layer {i}: {m['heads']} heads over {m['kv_heads']} key/value heads")
            if e.type == "retention" and len(m["decay"]) != m["heads"]:
                raise ValueError(f"layer {i}: {len(m['decay'])} decays for {m['heads']} heads")
            if e.type == "latent_attention" and m["rot_dim"] and m["rot"]["dims"] != m["rot_dim"]:
                raise ValueError(f"layer {i}: {m['rot']['dims']} rotated elements of a part of {m['rot_dim']}")
            if e.weights_of is not None:
                if not 0 <= e.weights_of < len(layers):
                    raise ValueError(f"layer {i}: weights of layer {e.weights_of}")
                o = layers[e.weights_of]
                if (o.type, o.mixer, o.mlp) != (e.type, e.mixer, e.mlp):
                    raise ValueError(f"layer {i} differs from layer {e.weights_of}, whose weights it uses")
        emb = cfg.get("embedding") or {}
        out = cls(cfg["vocab"], cfg["width"], float(cfg["norm"]["eps"]), layers, cfg["architecture"].lower(), float(cfg.get("residual_mult", 1.0)),
                  float(emb.get("scale", 1.0)), dict(emb["bigram"]) if emb.get("bigram") else None)
        for i in range(len(layers)):
            out.source(i)
        return out


def _mamba1_tensors(m, D):
    inner, r, n = m["inner"], m["dt_rank"], m["state"]
    return {"in": (2 * inner, D), "conv": (inner, m["conv"]), "conv.b": (inner,), "x": (r + 2 * n, inner), "dt": (inner, r), "dt.b": (inner,),
            "A_log": (inner, n), "D": (inner,), "o": (D, inner)}


def _retention_tensors(m, D):
    h, d, dv = m["heads"], m["dim"], m["vdim"]
    return {"q": (h * d, D), "k": (h * d, D), "v": (h * dv, D), "g": (h * dv, D), "o": (D, h * dv)}


def _diff_attention_tensors(m, D):
    h, g, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    return {"q": (2 * h * d, D), "k": (2 * g * d, D), "v": (g * dv, D), "q.norm": (d,), "k.norm": (d,), "lq1": (d,), "lk1": (d,), "lq2": (d,),
            "lk2": (d,), "o": (D, h * dv)}


def _delta_tensors(m, D, channel=False):
    h, g, d, dv, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
    out = {"q": (g * d, D), "q.conv": (g * d, taps), "k": (g * d, D), "k.conv": (g * d, taps), "v": (h * dv, D), "v.conv": (h * dv, taps),
           "b": (h, D), "A_log": (h,), "norm": (dv,), "o": (D, h * dv)}
    if channel:      # inner sizes of the low-rank products: the checkpoint's
        out.update({"a1": ("decay rank", D), "a2": (h * d, "decay rank"), "dt_bias": (h * d,), "g1": ("gate rank", D), "g2": (h * dv, "gate rank")})
    else:
        out.update({"a": (h, D), "dt_bias": (h,), "g": (h * dv, D)})
    return out


def _latent_attention_tensors(m, D):
    h, d, r, dv, R, Q = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
    return {"dq": (Q, D), "dq.norm": (Q,), "uq": (h * (d + r), Q), "dkv": (R + r, D), "dkv.norm": (R,), "uk": (h * d, R), "uv": (h * dv, R),
            "o": (D, h * dv)}


def _delta_cache(m, cap, dev, dt):
    return StateCache({"tail": (2 * m["kv_heads"] * m["dim"] + m["heads"] * m["vdim"], m["conv"] - 1), "kv": (m["heads"], m["dim"], m["vdim"])}, cap, dev)


# mixer type -> (tensor shapes, cache of one layer); a name instead of a size: any size, the same wherever a layer has the name
MIXERS = {
    "mamba1": (_mamba1_tensors, lambda m, cap, dev, dt: StateCache(
        {"tail": (m["inner"], m["conv"] - 1), "ssm": (m["inner"], m["state"])}, cap, dev)),
    "retention": (_retention_tensors, lambda m, cap, dev, dt: StateCache({"kv": (m["heads"], m["dim"], m["vdim"])}, cap, dev)),
    "attention": (_diff_attention_tensors, lambda m, cap, dev, dt: KVCache(
        2 * m["kv_heads"], m["dim"], cap, dev, dt, m["kv_heads"], m["vdim"])),
    "delta": (_delta_tensors, _delta_cache),
    "channel_delta": (lambda m, D: _delta_tensors(m, D, True), _delta_cache),
    "latent_attention": (_latent_attention_tensors, lambda m, cap, dev, dt: LatentCache(m["kv_rank"], m["rot_dim"], cap, dev, dt)),
}


class HybridLM:
    """Weights of a decoder whose layers name their mixers (selective scan, retention, differential attention, gated delta rules,
    latent attention): {tensor name: tensor} in the checkpoint's names, on one device, bfloat16 (the serving type) or float32."""

    def __init__(self, args, device="cuda", dtype=torch.bfloat16):
        assert dtype in (torch.bfloat16, torch.float32)
        self.args, self.device, self.dtype, self.w = args, torch.device(device), dtype, {}

    def shapes(self, sd=None, rank=None):
        """{name: shape}; sizes that only a checkpoint knows come from `sd`, or are `rank`."""
        a, ds = self.args, self.args.design
        D = a.hidden_size
        out = {"embed": (a.vocab_size, D), "final.norm": (D,)}
        if not ds.tied:
            out["head"] = (a.vocab_size, D)
        if a.bigram:
            out["bigram"] = (a.bigram["buckets"] + 1, D)
        for i, e in enumerate(a.layers):
            if e.weights_of is not None:
                continue
            free = {}
            for n, s in MIXERS[e.type][0](e.mixer, D).items():
                name = f"l{i}.mix.{n}"
                have = tuple(sd[name].shape) if sd is not None and name in sd else None
                for j, size in enumerate(s):
                    if isinstance(size, str):
                        free.setdefault(size, have[j] if have and len(have) == len(s) else rank or e.mixer["vdim"])
                out[name] = tuple(free[x] if isinstance(x, str) else x for x in s)
            out[f"l{i}.norm1"] = (D,)
            if not ds.prenorm:
                out[f"l{i}.dwa"] = (i + 2,)
            if e.mlp is not None:
                ff = e.mlp["ff"]
                out.update({f"l{i}.norm2": (D,), f"l{i}.mlp.up": (ff, D), f"l{i}.mlp.down": (D, ff)})
                out.update({f"l{i}.mlp.act": (2,)} if ds.act == "xielu" else {f"l{i}.mlp.gate": (ff, D)})
        return out

    def load_state_dict(self, sd):
        """sd: {name: tensor} with exactly the model's tensors."""
        shapes = self.shapes(sd)
        missing, extra = sorted(set(shapes) - set(sd)), sorted(set(sd) - set(shapes))
        if missing or extra:
            raise ValueError(f"checkpoint tensors: missing {missing[:5]}, unexpected {extra[:5]}")
        for n, s in shapes.items():
            if tuple(sd[n].shape) != tuple(s):
                raise ValueError(f"{n}: shape {tuple(sd[n].shape)}, expected {tuple(s)}")
            self.w[n] = sd[n].to(self.device, self.dtype).contiguous()
        return self

    @torch.no_grad()
    def init_random(self, seed=0, rank=None):
        """Seeded synthetic weights of the architecture."""
        g = torch.Generator(device=self.device).manual_seed(seed)
        for n, s in self.shapes(rank=rank).items():
            r = torch.randn(s, generator=g, device=self.device, dtype=torch.float32)
            leaf = n.split(".", 1)[-1]
            if leaf in ("norm1", "norm2", "norm", "mix.norm") or leaf.endswith((".norm", "mix.D")):
                r = 1.0 + 0.1 * r
            elif leaf == "dwa":
                r = 0.05 * r
                r[-1] += 1.0
            elif leaf.endswith("dt.b") or leaf == "mix.dt_bias":
                r -= 2.0
            elif len(s) == 2 and leaf != "mix.A_log" and not leaf.endswith("conv"):
                r /= s[1] ** 0.5
            else:
                r *= 0.3
            self.w[n] = r.to(self.dtype)
        return self


def make_prompt_cache(model, capacity, device=None):
    a = model.args
    if isinstance(model, HybridLM):
        device = device or model.device
        caches = [MIXERS[e.type][1](e.mixer, capacity, device, model.dtype) for e in a.layers]
        return caches + [TokenCache(capacity, device)] if a.bigram else caches
    device = device or model.model.embed_tokens.weight.device
    return [KVCache(a.num_key_value_heads, a.head_dim, capacity, device) for _ in model.model.layers]
