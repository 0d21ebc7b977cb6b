"""Plain NumPy float64 restatement of the Fabezen decoder (gated delta rules with a decay per head or per key channel, latent
attention in a sliding window, pre-norm residuals, a bigram embedding, layers that share weights): one function per mechanism,
token by token, no code shared with the product.  Test infrastructure only.

A model is (cfg, W): cfg the dictionary of a config.json, W {tensor name: array}.  `forward` runs one sequence from its start
and returns the logits and the residual stream after every layer."""
import numpy as np

f64 = np.float64


def rms_norm(x, w, eps):
    x = np.asarray(x, f64)
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * np.asarray(z, f64)))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, np.asarray(z, f64))


def gelu_tanh(z):
    z = np.asarray(z, f64)
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def embedding(W, cfg, tokens):
    """Scaled token row plus the row of the (previous, current) pair; the table's last row where there is no previous token."""
    e = cfg["embedding"]
    x = []
    for t, tok in enumerate(tokens):
        r = W["embed"][tok] * e["scale"]
        if e.get("bigram"):
            b = e["bigram"]
            row = b["buckets"] if t == 0 else (int(tokens[t - 1]) * b["mul_prev"] + int(tok) * b["mul_cur"]) % b["buckets"]
            r = r + W["bigram"][row]
        x.append(r)
    return np.array(x, f64)


def short_conv(x, w):
    """x [T, C], w [C, taps] (last column: the current token), zeros before the start, then silu."""
    T, taps = x.shape[0], w.shape[1]
    y = np.zeros(x.shape, f64)
    for t in range(T):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                y[t] += w[:, j] * x[s]
    return silu(y)


def unit(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


def log_decay(A_log, a, dt_bias):
    """A_log [H], a and dt_bias [..., H] or [..., H, d]: logarithm of the decay."""
    A = np.exp(np.asarray(A_log, f64))
    z = softplus(a + dt_bias)
    return -(A[:, None] if z.ndim == 3 else A) * z


def delta_rule(q, k, v, g, beta, S=None):
    """q, k [T, Hk, d] (q scaled), v [T, H, dv], g [T, H, d] decays, beta [T, H]:
    S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q.   Returns o and the last state."""
    T, Hk, d = q.shape
    H, dv = v.shape[1:]
    S = np.zeros((H, d, dv), f64) if S is None else np.array(S, f64)
    o = np.zeros((T, H, dv), f64)
    for t in range(T):
        for h in range(H):
            kh = h // (H // Hk)
            S[h] = g[t, h][:, None] * S[h]
            u = beta[t, h] * (v[t, h] - S[h].T @ k[t, kh])
            S[h] = S[h] + np.outer(k[t, kh], u)
            o[t, h] = S[h].T @ q[t, kh]
    return o, S


def mix_delta(W, p, m, eps, h, channel):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (short_conv(h @ W[p + n].T, W[p + n + ".conv"]) for n in "qkv")
    q = unit(q.reshape(T, G, d)) * d ** -0.5
    k = unit(k.reshape(T, G, d))
    beta = sigmoid(h @ W[p + "b"].T)
    if channel:
        a = ((h @ W[p + "a1"].T) @ W[p + "a2"].T).reshape(T, H, d)
        g = np.exp(log_decay(W[p + "A_log"], a, W[p + "dt_bias"].reshape(H, d)))
        gate = sigmoid((h @ W[p + "g1"].T) @ W[p + "g2"].T)
    else:
        g = np.exp(log_decay(W[p + "A_log"], h @ W[p + "a"].T, W[p + "dt_bias"]))[:, :, None] * np.ones(d)
        gate = silu(h @ W[p + "g"].T)
    o, _ = delta_rule(q, k, v.reshape(T, H, dv), g, beta)
    return (rms_norm(o, W[p + "norm"], eps).reshape(T, H * dv) * gate) @ W[p + "o"].T


def rotate_pairs(x, base, dims, pos):
    """x [T, ..., d]: (x_2i, x_2i+1) turned by pos * base^(-2i/dims) for 2i < dims; the rest unchanged."""
    out = np.array(x, f64)
    for t, p in enumerate(pos):
        for i in range(dims // 2):
            a = p * float(base) ** (-2.0 * i / dims)
            u, v = x[t, ..., 2 * i], x[t, ..., 2 * i + 1]
            out[t, ..., 2 * i], out[t, ..., 2 * i + 1] = u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)
    return out


def window_attention(q, k, v, scale, size):
    """One head: position i sees j with 0 <= i - j < size (None: every j up to i)."""
    out = np.zeros((q.shape[0], v.shape[1]), f64)
    for i in range(q.shape[0]):
        lo = 0 if size is None else max(0, i - size + 1)
        s = (k[lo:i + 1] @ q[i]) * scale
        p = np.exp(s - s.max())
        out[i] = (p / p.sum()) @ v[lo:i + 1]
    return out


def mix_latent(W, p, m, eps, h):
    T, H, d, r, dv, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    q = (rms_norm(h @ W[p + "dq"].T, W[p + "dq.norm"], eps) @ W[p + "uq"].T).reshape(T, H, d + r)
    ckr = h @ W[p + "dkv"].T
    c = rms_norm(ckr[:, :R], W[p + "dkv.norm"], eps)
    base, dims = (m["rot"]["base"], m["rot"]["dims"]) if r else (1.0, 0)
    kr = rotate_pairs(ckr[:, R:], base, dims, pos)
    qr = rotate_pairs(q[..., d:], base, dims, pos)
    k, v = (c @ W[p + "uk"].T).reshape(T, H, d), (c @ W[p + "uv"].T).reshape(T, H, dv)
    size = (m.get("mask") or {}).get("size")
    o = np.stack([window_attention(np.concatenate([q[:, i, :d], qr[:, i]], 1), np.concatenate([k[:, i], kr], 1), v[:, i], m["scale"], size)
                  for i in range(H)], 1)
    return o.reshape(T, H * dv) @ W[p + "o"].T


MIXERS = {"delta": lambda *a: mix_delta(*a, False), "channel_delta": lambda *a: mix_delta(*a, True), "latent_attention": mix_latent}


def feed_forward(W, p, h):
    return (gelu_tanh(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def forward(cfg, W, tokens):
    """-> logits [T, vocab], residual stream after every layer [layers, T, width]."""
    W = {k: np.asarray(v, f64) for k, v in W.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x, stream = embedding(W, cfg, tokens), []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i if layer.get('weights_of') is None else layer['weights_of']}."
        x = x + mult * MIXERS[layer["type"]](W, p + "mix.", layer["mixer"], eps, rms_norm(x, W[p + "norm1"], eps))
        if layer["mlp"] is not None:
            x = x + mult * feed_forward(W, p + "mlp.", rms_norm(x, W[p + "norm2"], eps))
        stream.append(x)
    return rms_norm(x, W["final.norm"], eps) @ W["embed"].T, np.stack(stream)


def random_weights(cfg, seed=0, sharp=1.0):
    """Seeded float32 weights of a configuration (sharp scales the attention queries so that single keys stand out)."""
    r = np.random.default_rng(seed)
    D, V = cfg["width"], cfg["vocab"]
    lin = lambda o, i, g=1.0: (r.standard_normal((o, i)) * g / np.sqrt(i)).astype(np.float32)      # noqa: E731
    vec = lambda n, m=1.0, s=0.2: (m + s * r.standard_normal(n)).astype(np.float32)                # noqa: E731
    W = {"embed": lin(V, D), "final.norm": vec(D)}
    if cfg["embedding"].get("bigram"):
        W["bigram"] = r.standard_normal((cfg["embedding"]["bigram"]["buckets"] + 1, D)).astype(np.float32)
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", layer["mixer"]
        q = p + "mix."
        W[p + "norm1"] = vec(D)
        if layer["type"] == "latent_attention":
            H, d, rd, dv, R, Q = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            W.update({q + "dq": lin(Q, D), q + "dq.norm": vec(Q, sharp), q + "uq": lin(H * (d + rd), Q), q + "dkv": lin(R + rd, D), q + "dkv.norm": vec(R),
                      q + "uk": lin(H * d, R), q + "uv": lin(H * dv, R), q + "o": lin(D, H * dv)})
        else:
            H, G, d, dv, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for n, c in (("q", G * d), ("k", G * d), ("v", H * dv)):
                W.update({q + n: lin(c, D), q + n + ".conv": lin(c, taps)})
            W.update({q + "b": lin(H, D), q + "A_log": vec(H, -1.0, 1.0), q + "norm": vec(dv), q + "o": lin(D, H * dv)})
            if layer["type"] == "channel_delta":
                ra, rg = m.get("ranks", (max(1, d // 3), max(1, dv // 4)))      # inner sizes of the two low-rank products: a test's own choice
                W.update({q + "a1": lin(ra, D), q + "a2": lin(H * d, ra), q + "dt_bias": vec(H * d, -1.0, 1.5), q + "g1": lin(rg, D),
                          q + "g2": lin(H * dv, rg)})
            else:
                W.update({q + "a": lin(H, D), q + "dt_bias": vec(H, -1.0, 1.5), q + "g": lin(H * dv, D)})
        if layer["mlp"] is not None:
            F = layer["mlp"]["ff"]
            W.update({p + "norm2": vec(D), p + "mlp.gate": lin(F, D, 2.0), p + "mlp.up": lin(F, D), p + "mlp.down": lin(D, F)})
    return W
