"""Plain NumPy float64 restatement of the hybrid decoder (host_model.HybridLM): one function per mechanism, token by token,
no code shared with the product.  Test infrastructure only.

A model is (cfg, W): cfg the dictionary of a config.json, W {tensor name: array}.  `forward` runs one sequence from its start
and returns the logits and the residual stream after every layer."""
import numpy as np

f64 = np.float64


def rms(x, eps):
    """x over its root mean square (last axis)."""
    x = np.asarray(x, f64)
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * np.asarray(z, f64)))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, np.asarray(z, f64))


def xielu(z, p, q):
    """softplus(p) z^2 + z/2 above zero; (1/2 + softplus(q)) (e^z - 1 - z) + z/2 at and below it."""
    z = np.asarray(z, f64)
    neg = np.minimum(z, 0.0)
    return np.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (np.expm1(neg) - neg)) + 0.5 * z


def causal_conv(x, w, b):
    """x [T, C], w [C, taps] (last column: the current token), zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    y = np.zeros(x.shape, f64)
    for t in range(T):
        for j in range(taps):
            s = t - (taps - 1 - j)
            if s >= 0:
                y[t] += w[:, j] * x[s]
    return y + b


def selective_scan(x, dt, A_log, B, C, D, S=None):
    """S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n,  y_c = sum_n S[c, n] C_n + D_c x_c.  Returns y and the last state."""
    A = -np.exp(np.asarray(A_log, f64))
    S = np.zeros(A.shape, f64) if S is None else S.copy()
    y = np.zeros(x.shape, f64)
    for t in range(x.shape[0]):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y, S


def rotate_half(x, base, dims, pos):
    """x [T, heads, d]: (x_i, x_{i + dims/2}) turned by pos * base^(-2i/dims), i < dims/2; the rest unchanged."""
    h = dims // 2
    ang = np.asarray(pos, f64)[:, None] * (float(base) ** (-2.0 * np.arange(h) / dims))[None, :]
    c, s = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
    out = np.array(x, f64)
    u, v = out[..., :h].copy(), out[..., h:dims].copy()
    out[..., :h], out[..., h:dims] = u * c - v * s, v * c + u * s
    return out


def retention(q, k, v, decay, S=None):
    """q, k [T, H, d] (k already scaled), v [T, H, dv]: S <- decay_h S + k v^T, o = S^T q.  Returns o and the last state."""
    T, H, d = q.shape
    S = np.zeros((H, d, v.shape[2]), f64) if S is None else S.copy()
    o = np.zeros((T, H, v.shape[2]), f64)
    for t in range(T):
        for h in range(H):
            S[h] = decay[h] * S[h] + np.outer(k[t, h], v[t, h])
            o[t, h] = q[t, h] @ S[h]
    return o, S


def causal_attention(q, k, v, scale):
    """One map of one head: q [T, d], k [T, d], v [T, dv]; softmax over every position up to the query's own."""
    out = np.zeros((q.shape[0], v.shape[1]), f64)
    for t in range(q.shape[0]):
        s = (k[:t + 1] @ q[t]) * scale
        p = np.exp(s - s.max())
        out[t] = (p / p.sum()) @ v[:t + 1]
    return out


def differential(a1, a2, lam, diff, eps):
    """rms(a1 - lambda a2) (1 - diff) over a head's values."""
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def diff_lambda(lq1, lk1, lq2, lk2, diff):
    return np.exp((np.asarray(lq1, f64) * lk1).sum()) - np.exp((np.asarray(lq2, f64) * lk2).sum()) + diff


def mix_mamba1(W, p, m, eps, h):
    xz = h @ W[p + "in"].T
    x, z = xz[:, :m["inner"]], xz[:, m["inner"]:]
    x = silu(causal_conv(x, W[p + "conv"], W[p + "conv.b"]))
    dbc = x @ W[p + "x"].T
    r, n = m["dt_rank"], m["state"]
    dt = softplus(dbc[:, :r] @ W[p + "dt"].T + W[p + "dt.b"])
    y, _ = selective_scan(x, dt, W[p + "A_log"], dbc[:, r:r + n], dbc[:, r + n:], W[p + "D"])
    return (y * silu(z)) @ W[p + "o"].T


def mix_retention(W, p, m, eps, h):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    pos = np.arange(T)
    q = rotate_half((h @ W[p + "q"].T).reshape(T, H, d), m["rot"]["base"], m["rot"]["dims"], pos)
    k = rotate_half((h @ W[p + "k"].T).reshape(T, H, d), m["rot"]["base"], m["rot"]["dims"], pos) * d ** -0.5
    o, _ = retention(q, k, (h @ W[p + "v"].T).reshape(T, H, dv), m["decay"])
    return (rms(o, eps).reshape(T, H * dv) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def mix_attention(W, p, m, eps, h):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ W[p + "q"].T).reshape(T, H, 2, d), eps) * W[p + "q.norm"]
    k = rms((h @ W[p + "k"].T).reshape(T, G, 2, d), eps) * W[p + "k.norm"]
    v = (h @ W[p + "v"].T).reshape(T, G, dv)
    lam = diff_lambda(W[p + "lq1"], W[p + "lk1"], W[p + "lq2"], W[p + "lk2"], m["diff"])
    o = np.zeros((T, H, dv), f64)
    for i in range(H):
        g = i // (H // G)
        a = [causal_attention(q[:, i, j], k[:, g, j], v[:, g], m["scale"]) for j in (0, 1)]
        o[:, i] = differential(a[0], a[1], lam, m["diff"], eps)
    return o.reshape(T, H * dv) @ W[p + "o"].T


MIXERS = {"mamba1": mix_mamba1, "retention": mix_retention, "attention": mix_attention}


def feed_forward(W, p, x):
    a = W[p + "act"]
    return xielu(x @ W[p + "up"].T, a[0], a[1]) @ W[p + "down"].T


def depth_average(X, w):
    """sum_j w_j X_j over the embedding output and every layer's result so far."""
    return sum(float(c) * x for c, x in zip(w, X))


def forward(cfg, W, tokens):
    """-> logits [T, vocab], residual stream after every layer [layers, T, width]."""
    W = {k: np.asarray(v, f64) for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)]
    X, stream = [x], []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + rms(MIXERS[layer["type"]](W, p + "mix.", layer["mixer"], eps, x), eps) * W[p + "norm1"]
        if layer["mlp"] is not None:
            x = x + rms(feed_forward(W, p + "mlp.", x), eps) * W[p + "norm2"]
        X.append(x)
        x = depth_average(X, W[p + "dwa"])
        stream.append(x)
    return (rms(x, eps) * W["final.norm"]) @ W["head"].T, np.stack(stream)


def random_weights(cfg, seed=0, sharp=1.0):
    """Seeded float32 weights of a configuration (sharp scales the query / key projections so that single keys stand out)."""
    r = np.random.default_rng(seed)
    D, V = cfg["width"], cfg["vocab"]
    lin = lambda o, i, g=1.0: (r.standard_normal((o, i)) * g / np.sqrt(i)).astype(np.float32)      # noqa: E731
    vec = lambda n, m=1.0, s=0.2: (m + s * r.standard_normal(n)).astype(np.float32)                # noqa: E731
    W = {"embed": r.standard_normal((V, D)).astype(np.float32), "final.norm": vec(D), "head": lin(V, D)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        W[p + "norm1"] = vec(D)
        W[p + "dwa"] = (r.standard_normal(i + 2) * 0.3 + (np.arange(i + 2) == i + 1)).astype(np.float32)
        q = p + "mix."
        if layer["type"] == "mamba1":
            I, R, N = m["inner"], m["dt_rank"], m["state"]
            W.update({q + "in": lin(2 * I, D), q + "conv": lin(I, m["conv"]), q + "conv.b": vec(I, 0.0), q + "x": lin(R + 2 * N, I),
                      q + "dt": lin(I, R), q + "dt.b": vec(I, -2.0, 1.0), q + "A_log": vec((I, N), 0.0, 1.0), q + "D": vec(I),
                      q + "o": lin(D, I)})
        elif layer["type"] == "retention":
            H, d, dv = m["heads"], m["dim"], m["vdim"]
            W.update({q + "q": lin(H * d, D, sharp), q + "k": lin(H * d, D), q + "v": lin(H * dv, D), q + "g": lin(H * dv, D),
                      q + "o": lin(D, H * dv)})
        else:
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            W.update({q + "q": lin(2 * H * d, D), q + "k": lin(2 * G * d, D), q + "v": lin(G * dv, D), q + "o": lin(D, H * dv),
                      q + "q.norm": vec(d, sharp), q + "k.norm": vec(d)})
            W.update({q + n: vec(d, 0.0, 0.3) for n in ("lq1", "lk1", "lq2", "lk2")})
        if layer["mlp"] is not None:
            F = layer["mlp"]["ff"]
            W.update({p + "norm2": vec(D), p + "mlp.up": lin(F, D), p + "mlp.down": lin(D, F), p + "mlp.act": vec(2, 0.5, 0.5)})
    return W
