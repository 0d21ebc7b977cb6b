"""Torch-level calls of the sequence-mixer kernels (include/scmx_mixers.h): matrix products for bfloat16 and float32 weights,
row kernels, selective scan, retention, differential attention, gated delta rules, latent attention.  Every function takes CUDA tensors and launches on torch's
current stream; there is no CPU path.  Activations are bfloat16 or float32 (the weights' type); the residual stream, norms,
scores and recurrent states are float32."""
import torch

from . import _lib

LOG2E = 1.4426950408889634


def _dt(t):
    if t.dtype == torch.bfloat16:
        return 0
    assert t.dtype == torch.float32, t.dtype
    return 1


def _ld(t):
    """Row pitch of a 2-D activation (unit column stride)."""
    assert t.dim() == 2 and (t.stride(1) == 1 or t.shape[1] == 1)
    return t.stride(0) if t.shape[0] > 1 else max(t.stride(0), t.shape[1])


def _round8(n):
    return (n + 7) // 8 * 8


def empty_rows(m, n, dtype, device):
    """[m, n] whose rows start 16-byte aligned."""
    return torch.empty((m, _round8(n)), dtype=dtype, device=device)[:, :n]


class XIELU:
    """Epilogue code and the two constants of an xIELU activation from its parameters (p, q): softplus(p) and 1/2 + softplus(q)."""

    code = 1

    def __init__(self, act):
        p, q = (torch.nn.functional.softplus(act.detach().double().cpu())).tolist()
        self.a_pos, self.a_neg = p, 0.5 + q


class GatedGELU:
    """gelu(gate) up (tanh form) of a product with W = GatedGELU.weight(gate, up): half as many outputs as rows."""
    code, a_pos, a_neg = 2, 0.0, 0.0

    @staticmethod
    def weight(gate, up):
        """Rows in turns of 16 gate and 16 up, zero padded to whole turns."""
        n, k = gate.shape
        m = (n + 15) // 16 * 16
        w = torch.zeros((2, m, k), dtype=gate.dtype, device=gate.device)
        w[0, :n], w[1, :n] = gate, up
        return w.view(2, m // 16, 16, k).transpose(0, 1).reshape(2 * m, k)


class Linear:
    """y = W x without bias.  W [N, K] bfloat16 (tcgen05 GEMM / GEMV kernels) or float32 (GEMV kernel for one row, the library's
    float32 product without reduced-precision modes otherwise)."""

    def __init__(self, w):
        self.N, self.K = w.shape
        ld = _round8(self.K)
        if ld == self.K:
            self.w = w.contiguous()
        else:
            self.w = torch.zeros((self.N, ld), dtype=w.dtype, device=w.device)
            self.w[:, :self.K] = w
        self.dt = _dt(w)

    def rows(self, r0, r1):
        """The product with some of the rows, on the same memory."""
        out = object.__new__(Linear)
        out.N, out.K, out.w, out.dt = r1 - r0, self.K, self.w[r0:r1], self.dt
        return out

    def _plan(self, M, splits, n_sm=148):
        """(tile, ranges of K computed side by side) for a product with few output tiles: the fewest bytes staged per SM, counting
        whole waves; at least 512 of K per range.  (0, 1): leave it to the kernel."""
        tm = -(-M // 128)
        if tm * -(-self.N // 64) >= n_sm or splits == 1:
            return 0, splits or 1
        cost = lambda tile, s: -(-tm * -(-self.N // tile) * s // n_sm) / s * (128 + tile)         # noqa: E731
        return min(((t, s) for t in (64, 128) for s in ([splits] if splits else range(1, max(1, min(8, self.K // 512)) + 1))),
                   key=lambda c: cost(*c))

    def __call__(self, x, out_dtype=None, act=None, tile=0, splits=None):
        """x [M, K] -> [M, N] (N / 2 with a gated activation) in out_dtype (default: the weights' type)."""
        out_dtype = out_dtype or self.w.dtype
        M = x.shape[0]
        assert x.shape[1] == self.K and x.dtype == self.w.dtype and x.is_cuda
        if self.dt == 1:
            with _full_float32():
                y = x @ self.w[:, :self.K].T
            if act is not None and act.code == 2:
                out = torch.empty((M, self.N // 2), dtype=y.dtype, device=y.device)
                _lib.mcall("scmx_gated_gelu", _lib.ptr(y), y.stride(0), M, self.N // 2, _lib.ptr(out), _lib.stream())
                return out
            if act is not None:
                _lib.mcall("scmx_xielu", _lib.ptr(y), y.numel(), act.a_pos, act.a_neg, _lib.stream())
            return y
        if _ld(x) % 8 or x.data_ptr() % 16:
            x = empty_rows(M, self.K, x.dtype, x.device).copy_(x)
        nout = self.N // 2 if act is not None and act.code == 2 else self.N
        y = empty_rows(M, nout, out_dtype, x.device)
        if tile == 0:
            tile, splits = self._plan(M, 1 if act is not None else splits)
        splits = splits or 1
        part = torch.empty(splits * M * ((self.N + 3) // 4 * 4), dtype=torch.float32, device=x.device) if splits > 1 else None
        _lib.mcall("scmx_gemm_bf16", _lib.ptr(x), _ld(x), _lib.ptr(self.w), self.w.shape[1], M, self.N, self.K, act.code if act else 0,
                   act.a_pos if act else 0.0, act.a_neg if act else 0.0, _lib.ptr(y), int(out_dtype == torch.float32), _round8(nout), tile, splits,
                   _lib.ptr(part), _lib.ptr(_lib.mixer_status_buffer()), _lib.stream())
        return y

    def vec(self, x, act=None, conv=None, out=None):
        """One float32 row [K] -> float32 [N] (N / 2 with a gated activation); conv = (weights [C, taps], bias [C] or None, tail) for
        the convolution epilogue."""
        assert x.dtype == torch.float32 and x.numel() == self.K and x.is_contiguous()
        epi = 2 if conv is not None else 0 if act is None else (0, 1, 3)[act.code]
        if out is None:
            out = torch.empty(self.N // 2 if epi == 3 else self.N, dtype=torch.float32, device=x.device)
        cw, cb, tail = conv if conv is not None else (None, None, None)
        _lib.mcall("scmx_gemv_x", _lib.ptr(self.w), self.w.shape[1], self.dt, _lib.ptr(x), self.N, self.K, epi, act.a_pos if act else 0.0,
                   act.a_neg if act else 0.0, _lib.ptr(cw), _lib.ptr(cb), _lib.ptr(tail), 0 if cw is None else cw.shape[0],
                   0 if cw is None else cw.shape[1], _lib.ptr(out), _lib.stream())
        return out


class _full_float32:
    """No TF32 in the float32 products, whatever the process-wide setting."""

    def __enter__(self):
        self.old = torch.backends.cuda.matmul.allow_tf32
        torch.backends.cuda.matmul.allow_tf32 = False

    def __exit__(self, *a):
        torch.backends.cuda.matmul.allow_tf32 = self.old


def embed(tokens, table, x, h=None):
    """x [T, W] float32 <- table rows; h: the same in the table's type."""
    _lib.require_cuda(tokens, table, x, h)
    _lib.mcall("scmx_embed", _lib.ptr(tokens), _lib.ptr(table), _dt(table), table.shape[0], tokens.numel(), table.shape[1], _lib.ptr(x),
               _lib.ptr(h), _lib.stream())


def embed_pair(tokens, table, x, scale, pairs=None, rule=(1, 0, 0), prev=None):
    """x [T, W] float32 <- scale table rows + pair-table rows, rule = (buckets, mul_prev, mul_cur); prev int64 [1] is advanced."""
    _lib.require_cuda(tokens, table, x, pairs, prev)
    _lib.mcall("scmx_embed_pair", _lib.ptr(tokens), _lib.ptr(table), _lib.ptr(pairs), _dt(table), table.shape[0], tokens.numel(), table.shape[1],
               scale, *rule, _lib.ptr(prev), _lib.ptr(x), _lib.stream())


def add_norm(y, x, w, mult, eps, h):
    """x <- x + mult y in place (y None: unchanged); h = x / rms(x) w in h's type."""
    _lib.mcall("scmx_add_norm", _lib.ptr(y), 0 if y is None else _ld(y), _lib.ptr(x), _lib.ptr(w), mult, eps, x.shape[0], x.shape[1], _lib.ptr(x),
               _lib.ptr(h), _dt(h), _lib.stream())


def res_norm(y, x, w, eps, x_out, h_out=None, average=None):
    """x_out = x + w * y / rms(y), or with average = (xs [n, T, W], weights [n], keep) the weighted sum of xs[: n - 1] and that
    value (stored at xs[n - 1] when keep)."""
    T, W = x.shape
    xs, dwa, keep = average if average is not None else (None, None, False)
    n = 0 if dwa is None else dwa.numel()
    _lib.mcall("scmx_res_norm", _lib.ptr(y), _ld(y), _lib.ptr(x), _lib.ptr(w), eps, T, W, _lib.ptr(xs), 0 if xs is None else xs.stride(0),
               _lib.ptr(dwa), n, int(keep), _lib.ptr(x_out), _lib.ptr(h_out), 1 if h_out is None else _dt(h_out), _lib.stream())


def norm_rows(x, w, eps, dtype, rows=None):
    M = x.shape[0] if rows is None else rows.numel()
    out = torch.empty((M, x.shape[1]), dtype=dtype, device=x.device)
    _lib.mcall("scmx_norm_rows", _lib.ptr(x), _lib.ptr(rows), _lib.ptr(w), eps, M, x.shape[1], _lib.ptr(out), _dt(out), _lib.stream())
    return out


def conv_silu(x, w, b, tail):
    """x [T, C] (row pitch free) -> silu(causal convolution); b may be None; tail is advanced."""
    T, C = x.shape
    out = empty_rows(T, C, x.dtype, x.device)
    _lib.mcall("scmx_conv_silu", _lib.ptr(x), _ld(x), _dt(x), T, C, w.shape[1], _lib.ptr(w), _lib.ptr(b), _lib.ptr(tail), _lib.ptr(out),
               _ld(out), _lib.stream())
    return out


def selective_scan(x, dtp, bc, z, dt_bias, A2, D, state):
    """x, z [T, C], dtp [T, C] float32, bc [T, 2 N] -> gated output [T, C]; state [C, N] is advanced."""
    T, C = x.shape
    y = empty_rows(T, C, x.dtype, x.device)
    _lib.mcall("scmx_selective_scan", _lib.ptr(x), _ld(x), _lib.ptr(dtp), _ld(dtp), _lib.ptr(bc), _ld(bc), _lib.ptr(z), _ld(z), _dt(x), T, C,
               A2.shape[1], _lib.ptr(dt_bias), _lib.ptr(A2), _lib.ptr(D), _lib.ptr(state), _lib.ptr(y), _ld(y), _lib.stream())
    return y


def scan_step(x, z, dbc, w_dt, dt_bias, A2, D, state, y):
    C, N = A2.shape
    _lib.mcall("scmx_scan_step", _lib.ptr(x), _lib.ptr(z), _lib.ptr(dbc), _lib.ptr(w_dt.w), w_dt.w.shape[1], w_dt.dt, C, N, w_dt.K,
               _lib.ptr(dt_bias), _lib.ptr(A2), _lib.ptr(D), _lib.ptr(state), _lib.ptr(y), _lib.stream())
    return y


DELTA_TC_MIN = 48           # shorter portions go token by token


def delta(q, k, v, b, a, channel, nA, dt_bias, state, form=0):
    """q, k [T, G d], v [T, H dv], b [T, H] -> o [T, H, dv] float32; a: decay logits [T, H], or float32 [T, H d] with `channel`; state
    [H, d, dv] is advanced.  form: 0 automatic, 1 token by token, 2 chunks on tensor cores (bfloat16)."""
    T, (H, d, dv) = q.shape[0], state.shape
    o = torch.empty((T, H, dv), dtype=torch.float32, device=q.device)
    assert not channel or a.dtype == torch.float32
    nbytes = 0
    if q.dtype == torch.bfloat16 and form != 1 and (form == 2 or T >= DELTA_TC_MIN):
        rows = (q, k, v, a) if channel else (q, k, v)
        aligned = not any(x.data_ptr() % 16 or _ld(x) % 8 for x in rows)
        nbytes = _lib.mixers().scmx_delta_scratch(T, H, d, dv, _ld(v)) if aligned else 0
    assert nbytes or form != 2, "no tensor-core form for these sizes"
    scratch = torch.empty(nbytes, dtype=torch.uint8, device=q.device) if nbytes else None
    _lib.mcall("scmx_delta", _lib.ptr(q), _ld(q), _lib.ptr(k), _ld(k), _lib.ptr(v), _ld(v), _lib.ptr(b), _ld(b), _lib.ptr(a), _ld(a), _dt(q), int(channel),
               T, H, q.shape[1] // d, d, dv, _lib.ptr(nA), _lib.ptr(dt_bias), _lib.ptr(state), _lib.ptr(o), _lib.ptr(scratch), nbytes,
               _lib.ptr(_lib.mixer_status_buffer()), _lib.stream())
    return o


def delta_step(q, k, v, b, a, g, wa, wg, nA, dt_bias, w, eps, state, y):
    """One token; wa, wg: the low-rank second products (Linear) of a decay per channel, or None."""
    H, d, dv = state.shape
    _lib.mcall("scmx_delta_step", _lib.ptr(q), _lib.ptr(k), _lib.ptr(v), _lib.ptr(b), _lib.ptr(a), _lib.ptr(g), None if wa is None else _lib.ptr(wa.w),
               0 if wa is None else wa.w.shape[1], 0 if wa is None else wa.K, None if wg is None else _lib.ptr(wg.w),
               0 if wg is None else wg.w.shape[1], 0 if wg is None else wg.K, 0 if wa is None else wa.dt, H, q.numel() // d, d, dv, _lib.ptr(nA),
               _lib.ptr(dt_bias), _lib.ptr(w), eps, _lib.ptr(state), _lib.ptr(y), _lib.stream())
    return y


def latent_append(y, Q, R, r, qw, cw, cs, eps, cache, cq_dtype, pos_dev=None):
    """y [T, Q + R + r]: normalized query latents [T, Q]; latents and rotated key parts go to rows cache.offset .. of the cache."""
    T = y.shape[0]
    cq = empty_rows(T, Q, cq_dtype, y.device)
    _lib.mcall("scmx_latent_append", _lib.ptr(y), _ld(y), _dt(y), _dt(cache.c), _dt(cq), T, Q, R, r, _lib.ptr(qw), _lib.ptr(cw), _lib.ptr(cs), cs.shape[0],
               eps, cache.offset, _lib.ptr(pos_dev), _lib.ptr(cq), _ld(cq), _lib.ptr(cache.c), cache.c.shape[1], cache.capacity, _lib.stream())
    return cq


def latent_rows(q, wuk, wuv, cs, cache, H, d, r, dv, window, scale, out_dtype, pos_dev=None, n_sm=148):
    """q [T, H (d + r)] (parts not rotated) at positions cache.offset .. -> [T, H dv], through queries in the latent space."""
    T, R, dev = q.shape[0], wuk.K, q.device
    qa = torch.empty((T, H, R + r), dtype=torch.float32, device=dev)
    pos, pd = cache.offset, _lib.ptr(pos_dev)
    _lib.mcall("scmx_latent_absorb", _lib.ptr(q), _ld(q), _dt(q), _lib.ptr(wuk.w), wuk.w.shape[1], wuk.dt, _lib.ptr(cs), cs.shape[0], T, H, d, R, r, pos, pd,
               _lib.ptr(qa), _lib.stream())
    groups = -(-H // 8)
    nsplit = max(1, min(64, n_sm // (groups * T)))
    part = torch.empty((T, H, nsplit, (R + 3) // 4 * 4 + 4), dtype=torch.float32, device=dev)
    _lib.mcall("scmx_latent_rows", _lib.ptr(qa), _lib.ptr(cache.c), cache.c.shape[1], _dt(cache.c), T, pos, pd, cache.capacity, window, H, R, r, scale,
               nsplit, _lib.ptr(part), _lib.stream())
    o = empty_rows(T, H * dv, out_dtype, dev)
    _lib.mcall("scmx_latent_value", _lib.ptr(part), _lib.ptr(wuv.w), wuv.w.shape[1], wuv.dt, T, pos, pd, cache.capacity, window, H, R, dv, nsplit,
               _lib.ptr(o), _ld(o), _dt(o), _lib.stream())
    return o


LATENT_TC_MIN = 32          # shorter portions are attended in the latent space


def latent_prompt_supported(q, d, r, dv, scale):
    return q.dtype == torch.bfloat16 and not (d % 8 or r % 8 or dv % 8) and d <= 128 and r <= 64 and dv <= 128 and scale > 0


def latent_prompt(q, ukv, cs, cache, H, d, r, dv, R, window, scale):
    """The same for a bfloat16 prompt portion on tensor cores: keys and values of every visible position are products of its latent
    (ukv: W_uk over W_uv); q's rotated parts are turned in place."""
    T, pos = q.shape[0], cache.offset
    k0 = max(0, pos + 1 - window) if window else 0
    rows = cache.c[k0:pos + T]
    kv = ukv(rows[:, :R])
    _lib.mcall("scmx_latent_rotate", _lib.ptr(q), _ld(q), _dt(q), _lib.ptr(cs[pos:]), T, H, d, r, _lib.stream())
    o = torch.empty((T, H * dv), dtype=q.dtype, device=q.device)
    _lib.mcall("scmx_latent_attn", _lib.ptr(q), _ld(q), _lib.ptr(kv), _ld(kv), _lib.ptr(rows[:, _round8(R):]) if r else None, rows.shape[1], T, pos, k0,
               window, H, d, r, dv, scale, _lib.ptr(o), _lib.ptr(_lib.mixer_status_buffer()), _lib.stream())
    return o


def rotary_table(base, dims, rows, device):
    """float32 [rows, dims]: cos then sin of position * base^(-2i/dims), angles in float64."""
    f = float(base) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64, device=device) / max(dims, 1))
    ang = torch.arange(rows, dtype=torch.float64, device=device)[:, None] * f[None, :]
    return torch.cat([torch.cos(ang), torch.sin(ang)], 1).float().contiguous()


RETENTION_TC_MIN = 32       # shorter portions go token by token


def retention(q, k, v, cs, dims, kscale, decay, state, form=0):
    """q, k [T, H d], v [T, H dv] -> o [T, H, dv] float32; cs: the table rows of this portion; state [H, d, dv] is advanced.
    form: 0 automatic, 1 token by token, 2 chunks on tensor cores (bfloat16, positive decays)."""
    T, (H, d, dv) = q.shape[0], state.shape
    o = torch.empty((T, H, dv), dtype=torch.float32, device=q.device)
    nbytes = 0
    if q.dtype == torch.bfloat16 and form != 1 and (form == 2 or T >= RETENTION_TC_MIN):
        nbytes = 0 if v.data_ptr() % 16 else _lib.mixers().scmx_retention_scratch(T, H, d, dv, dims, _ld(v))
    assert nbytes or form != 2, "no tensor-core form for these sizes"
    scratch = torch.empty(nbytes, dtype=torch.uint8, device=q.device) if nbytes else None
    _lib.mcall("scmx_retention", _lib.ptr(q), _ld(q), _lib.ptr(k), _ld(k), _lib.ptr(v), _ld(v), _dt(q), T, H, d, dv, _lib.ptr(cs), dims, kscale,
               _lib.ptr(decay), _lib.ptr(state), _lib.ptr(o), _lib.ptr(scratch), nbytes, _lib.ptr(_lib.mixer_status_buffer()), _lib.stream())
    return o


def head_norm_gate(o, g, eps, w=None, gate=0):
    """o [T, H, dv] / rms * w * gate(g), gate 0 = SiLU, 1 = sigmoid."""
    T, H, dv = o.shape
    out = torch.empty((T, H * dv), dtype=g.dtype, device=o.device)
    _lib.mcall("scmx_head_norm_gate", _lib.ptr(o), _lib.ptr(g), _ld(g), _dt(g), _lib.ptr(w), gate, T, H, dv, eps, _lib.ptr(out), _lib.stream())
    return out


def retention_step(q, k, v, g, table, dims, kscale, decay, eps, state, y, pos=0, pos_dev=None):
    H, d, dv = state.shape
    _lib.mcall("scmx_retention_step", _lib.ptr(q), _lib.ptr(k), _lib.ptr(v), _lib.ptr(g), H, d, dv, _lib.ptr(table), max(1, table.shape[0]), dims,
               pos, _lib.ptr(pos_dev), kscale, _lib.ptr(decay), eps, _lib.ptr(state), _lib.ptr(y), _lib.stream())
    return y


def qk_norm_append(q, k, v, H, G, qw, kw, eps, cache, q_dtype, pos_dev=None):
    """q [T, 2 H d], k [T, 2 G d], v [T, G dv]: normalized q [2 H, T, d]; normalized k and v go to rows cache.offset .. of the cache."""
    T, d, dv, cap = q.shape[0], qw.numel(), cache.v.shape[2], cache.k.shape[1]
    qo = torch.empty((2 * H, T, d), dtype=q_dtype, device=q.device)
    _lib.mcall("scmx_qk_norm_append", _lib.ptr(q), _ld(q), _lib.ptr(k), _ld(k), _lib.ptr(v), _ld(v), _dt(q), _dt(cache.k), _dt(qo), T, H, G, d, dv,
               _lib.ptr(qw), _lib.ptr(kw), eps, cache.offset, _lib.ptr(pos_dev), _lib.ptr(qo), _lib.ptr(cache.k), _lib.ptr(cache.v), cap,
               _lib.stream())
    return qo


def diff_attention(q, cache, H, G, scale, lam, diff, eps, form=0):
    """q [2 H, T, d] at positions cache.offset .. (their keys and values already in the cache) -> [T, H dv].  form: 0 automatic,
    1 CUDA cores, 2 tensor cores."""
    T, d, dv = q.shape[1], q.shape[2], cache.v.shape[2]
    o = torch.empty((T, H * dv), dtype=q.dtype, device=q.device)
    _lib.mcall("scmx_diff_attn", _lib.ptr(q), _lib.ptr(cache.k), _lib.ptr(cache.v), _dt(q), T, cache.offset, cache.k.shape[1], H, G, d, dv, scale,
               lam, diff, eps, _lib.ptr(o), form, _lib.ptr(_lib.mixer_status_buffer()), _lib.stream())
    return o


class DiffDecodeAttention:
    """One query row of differential attention over the cache, with its scratch."""

    def __init__(self, H, G, d, dv, device, n_sm=148):
        self.H, self.G, self.d, self.dv = H, G, d, dv
        self.nsplit = max(1, min(32, 2 * n_sm // G))
        self.part = torch.empty((G, self.nsplit, 2 * (H // G), dv + 2), dtype=torch.float32, device=device)
        self.counters = torch.zeros(H, dtype=torch.int32, device=device)

    def __call__(self, q, cache, scale, lam, diff, eps, o, n_pos=None, pos_dev=None):
        _lib.mcall("scmx_diff_decode", _lib.ptr(q), _lib.ptr(cache.k), _lib.ptr(cache.v), _dt(cache.k), int(n_pos or 0), _lib.ptr(pos_dev),
                   cache.k.shape[1], self.H, self.G, self.d, self.dv, scale, lam, diff, eps, self.nsplit, _lib.ptr(self.part),
                   _lib.ptr(self.counters), _lib.ptr(o), _lib.stream())
        return o
