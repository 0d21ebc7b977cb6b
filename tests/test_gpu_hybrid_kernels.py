"""GPU: every kernel of the sequence mixers against the plain float64 oracle, at sizes on and off the tiles' borders, carried
states over portions, far and near keys, reused slots."""
import numpy as np
import pytest
import torch

import hybrid_oracle as O

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32


@pytest.fixture(scope="module")
def X(scmx):
    return scmx.sc_mixers


@pytest.fixture(autouse=True)
def _no_wait_ran_out(scmx):
    yield
    torch.cuda.synchronize()
    scmx._lib.check_mixer_status()


def rnd(seed, *shape, scale=1.0, dtype=F32):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(shape, generator=g) * scale).to(dtype).cuda()


def npy(t):
    return t.detach().double().cpu().numpy()


def err(got, want):
    """Largest difference relative to the wanted value plus the root mean square of all of them."""
    want = np.asarray(want, np.float64)
    return float((np.abs(npy(got) - want) / (np.abs(want) + np.sqrt((want ** 2).mean()) + 1e-30)).max())


# ---- matrix products --------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("M,N,K,tile", [(1, 40, 24, 0), (2, 8, 16, 64), (130, 72, 100, 64), (200, 300, 264, 128), (300, 520, 192, 256), (129, 256, 64, 256),
                                        (513, 1000, 72, 256), (77, 33, 13, 0)])
@pytest.mark.parametrize("out", [BF, F32])
def test_gemm(X, M, N, K, tile, out):
    x, w = rnd(1, M, K, dtype=BF), rnd(2, N, K, scale=K ** -0.5, dtype=BF)
    y = X.Linear(w)(x, out, tile=tile)
    assert err(y, npy(x) @ npy(w).T) < (2e-2 if out == BF else 2e-5)


@pytest.mark.parametrize("M,N,K,tile,splits", [(40, 24, 1000, 64, 3), (300, 72, 2048, 128, 8), (130, 300, 640, 256, 2), (5, 160, 4096, 0, None)])
@pytest.mark.parametrize("out", [BF, F32])
def test_gemm_split_inner(X, M, N, K, tile, splits, out):
    x, w = rnd(1, M, K, dtype=BF), rnd(2, N, K, scale=K ** -0.5, dtype=BF)
    y = X.Linear(w)(x, out, tile=tile, splits=splits)
    assert err(y, npy(x) @ npy(w).T) < (2e-2 if out == BF else 2e-5)


def test_gemm_strided_input_and_activation(X):
    x, w = rnd(3, 150, 96, dtype=BF)[:, :40], rnd(4, 136, 40, scale=0.3, dtype=BF)
    act = X.XIELU(torch.tensor([-0.8, 1.3]))
    want = O.xielu(npy(x) @ npy(w).T, -0.8, 1.3)
    assert err(X.Linear(w)(x, F32, act=act), want) < 3e-5
    assert err(X.Linear(w)(x, act=act), want) < 3e-2
    assert err(X.Linear(w.float())(x.float(), act=act), want) < 3e-5


@pytest.mark.parametrize("N,K", [(5, 7), (64, 40), (300, 1000), (1030, 2048), (96, 4104)])
@pytest.mark.parametrize("dt", [BF, F32])
def test_gemv(X, N, K, dt):
    x, w = rnd(5, K), rnd(6, N, K, scale=K ** -0.5, dtype=dt)
    y = npy(w) @ npy(x)
    assert err(X.Linear(w).vec(x), y) < 1e-5
    act = X.XIELU(torch.tensor([0.4, -0.2]))
    assert err(X.Linear(w).vec(x, act=act), O.xielu(y, 0.4, -0.2)) < 2e-5


@pytest.mark.parametrize("taps", [1, 2, 4, 6])
def test_gemv_convolution_epilogue(X, taps):
    N, K, C, T = 50, 24, 30, 9
    w, xs = rnd(7, N, K, scale=0.3, dtype=BF), rnd(8, T, K)
    cw, cb, tail = rnd(9, C, taps), rnd(10, C), torch.zeros(C, taps - 1).cuda()
    got = torch.stack([X.Linear(w).vec(x, conv=(cw, cb, tail)) for x in xs])
    y = npy(xs) @ npy(w).T
    want = np.concatenate([O.silu(O.causal_conv(y[:, :C], npy(cw), npy(cb))), y[:, C:]], 1)
    assert err(got, want) < 2e-5
    if taps > 1:
        assert err(tail, y[T - taps + 1:, :C].T) < 1e-5


# ---- row kernels ------------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("T,W", [(1, 40), (1, 2048), (3, 1030), (70, 516), (200, 33)])
@pytest.mark.parametrize("n", [0, 2, 5])
def test_res_norm(X, T, W, n):
    y, x, w = rnd(11, T, W), rnd(12, T, W), rnd(13, W)
    xs, dwa = rnd(14, max(n, 1), T, W), rnd(15, n) if n else None
    r = npy(x) + O.rms(npy(y), 1e-3) * npy(w)
    want = r if n == 0 else O.depth_average(list(npy(xs)[:n - 1]) + [r], npy(dwa))
    out, h = torch.empty(T, W).cuda(), torch.empty(T, W, dtype=BF).cuda()
    X.res_norm(y, x, w, 1e-3, out, h, (xs, dwa, True) if n else None)
    assert err(out, want) < 1e-5 and torch.equal(h, out.to(BF))
    if n:
        assert err(xs[n - 1], r) < 1e-5
    X.res_norm(y, x, w, 1e-3, x, None, (xs, dwa, False) if n else None)      # in place, nothing kept
    assert torch.equal(x, out)


def test_embed_and_norm_rows(X):
    tab, ids = rnd(16, 30, 44, dtype=BF), torch.tensor([3, 29, 0, 3]).cuda()
    x, h = torch.empty(4, 44).cuda(), torch.empty(4, 44, dtype=BF).cuda()
    X.embed(ids, tab, x, h)
    assert torch.equal(h, tab[ids]) and torch.equal(x, tab[ids].float())
    w, rows = rnd(17, 44), torch.tensor([2, 0]).cuda()
    assert err(X.norm_rows(x, w, 1e-2, F32, rows), O.rms(npy(x)[[2, 0]], 1e-2) * npy(w)) < 1e-5
    assert err(X.norm_rows(x, w, 1e-2, BF), O.rms(npy(x), 1e-2) * npy(w)) < 2e-2


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
@pytest.mark.parametrize("dt", [BF, F32])
def test_conv_portions(X, taps, dt):
    T, C = 53, 37
    x, w, b = rnd(18, T, C, dtype=dt), rnd(19, C, taps), rnd(20, C)
    want = O.silu(O.causal_conv(npy(x), npy(w), npy(b)))
    for cuts in ([53], [2] * 26 + [1], [17, 1, 1, 16, 18], [1, 52]):
        tail, got = torch.zeros(C, taps - 1).cuda(), []
        for part in x.split(cuts):
            got.append(X.conv_silu(part, w, b, tail))
        assert err(torch.cat(got), want) < (2e-2 if dt == BF else 1e-5), cuts


def test_head_norm_gate(X):
    o, g = rnd(21, 9, 3, 20), rnd(22, 9, 3 * 20 + 4)[:, 4:]
    want = (O.rms(npy(o), 1e-2).reshape(9, 60)) * O.silu(npy(g))
    assert err(X.head_norm_gate(o, g, 1e-2), want) < 1e-5


# ---- selective scan ---------------------------------------------------------------------------------------------------------

def scan_case(C, N, T, dt):
    x, z, bc = rnd(30, T, C, dtype=dt), rnd(31, T, C, dtype=dt), rnd(32, T, 2 * N, dtype=dt)
    dtp, bias, A_log, D = rnd(33, T, C), rnd(34, C) - 1, rnd(35, C, N), rnd(36, C)
    A2 = (-torch.exp(A_log.double()) * 1.4426950408889634).float()
    y, S = O.selective_scan(npy(x), O.softplus(npy(dtp) + npy(bias)), npy(A_log), npy(bc)[:, :N], npy(bc)[:, N:], npy(D))
    return (x, dtp, bc, z, bias, A2, D), y * O.silu(npy(z)), S


@pytest.mark.parametrize("C,N,T", [(5, 1, 40), (130, 5, 33), (70, 16, 100), (36, 24, 65), (33, 12, 64), (10, 40, 31), (9, 130, 20), (6, 256, 18)])
@pytest.mark.parametrize("dt", [BF, F32])
def test_scan_portions(X, C, N, T, dt):
    args, want, S = scan_case(C, N, T, dt)
    for cuts in ([T], [2, 1, 9, T - 12], [T - 1, 1]):
        state, got = torch.zeros(C, N).cuda(), []
        for x, dtp, bc, z in zip(*(a.split(cuts) for a in args[:4])):
            got.append(X.selective_scan(x, dtp, bc, z, *args[4:], state))
        assert err(torch.cat(got), want) < (3e-2 if dt == BF else 3e-5), cuts
        assert err(state, S) < 3e-5


@pytest.mark.parametrize("C,N,R", [(40, 16, 8), (70, 5, 3), (33, 24, 100), (8, 130, 20)])
@pytest.mark.parametrize("dt", [BF, F32])
def test_scan_steps(X, C, N, R, dt):
    T = 12
    (x, _, bc, z, bias, A2, D), _, _ = scan_case(C, N, T, F32)
    r, w, A_log = rnd(37, T, R), rnd(38, C, R, scale=0.4, dtype=dt), np.log(-npy(A2) / 1.4426950408889634)
    y, S = O.selective_scan(npy(x), O.softplus(npy(r) @ npy(w).T + npy(bias)), A_log, npy(bc)[:, :N], npy(bc)[:, N:], npy(D))
    state, lin, out = torch.zeros(C, N).cuda(), X.Linear(w), []
    for t in range(T):
        out.append(X.scan_step(x[t], z[t], torch.cat([r[t], bc[t]]), lin, bias, A2, D, state, torch.empty(C).cuda()))
    assert err(torch.stack(out), y * O.silu(npy(z))) < 3e-5 and err(state, S) < 3e-5


# ---- retention --------------------------------------------------------------------------------------------------------------

def ret_case(X, T, H, d, dv, dims, dt, decay=None):
    qkv = rnd(40, T, 2 * H * d + H * dv, dtype=dt)
    q, k, v = qkv.split([H * d, H * d, H * dv], 1)
    decay = decay or [1 - 2.0 ** (-1 - 1.3 * h) for h in range(H)]
    table = X.rotary_table(70.0, dims, T, "cuda")
    shape = lambda t, n: npy(t).reshape(T, H, n)                                          # noqa: E731
    qq, kk = O.rotate_half(shape(q, d), 70.0, dims, range(T)), O.rotate_half(shape(k, d), 70.0, dims, range(T)) * d ** -0.5
    return (q, k, v, table, torch.tensor(decay).cuda()), O.retention(qq, kk, shape(v, dv), decay)


def run_ret(X, case, H, d, dv, dims, cuts, form):
    (q, k, v, table, decay), _ = case
    state, got, pos = torch.zeros(H, d, dv).cuda(), [], 0
    for a, b, c in zip(*(t.split(cuts) for t in (q, k, v))):
        got.append(X.retention(a, b, c, table[pos:], dims, d ** -0.5, decay, state, form))
        pos += a.shape[0]
    return torch.cat(got), state


@pytest.mark.parametrize("H,d,dv,dims,T", [(3, 16, 24, 8, 70), (1, 5, 33, 4, 40), (2, 64, 40, 64, 33), (2, 20, 8, 0, 30)])
@pytest.mark.parametrize("dt", [BF, F32])
def test_retention_token_by_token(X, H, d, dv, dims, T, dt):
    case = ret_case(X, T, H, d, dv, dims, dt)
    for cuts in ([T], [2, 1, 8, T - 11]):
        o, S = run_ret(X, case, H, d, dv, dims, cuts, 1)
        assert err(o, case[1][0]) < 2e-5 and err(S, case[1][1]) < 2e-5


@pytest.mark.parametrize("H,d,dv,dims", [(2, 8, 8, 8), (3, 32, 64, 16), (2, 72, 40, 72), (1, 128, 136, 64), (2, 64, 200, 0), (1, 256, 72, 256), (1, 136, 64, 8)])
def test_retention_chunks(X, H, d, dv, dims):
    """Float32-like precision although the operands are bfloat16 terms; cuts at and around tile and chunk borders."""
    T = 530
    case = ret_case(X, T, H, d, dv, dims, BF)
    for cuts in ([T], [255, 257, 2, 16], [128, 129, 1, 272], [1, 256, 273]):
        o, S = run_ret(X, case, H, d, dv, dims, cuts, 2)
        assert err(o, case[1][0]) < 2e-4, cuts
        assert err(S, case[1][1]) < 2e-4, cuts


@pytest.mark.parametrize("decay", [[1.0, 0.25], [0.999, 1e-3], [0.0, 0.5]])
def test_retention_extreme_decays(X, decay):
    case = ret_case(X, 300, 2, 16, 16, 16, BF, decay)
    for form in (1, 2):
        if form == 2 and min(decay) == 0:
            continue
        o, S = run_ret(X, case, 2, 16, 16, 16, [300], form)
        assert err(o, case[1][0]) < 2e-4 and err(S, case[1][1]) < 2e-4


def test_retention_far_key(X):
    """One key of the first tokens dominates with a decay of 1: it must reach every later chunk unchanged."""
    T, H, d = 700, 1, 32
    case = ret_case(X, T, H, d, 32, 0, BF, [1.0])
    q, k, v, table, decay = case[0]
    with torch.no_grad():
        k[3] *= 30
    shape = lambda t: npy(t).reshape(T, H, 32)                                            # noqa: E731
    want = O.retention(shape(q), shape(k) * d ** -0.5, shape(v), [1.0])
    o, S = run_ret(X, (case[0], None), H, d, 32, 0, [300, 400], 2)
    assert err(o, want[0]) < 2e-4 and err(S, want[1]) < 2e-4


@pytest.mark.parametrize("H,d,dv,dims", [(3, 16, 24, 8), (1, 6, 33, 4), (2, 64, 256, 64), (1, 8, 520, 0)])
def test_retention_steps(X, H, d, dv, dims):
    T = 9
    case = ret_case(X, T, H, d, dv, dims, F32)
    (q, k, v, table, decay), (o, S) = case
    g, state, got = rnd(41, T, H * dv), torch.zeros(H, d, dv).cuda(), []
    pos_dev = torch.zeros(1, dtype=torch.int32).cuda()
    for t in range(T):
        kw = dict(pos=t) if t % 2 else dict(pos_dev=pos_dev.fill_(t))
        got.append(X.retention_step(q[t], k[t], v[t], g[t], table, dims, d ** -0.5, decay, 1e-3, state, torch.empty(H * dv).cuda(), **kw))
    want = O.rms(o, 1e-3).reshape(T, H * dv) * O.silu(npy(g))
    assert err(torch.stack(got), want) < 3e-5 and err(state, S) < 2e-5


# ---- differential attention -------------------------------------------------------------------------------------------------

class Case:
    """Queries, and a cache with `cap` rows of which the first T are filled; stale rows hold large values."""

    def __init__(self, scmx, T, H, G, d, dv, dt, cap=None, seed=50):
        self.T, self.H, self.G, self.d, self.dv = T, H, G, d, dv
        self.scale, self.lam, self.diff, self.eps = 0.9 * d ** -0.5, 0.37, 0.45, 1e-4
        cap = cap or T + 40
        self.cache = scmx.host_model.KVCache(2 * G, d, cap, "cuda", dt, G, dv)
        self.cache.k.fill_(50.0)
        self.cache.v.fill_(float("nan"))
        self.q, self.k, self.v = rnd(seed, 2 * H, T, d, dtype=dt), rnd(seed + 1, 2 * G, T, d, dtype=dt), rnd(seed + 2, G, T, dv, dtype=dt)

    def fill(self):
        self.cache.k[:, :self.T], self.cache.v[:, :self.T] = self.k, self.v

    def want(self, rows):
        q, k, v = npy(self.q), npy(self.k), npy(self.v)
        out = np.zeros((len(rows), self.H, self.dv))
        for h in range(self.H):
            g = h // (self.H // self.G)
            a = []
            for m in range(2):
                s = (q[2 * h + m][rows] @ k[2 * g + m].T) * self.scale
                s = np.where(np.arange(self.T)[None] <= np.asarray(rows)[:, None], s, -np.inf)
                p = np.exp(s - s.max(1, keepdims=True))
                a.append(p / p.sum(1, keepdims=True) @ v[g])
            out[:, h] = O.differential(a[0], a[1], self.lam, self.diff, self.eps)
        return out.reshape(len(rows), self.H * self.dv)

    def prefill(self, X, lo, hi, form):
        self.cache.offset = lo
        o = X.diff_attention(self.q[:, lo:hi].contiguous(), self.cache, self.H, self.G, self.scale, self.lam, self.diff, self.eps, form)
        return o

    def decode(self, X, t, pos_dev=None):
        self.cache.offset = t if pos_dev is None else 0
        at = X.DiffDecodeAttention(self.H, self.G, self.d, self.dv, "cuda")
        return at(self.q[:, t].float().contiguous(), self.cache, self.scale, self.lam, self.diff, self.eps,
                  torch.empty(self.H * self.dv).cuda(), n_pos=None if pos_dev is not None else t + 1, pos_dev=pos_dev)


SIZES = [(2, 1, 8, 8), (4, 2, 32, 64), (3, 3, 64, 128), (2, 2, 72, 40), (2, 1, 128, 128), (4, 4, 16, 24)]


@pytest.mark.parametrize("H,G,d,dv", SIZES)
def test_attention_tensor_cores(X, scmx, H, G, d, dv):
    T = 400
    c = Case(scmx, T, H, G, d, dv, BF)
    c.fill()
    want = c.want(list(range(T)))
    for lo, hi in ((0, 400), (0, 1), (0, 128), (127, 130), (128, 400), (250, 400), (398, 400), (3, 390)):
        assert err(c.prefill(X, lo, hi, 2), want[lo:hi]) < 2.5e-2, (lo, hi)


@pytest.mark.parametrize("H,G,d,dv", SIZES + [(2, 1, 5, 7), (1, 1, 20, 200)])
@pytest.mark.parametrize("dt", [BF, F32])
def test_attention_cuda_cores(X, scmx, H, G, d, dv, dt):
    T = 90
    c = Case(scmx, T, H, G, d, dv, dt)
    c.fill()
    want = c.want(list(range(T)))
    for lo, hi in ((0, 90), (31, 34), (15, 17), (64, 90)):
        assert err(c.prefill(X, lo, hi, 1), want[lo:hi]) < (2.5e-2 if dt == BF else 3e-5), (lo, hi)


@pytest.mark.parametrize("H,G,d,dv", SIZES + [(2, 1, 5, 7), (16, 1, 24, 128), (6, 2, 128, 256), (36, 2, 16, 8)])
@pytest.mark.parametrize("dt", [BF, F32])
def test_attention_decode(X, scmx, H, G, d, dv, dt):
    T = 700
    c = Case(scmx, T, H, G, d, dv, dt)
    c.fill()
    rows = [0, 1, 62, 63, 64, 65, 127, 128, 511, 699]
    want = c.want(rows)
    pos_dev = torch.zeros(1, dtype=torch.int32).cuda()
    for i, t in enumerate(rows):
        assert err(c.decode(X, t), want[i]) < 3e-5, t
        assert err(c.decode(X, t, pos_dev.fill_(t)), want[i]) < 3e-5, t


def test_attention_single_keys_stand_out(X, scmx):
    """Each probed query meets one key with a score far above the rest - the first token, tile borders, its own position - so that a
    key that is missing, or one too many, changes the result completely."""
    T, H, G, d, dv = 700, 2, 1, 32, 64
    c = Case(scmx, T, H, G, d, dv, BF)
    pairs = [(5, 0), (127, 127), (128, 127), (129, 128), (300, 255), (300 + 84, 256), (511, 0), (600, 383), (640, 640), (699, 1)]
    for m in range(2):
        for t, j in pairs:
            c.q[m, t] = c.k[m, j] * 6 if m == 0 else -c.k[m, j] * 6
    c.fill()
    rows = [t for t, _ in pairs]
    want = c.want(rows)
    # the dominant key decides map 1
    assert np.abs(want).max() > 1
    full = c.prefill(X, 0, T, 2)[rows]
    assert err(full, want) < 2.5e-2
    late = c.prefill(X, 100, T, 2)
    assert err(late[[t - 100 for t in rows[1:]]], want[1:]) < 2.5e-2
    for i, t in enumerate(rows):
        assert err(c.decode(X, t), want[i]) < 1e-4, t
    # a key just beyond the query must not be seen: make the next key enormous
    c.cache.k[:, 301:, :] = 40.0
    assert err(c.prefill(X, 290, 301, 2)[10], want[4]) < 2.5e-2 and err(c.decode(X, 300), want[4]) < 1e-4


def test_attention_growing_scores(X, scmx):
    """Scores that keep rising along the keys: the running maximum has to be raised and the outputs rescaled at many tiles."""
    T, H, G, d, dv = 900, 1, 1, 16, 32
    c = Case(scmx, T, H, G, d, dv, BF)
    ramp = torch.linspace(0.2, 9.0, T).cuda()[:, None]
    for m in range(2):
        base = rnd(60 + m, d)
        c.q[m] = (base * 3).to(BF)
        c.k[m] = (base * ramp + 0.05 * rnd(62 + m, T, d)).to(BF)
    c.fill()
    rows = list(range(0, T, 37)) + [T - 1]
    want = c.want(rows)
    assert err(c.prefill(X, 0, T, 2)[rows], want) < 4e-2
    assert err(c.decode(X, T - 1), want[-1]) < 1e-3


@pytest.mark.parametrize("dt", [BF, F32])
def test_qk_norm_append(X, scmx, dt):
    T, H, G, d, dv, pos = 7, 3, 1, 20, 12, 5
    cache = scmx.host_model.KVCache(2 * G, d, 30, "cuda", dt, G, dv)
    cache.k.zero_(), cache.v.zero_()
    cache.offset = pos
    qkv = rnd(70, T, 2 * H * d + 2 * G * d + G * dv, dtype=dt)
    q, k, v = qkv.split([2 * H * d, 2 * G * d, G * dv], 1)
    qw, kw = rnd(71, d), rnd(72, d)
    tol = 2e-2 if dt == BF else 1e-5
    got = X.qk_norm_append(q, k, v, H, G, qw, kw, 1e-2, cache, dt)
    assert err(got, (O.rms(npy(q).reshape(T, 2 * H, d), 1e-2) * npy(qw)).transpose(1, 0, 2)) < tol
    assert err(cache.k[:, pos:pos + T], (O.rms(npy(k).reshape(T, 2 * G, d), 1e-2) * npy(kw)).transpose(1, 0, 2)) < tol
    assert torch.equal(cache.v[:, pos:pos + T], v.reshape(T, G, dv).transpose(0, 1))
    assert float(cache.k[:, :pos].float().abs().sum() + cache.k[:, pos + T:].float().abs().sum()) == 0.0
    # one row at a device-side position, float32 in
    X.qk_norm_append(q[:1].float(), k[:1].float(), v[:1].float(), H, G, qw, kw, 1e-2, cache, F32, torch.tensor([20], dtype=torch.int32).cuda())
    assert err(cache.k[:, 20], O.rms(npy(k[:1]).reshape(2 * G, d), 1e-2) * npy(kw)) < tol
    before = cache.k.clone()
    X.qk_norm_append(q[:1].float(), k[:1].float(), v[:1].float(), H, G, qw, kw, 1e-2, cache, F32, torch.tensor([30], dtype=torch.int32).cuda())
    assert torch.equal(before, cache.k)          # beyond the cache: dropped
