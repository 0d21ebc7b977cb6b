"""GPU: the kernels of gated delta rules, latent attention and pre-norm residuals against the plain float64 oracle: sizes on and off
the tiles' borders, carried states over portions, strong and weak decays, keys just inside and outside a window, far keys."""
import numpy as np
import pytest
import torch

import fabezen_oracle as O

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


# ---- embedding, residual, feed-forward, norms -------------------------------------------------------------------------------

@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("W,buckets,mp,mc", [(40, 17, 31, 5), (260, 1, 1, 1), (64, 1000, 2 ** 40 + 7, 2 ** 33 + 1)])
def test_embed_pair(X, dt, W, buckets, mp, mc):
    V = 50
    table, pairs = rnd(1, V, W, dtype=dt), rnd(2, buckets + 1, W, dtype=dt)
    ids = torch.randint(0, V, (29,), generator=torch.Generator().manual_seed(3))
    cfg = {"embedding": {"scale": 2.5, "bigram": {"buckets": buckets, "mul_prev": mp, "mul_cur": mc}}}
    want = O.embedding({"embed": npy(table), "bigram": npy(pairs)}, cfg, ids.tolist())
    prev = torch.full((1,), -1, dtype=torch.long, device="cuda")
    x, lo = torch.empty(29, W).cuda(), 0
    for n in (1, 1, 2, 20, 5):                     # the token before a portion is carried
        X.embed_pair(ids[lo:lo + n].cuda(), table, x[lo:lo + n], 2.5, pairs, (buckets, mp, mc), prev)
        lo += n
        assert int(prev) == int(ids[lo - 1])
    assert err(x, want) < 1e-6
    X.embed_pair(ids.cuda(), table, x, 0.5)
    assert err(x, 0.5 * npy(table)[ids]) < 1e-6


@pytest.mark.parametrize("T,W", [(1, 40), (1, 2048), (1, 8200), (3, 1030), (70, 516), (200, 33), (160, 4100)])
@pytest.mark.parametrize("dt,tol", [(BF, 6e-3), (F32, 2e-6)])
def test_add_norm(X, T, W, dt, tol):
    y, x, w = rnd(11, T, W), rnd(12, T, W), rnd(13, W)
    r = npy(x) + 0.3 * npy(y)
    h = torch.empty(T, W, dtype=dt).cuda()
    X.add_norm(None, x, w, 7.0, 1e-2, h)
    assert err(h, O.rms_norm(npy(x), npy(w), 1e-2)) < tol
    X.add_norm(y, x, w, 0.3, 1e-2, h)
    assert err(x, r) < 1e-6 and err(h, O.rms_norm(r, npy(w), 1e-2)) < tol


@pytest.mark.parametrize("T,C,taps", [(1, 24, 4), (40, 33, 3), (9, 130, 2), (17, 64, 1), (3, 10, 6), (2, 16, 4)])
@pytest.mark.parametrize("dt,tol", [(BF, 8e-3), (F32, 2e-6)])
def test_conv_without_bias(X, T, C, taps, dt, tol):
    x, w, tail = rnd(14, 2 * T, C, dtype=dt), rnd(15, C, taps), torch.zeros(C, taps - 1).cuda()
    got = torch.cat([X.conv_silu(x[:T], w, None, tail), X.conv_silu(x[T:], w, None, tail)])
    assert err(got, O.short_conv(npy(x), npy(w))) < tol
    lin, one = X.Linear(torch.eye(C, dtype=dt).cuda()), torch.zeros(C, taps - 1).cuda()
    step = torch.stack([lin.vec(r.float(), conv=(w, None, one)) for r in x])
    assert err(step, O.short_conv(npy(x), npy(w))) < 2e-6
    assert torch.allclose(one, tail, atol=1e-6)


@pytest.mark.parametrize("T,H,dv", [(3, 2, 8), (50, 3, 33), (4, 5, 128), (2, 1, 300)])
@pytest.mark.parametrize("dt,tol", [(BF, 8e-3), (F32, 2e-6)])
def test_head_norm_gate(X, T, H, dv, dt, tol):
    o, g, w = rnd(16, T, H, dv), rnd(17, T, H * dv, dtype=dt), rnd(18, dv)
    n = O.rms_norm(npy(o), npy(w), 1e-3).reshape(T, -1)
    assert err(X.head_norm_gate(o, g, 1e-3, w, 1), n * O.sigmoid(npy(g))) < tol
    assert err(X.head_norm_gate(o, g, 1e-3, w), n * O.silu(npy(g))) < tol
    assert err(X.head_norm_gate(o, g, 1e-3), O.rms_norm(npy(o), 1.0, 1e-3).reshape(T, -1) * O.silu(npy(g))) < tol


@pytest.mark.parametrize("M,ff,K,tile", [(1, 5, 16, 0), (70, 40, 100, 64), (200, 200, 264, 128), (300, 520, 192, 256), (257, 33, 72, 256), (130, 96, 64, 0)])
def test_gated_gelu(X, M, ff, K, tile):
    gate, up, x = rnd(19, ff, K, scale=2 * K ** -0.5, dtype=BF), rnd(20, ff, K, scale=K ** -0.5, dtype=BF), rnd(21, M, K, dtype=BF)
    act = X.GatedGELU()
    want = O.gelu_tanh(npy(x) @ npy(gate).T) * (npy(x) @ npy(up).T)
    lin = X.Linear(act.weight(gate, up))
    assert err(lin(x, F32, act=act, tile=tile)[:, :ff], want) < 3e-5
    assert err(lin(x, act=act, tile=tile)[:, :ff], want) < 1e-2
    assert err(lin.vec(x[0].float(), act=act)[:ff], want[0]) < 3e-5
    full = X.Linear(act.weight(gate.float(), up.float()))
    assert err(full(x.float(), act=act)[:, :ff], want) < 3e-5
    assert err(full.vec(x[0].float(), act=act)[:ff], want[0]) < 3e-5


# ---- gated delta rule -------------------------------------------------------------------------------------------------------

class DeltaCase:
    """Inputs as the kernels read them (after convolution and SiLU) and the oracle's outputs."""

    def __init__(self, X, T, H, G, d, dv, channel, dt, seed=0, strength=0.0, spread=1.0):
        self.X, self.H, self.d, self.dv, self.channel = X, H, d, dv, channel
        qkv = rnd(30 + seed, T, 2 * G * d + H * dv, dtype=dt)
        self.q, self.k, self.v = qkv.split([G * d, G * d, H * dv], 1)
        self.b = rnd(31 + seed, T, H, dtype=dt)
        n = H * d if channel else H
        self.a = rnd(32 + seed, T, n, scale=spread, dtype=F32 if channel else dt)
        self.nA, self.dtb = -torch.exp(rnd(33 + seed, H, scale=0.5) + strength), rnd(34 + seed, n) - 1.0
        self.state = torch.zeros(H, d, dv).cuda()

    def run(self, cuts, form, scmx=None):
        out, lo = [], 0
        for n in cuts:
            s = slice(lo, lo + n)
            out.append(self.X.delta(self.q[s], self.k[s], self.v[s], self.b[s], self.a[s], self.channel, self.nA, self.dtb, self.state, form))
            lo += n
        return torch.cat(out)

    def oracle(self, S=None):
        T, H, d, dv = self.q.shape[0], self.H, self.d, self.dv
        q = O.unit(npy(self.q).reshape(T, -1, d)) * d ** -0.5
        k = O.unit(npy(self.k).reshape(T, -1, d))
        shape = (H, d) if self.channel else (H,)
        z = O.softplus(npy(self.a).reshape(T, *shape) + npy(self.dtb).reshape(shape))
        g = np.exp(npy(self.nA)[:, None] * z if self.channel else npy(self.nA) * z)
        g = g if self.channel else g[:, :, None] * np.ones(d)
        return O.delta_rule(q, k, npy(self.v).reshape(T, H, dv), g, O.sigmoid(npy(self.b)), S)


@pytest.mark.parametrize("H,G,d,dv", [(2, 2, 16, 24), (4, 2, 48, 32), (3, 1, 5, 7), (2, 1, 128, 40), (1, 1, 200, 70), (6, 3, 24, 64)])
@pytest.mark.parametrize("channel", [False, True])
@pytest.mark.parametrize("dt", [BF, F32])
def test_delta_token_by_token(X, H, G, d, dv, channel, dt):
    for cuts in ([50], [1, 2, 8, 9, 30]):
        c = DeltaCase(X, 50, H, G, d, dv, channel, dt)
        o, S = c.oracle()
        assert err(c.run(cuts, 1), o) < 2e-5 and err(c.state, S) < 2e-5, cuts


@pytest.mark.parametrize("H,G,d,dv", [(2, 2, 64, 64), (4, 2, 128, 128), (3, 1, 24, 40), (2, 1, 128, 200), (2, 2, 64, 256), (6, 6, 8, 8)])
@pytest.mark.parametrize("channel", [False, True])
@pytest.mark.parametrize("cuts", [[64], [1], [150], [63, 65, 2, 70], [128, 129]])
def test_delta_chunks(X, H, G, d, dv, channel, cuts):
    c = DeltaCase(X, sum(cuts), H, G, d, dv, channel, BF, seed=1)
    o, S = c.oracle()
    assert err(c.run(cuts, 2), o) < 3e-4 and err(c.state, S) < 3e-4


@pytest.mark.parametrize("channel", [False, True])
@pytest.mark.parametrize("strength,spread", [(-6.0, 1.0), (2.0, 4.0), (4.0, 8.0)])
def test_delta_chunks_weak_and_strong_decays(X, channel, strength, spread):
    """Decays close to one (long memory) and down to exact zero within a token; every key equal to its neighbours' so that the
    corrections are large."""
    c = DeltaCase(X, 400, 2, 1, 64, 48, channel, BF, seed=2, strength=strength, spread=spread)
    c.k[1::2] = c.k[0::2]
    c.q[200:] = c.k[:200]
    o, S = c.oracle()
    assert err(c.run([400], 2), o) < 5e-4 and err(c.state, S) < 5e-4
    c.state.zero_()
    assert err(c.run([100, 300], 1), o) < 5e-5 and err(c.state, S) < 5e-5


@pytest.mark.parametrize("H,G,d,dv", [(2, 1, 64, 40), (1, 1, 128, 200), (3, 3, 40, 128), (16, 8, 16, 128), (32, 16, 8, 120)])
@pytest.mark.parametrize("channel", [False, True])
@pytest.mark.parametrize("cuts", [[1000], [530, 770]])
def test_delta_segments(X, H, G, d, dv, channel, cuts):
    """Long portions with few heads run as segments side by side, with a state carried in."""
    c = DeltaCase(X, sum(cuts), H, G, d, dv, channel, BF, seed=5, strength=-5.0)
    start = rnd(49, H, d, dv, scale=0.3)
    c.state.copy_(start)
    o, S = c.oracle(npy(start))
    assert err(c.run(cuts, 2), o) < 5e-4 and err(c.state, S) < 5e-4


def test_delta_far_value_is_read_back(X):
    """A value written once under its own key and asked for 700 tokens later, almost without decay."""
    for channel in (False, True):
        c = DeltaCase(X, 760, 1, 1, 64, 16, channel, BF, seed=3, strength=-14.0)
        c.b[:] = -8.0
        c.b[40] = 8.0
        c.v[40] *= 20
        c.q[740] = c.k[40]
        o, _ = c.oracle()
        for form in (1, 2):
            c.state.zero_()
            got = npy(c.run([760], form))
            assert np.abs(got[740] - o[740]).max() < 2e-3 * np.abs(o[740]).max()
            assert np.abs(o[740]).max() > 1.0


@pytest.mark.parametrize("H,G,d,dv,ra,rg", [(2, 1, 16, 24, 5, 9), (4, 4, 64, 72, 24, 40), (3, 3, 130, 100, 16, 40), (2, 2, 128, 300, 128, 64), (1, 1, 7, 5, 1, 1)])
@pytest.mark.parametrize("channel", [False, True])
@pytest.mark.parametrize("dt", [BF, F32])
def test_delta_step(X, H, G, d, dv, ra, rg, channel, dt):
    T, eps = 6, 1e-3
    c = DeltaCase(X, T, H, G, d, dv, channel, F32, seed=4)
    w = rnd(40, dv)
    wa = wg = None
    if channel:
        wa, wg = X.Linear(rnd(41, H * d, ra, scale=ra ** -0.5, dtype=dt)), X.Linear(rnd(42, H * dv, rg, scale=rg ** -0.5, dtype=dt))
        a, g = rnd(43, T, ra), rnd(44, T, rg)
        c.a = torch.from_numpy(npy(a) @ npy(wa.w[:, :ra]).T).float().cuda()
        gate = O.sigmoid(npy(g) @ npy(wg.w[:, :rg]).T)
    else:
        a, g = c.a, rnd(45, T, H * dv)
        gate = O.silu(npy(g))
    start = rnd(46, H, d, dv, scale=0.3)
    o, S = c.oracle(npy(start))
    state, y = start.clone(), torch.empty(T, H * dv).cuda()
    for t in range(T):
        X.delta_step(c.q[t].contiguous(), c.k[t].contiguous(), c.v[t].contiguous(), c.b[t], a[t], g[t], wa, wg, c.nA, c.dtb, w, eps, state, y[t])
    assert err(y, O.rms_norm(o, npy(w), eps).reshape(T, -1) * gate) < 5e-5 and err(state, S) < 2e-5


# ---- latent attention -------------------------------------------------------------------------------------------------------

class LatentCase:
    def __init__(self, scmx, T, H, d, r, dv, R, window, dt, seed=0, Q=12, capacity=None):
        self.X, self.sizes = scmx.sc_mixers, (H, d, r, dv, R)
        self.window, self.scale, self.dt, self.Q = window, (d + r) ** -0.5, dt, Q
        self.y = rnd(50 + seed, T, Q + R + r, dtype=dt)
        self.qw, self.cw = rnd(51 + seed, Q), rnd(52 + seed, R)
        self.q = rnd(53 + seed, T, H * (d + r), scale=2.0, dtype=dt)
        self.wuk, self.wuv = rnd(54 + seed, H * d, R, scale=R ** -0.5, dtype=dt), rnd(55 + seed, H * dv, R, scale=R ** -0.5, dtype=dt)
        self.cs = self.X.rotary_table(500.0, r, 1024, "cuda")
        self.cache = scmx.host_model.LatentCache(R, r, capacity or T, "cuda", dt)
        self.lin = self.X.Linear(torch.cat([self.wuk, self.wuv]))

    def append(self, lo, n):
        H, d, r, dv, R = self.sizes
        self.cache.offset = lo
        return self.X.latent_append(self.y[lo:lo + n], self.Q, R, r, self.qw, self.cw, self.cs, 1e-3, self.cache, self.dt)

    def attend(self, lo, n, tc, out=None):
        H, d, r, dv, R = self.sizes
        self.cache.offset = lo
        q = self.q[lo:lo + n].clone()
        if tc:
            return self.X.latent_prompt(q, self.lin, self.cs, self.cache, H, d, r, dv, R, self.window, self.scale)
        return self.X.latent_rows(q, self.lin.rows(0, H * d), self.lin.rows(H * d, H * (d + dv)), self.cs, self.cache, H, d, r, dv, self.window, self.scale,
                                  out or self.dt)

    def oracle(self):
        """From the cached latents (as stored): attention outputs [T, H dv]."""
        H, d, r, dv, R = self.sizes
        T = self.q.shape[0]
        c, kr = npy(self.cache.c[:T, :R]), npy(self.cache.c[:T, (R + 7) // 8 * 8:][:, :r])
        q = npy(self.q).reshape(T, H, d + r)
        qr = O.rotate_pairs(q[..., d:], 500.0, r, range(T))
        k, v = (c @ npy(self.wuk).T).reshape(T, H, d), (c @ npy(self.wuv).T).reshape(T, H, dv)
        return np.concatenate([O.window_attention(np.concatenate([q[:, i, :d], qr[:, i]], 1), np.concatenate([k[:, i], kr], 1), v[:, i], self.scale,
                                                  self.window or None) for i in range(H)], 1)


@pytest.mark.parametrize("Q,R,r", [(12, 20, 6), (80, 104, 24), (7, 13, 0), (300, 512, 64), (1536, 512, 64)])
@pytest.mark.parametrize("dt,tol", [(BF, 1e-2), (F32, 3e-6)])
def test_latent_append(scmx, Q, R, r, dt, tol):
    c = LatentCase(scmx, 30, 1, 8, r, 8, R, 0, dt, Q=Q, capacity=33)
    cq = torch.cat([c.append(0, 17), c.append(17, 13)])
    y = npy(c.y)
    assert err(cq, O.rms_norm(y[:, :Q], npy(c.qw), 1e-3)) < tol
    assert err(c.cache.c[:30, :R], O.rms_norm(y[:, Q:Q + R], npy(c.cw), 1e-3)) < tol
    up = (R + 7) // 8 * 8
    if r:
        assert err(c.cache.c[:30, up:up + r], O.rotate_pairs(y[:, Q + R:], 500.0, r, range(30))) < tol
    assert float(c.cache.c[:, R:up].abs().sum()) == 0.0 and float(c.cache.c[:, up + r:].abs().sum()) == 0.0 and float(c.cache.c[30:].abs().sum()) == 0.0


@pytest.mark.parametrize("H,d,r,dv,R", [(1, 8, 2, 8, 12), (4, 72, 24, 56, 88), (3, 10, 6, 14, 21), (6, 24, 0, 16, 40), (20, 16, 8, 24, 64), (2, 32, 16, 40, 700),
                                        (18, 8, 2, 8, 600)])
@pytest.mark.parametrize("window", [0, 1, 33, 70])
@pytest.mark.parametrize("dt,tol", [(BF, 1.5e-2), (F32, 1e-5)])
def test_latent_rows(scmx, H, d, r, dv, R, window, dt, tol):
    T = 110
    c = LatentCase(scmx, T, H, d, r, dv, R, window, dt)
    c.append(0, T)
    want = c.oracle()
    assert err(torch.cat([c.attend(0, 1, False), c.attend(1, 3, False), c.attend(4, T - 5, False), c.attend(T - 1, 1, False)]), want) < tol


@pytest.mark.parametrize("H,d,r,dv,R", [(2, 56, 40, 64, 80), (3, 128, 64, 128, 64), (1, 24, 8, 40, 16), (2, 40, 0, 24, 32), (2, 96, 16, 128, 48), (2, 128, 0, 72, 40)])
@pytest.mark.parametrize("window", [0, 1, 40, 128, 129, 300])
def test_latent_prompt(scmx, H, d, r, dv, R, window):
    T = 420
    c = LatentCase(scmx, T, H, d, r, dv, R, window, BF, seed=1)
    c.append(0, T)
    want = c.oracle()
    for cuts in ([T], [33, 256, 131], [255, 2, 163]):
        got, lo = [], 0
        for n in cuts:
            got.append(c.attend(lo, n, True))
            lo += n
        assert err(torch.cat(got), want) < 2.5e-2, cuts


@pytest.mark.parametrize("tc", [False, True])
@pytest.mark.parametrize("window", [50, 128, 200])
def test_latent_window_edges(scmx, tc, window):
    """One key that outweighs all others: it decides every row that sees it, and no row beyond the window."""
    H, d, r, dv, R, T, at = 2, 32, 8, 16, 24, 400, 90
    c = LatentCase(scmx, T, H, d, r, dv, R, window, BF, seed=2)
    c.append(0, T)
    c.cache.c[at, :R] *= 6                        # a long latent along every query
    kh = npy(c.cache.c[at, :R]) @ npy(c.wuk).T
    for h in range(H):
        c.q[:, h * (d + r):h * (d + r) + d] = torch.from_numpy(kh[h * d:(h + 1) * d] * 0.5).to(BF).cuda()
    want = c.oracle()
    got = npy(c.attend(0, T, tc))
    assert np.abs(got - want).max() < 0.03 * np.abs(want).max()
    v = npy(c.cache.c[at, :R]) @ npy(c.wuv).T
    near = [at, at + 1, at + window - 1]
    assert np.abs(got[near] - v).max() < 0.05 * np.abs(v).max()                       # just inside: that value alone
    assert all(np.abs(got[t] - v).max() > 0.3 * np.abs(v).max() for t in (at - 1, at + window, at + window + 1))
    rows = torch.cat([c.attend(t, 1, False) for t in near + [at + window]])
    assert np.abs(npy(rows) - want[near + [at + window]]).max() < 0.03 * np.abs(want).max()


def test_latent_position_on_the_device(scmx):
    """A device-side position replaces the host's and the cache's borders hold."""
    H, d, r, dv, R, T = 2, 16, 4, 8, 20, 70
    c = LatentCase(scmx, T, H, d, r, dv, R, 30, F32, seed=3)
    c.append(0, T)
    X, host = scmx.sc_mixers, c.attend(65, 1, False)
    pos = torch.tensor([65], dtype=torch.int32, device="cuda")
    c.cache.offset = 0
    dev = X.latent_rows(c.q[65:66], c.lin.rows(0, H * d), c.lin.rows(H * d, H * (d + dv)), c.cs, c.cache, H, d, r, dv, 30, c.scale, F32, pos)
    assert torch.equal(host, dev)
    before = c.cache.c.clone()
    pos.fill_(T)                                   # past the end: the row is dropped
    X.latent_append(c.y[:1], c.Q, R, r, c.qw, c.cw, c.cs, 1e-3, c.cache, F32, pos)
    assert torch.equal(before, c.cache.c)
