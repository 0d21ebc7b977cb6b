"""CPU: configuration, tensor names, shared layers, caches and bindings of the Fabezen decoders; the plain oracle against closed forms;
the argument checks the kernels make before a launch."""
import copy
import ctypes

import numpy as np
import pytest
import torch

import fabezen_oracle as O


def small_config():
    cd = {"type": "channel_delta", "mixer": {"heads": 2, "kv_heads": 1, "dim": 6, "vdim": 10, "conv": 3, "ranks": [4, 5]}, "mlp": None}
    return {"architecture": "Fabezen", "vocab": 40, "width": 24, "norm": {"eps": 1e-6}, "residual_mult": 0.5,
            "embedding": {"scale": 3.0, "bigram": {"buckets": 11, "mul_prev": 5, "mul_cur": 2}}, "layers": [
                {"type": "delta", "mixer": {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 12, "conv": 4}, "mlp": {"kind": "dense", "ff": 20}},
                cd, {**cd, "weights_of": 1},
                {"type": "latent_attention", "mixer": {"heads": 2, "dim": 6, "rot_dim": 4, "vdim": 8, "kv_rank": 13, "q_rank": 9, "scale": 0.3,
                                                       "mask": {"size": 7}, "rot": {"base": 100.0, "dims": 4}}, "mlp": None}]}


def test_arguments_are_checked_before_a_launch(scmx):
    lib, p = scmx._lib.mixers(), ctypes.c_void_p(256)
    assert lib.scmx_embed_pair(p, p, p, 0, 4, 4, 4, 1.0, 0, 1, 1, p, p, None) == -1            # a pair table without buckets
    assert lib.scmx_add_norm(p, 4, p, p, 1.0, 1e-5, 4, 8, p, p, 0, None) == -1                 # pitch below the width
    assert lib.scmx_head_norm_gate(p, p, 8, 0, p, 2, 4, 1, 8, 1e-5, p, None) == -1 and b"gate=2" in lib.scmx_last_error_string()
    assert lib.scmx_gated_gelu(p, 40, 4, 20, p, None) == -1
    assert lib.scmx_gemm_bf16(p, 16, p, 16, 4, 40, 16, 2, 0.0, 0.0, p, 0, 24, 0, 1, None, p, None) == -1     # columns in turns of 16
    assert lib.scmx_gemv_x(p, 16, 0, p, 40, 16, 3, 0.0, 0.0, None, None, None, 0, 0, p, None) == -1
    d = lambda H, G, dd, scratch=None, n=4: lib.scmx_delta(p, 64, p, 64, p, 64, p, 8, p, 8, 0, 0, n, H, G, dd, 8, p, p, p, p, scratch, 0, p, None)   # noqa: E731
    assert d(3, 2, 8) == -1 and d(2, 2, 300) == -5 and d(2, 2, 12, p) == -5 and d(2, 2, 8, p) == -1
    assert d(2, 2, 8, n=0) == 0
    assert lib.scmx_delta_scratch(100, 2, 12, 8, 64) == 0 and lib.scmx_delta_scratch(100, 2, 136, 8, 64) == 0
    assert lib.scmx_delta_scratch(65, 2, 16, 8, 64) > lib.scmx_delta_scratch(64, 2, 16, 8, 64) > 0
    assert lib.scmx_delta_step(p, p, p, p, p, p, p, 8, 4, None, 0, 0, 0, 2, 2, 8, 8, p, p, p, 1e-5, p, p, None) == -1    # one low-rank product
    assert lib.scmx_latent_append(p, 40, 0, 0, 0, 4, 8, 16, 3, p, p, p, 64, 1e-5, 0, None, p, 8, p, 24, 64, None) == -1    # odd rotated part
    assert lib.scmx_latent_append(p, 40, 0, 0, 0, 4, 8, 16, 4, p, p, p, 64, 1e-5, 61, None, p, 8, p, 24, 64, None) == -1
    assert b"cache of 64" in lib.scmx_last_error_string()
    assert lib.scmx_latent_rows(p, p, 24, 0, 1, 0, None, 64, 0, 2, 1040, 4, 1.0, 4, p, None) == -1
    assert lib.scmx_latent_rows(p, p, 1048, 0, 1, 0, None, 64, 0, 2, 1040, 4, 1.0, 4, p, None) == -5
    assert lib.scmx_latent_rows(p, p, 24, 0, 1, 0, None, 64, 0, 2, 16, 4, 1.0, 65, p, None) == -1
    la = lambda k0, dd=64, pos=100, window=50: lib.scmx_latent_attn(p, 512, p, 512, p, 128, 4, pos, k0, window, 2, dd, 8, 64, 1.0, p, p, None)   # noqa: E731
    assert la(52) == -1 and la(0, 12) == -5 and la(0, 136) == -5 and la(1, window=0) == -1


def test_config_and_tensor_names(scmx):
    HM = scmx.host_model
    cfg = small_config()
    a = HM.HybridArgs.from_config(cfg)
    assert (a.vocab_size, a.hidden_size, a.rms_norm_eps, len(a.layers), a.residual_mult, a.embed_scale) == (40, 24, 1e-6, 4, 0.5, 3.0)
    assert a.design.prenorm and a.design.tied and [a.source(i) for i in range(4)] == [0, 1, 1, 3]
    W = O.random_weights(cfg)
    sd = {k: torch.from_numpy(v) for k, v in W.items()}
    model = HM.HybridLM(a, "cpu", torch.float32).load_state_dict(sd)
    assert {k: v.shape for k, v in W.items()} == model.shapes(sd)
    assert not any(k.startswith("l2.") for k in model.w) and model.w["l1.mix.a2"].shape == (12, 4) and model.w["l1.mix.g2"].shape == (20, 5)
    assert model.w["bigram"].shape == (12, 24) and "head" not in model.w
    for name, other in (("l1.mix.a2", sd["l1.mix.a2"][:, :-1]), ("bigram", sd["bigram"][:-1]), ("l3.mix.dkv", sd["l3.mix.dkv"][:-1])):
        with pytest.raises(ValueError, match=name):
            HM.HybridLM(a, "cpu").load_state_dict({**sd, name: other})
    with pytest.raises(ValueError, match="l2.norm1"):
        HM.HybridLM(a, "cpu").load_state_dict({**sd, "l2.norm1": sd["l1.norm1"]})
    rnd = HM.HybridLM(a, "cpu", torch.float32).init_random(1, rank=3)
    assert rnd.w["l1.mix.a1"].shape == (3, 24)


@pytest.mark.parametrize("path,value,word", [
    (("layers", 0, "mixer", "kv_heads"), 3, "key/value"), (("layers", 1, "type"), "window", "mixer 'window'"), (("layers", 2, "weights_of"), 4, "weights of layer 4"),
    (("layers", 2, "weights_of"), 0, "differs"), (("layers", 2, "weights_of"), 2, "its own"), (("layers", 3, "mixer", "rot", "dims"), 2, "rotated"),
    (("layers", 0, "mlp", "kind"), "experts", "experts")])
def test_contradictions_are_refused(scmx, path, value, word):
    cfg = copy.deepcopy(small_config())
    e = cfg
    for k in path[:-1]:
        e = e[k]
    e[path[-1]] = value
    with pytest.raises(ValueError, match=word):
        scmx.host_model.HybridArgs.from_config(cfg)


def test_registry_and_caches(scmx):
    HM = scmx.host_model
    assert scmx.registry.architecture(small_config()) == "fabezen"
    model = HM.HybridLM(HM.HybridArgs.from_config(small_config()), "cpu", torch.bfloat16)
    c = HM.make_prompt_cache(model, 50)
    assert [type(x).__name__ for x in c] == ["StateCache", "StateCache", "StateCache", "LatentCache", "TokenCache"]
    assert c[0].tail.shape == (2 * 16 + 48, 3) and c[0].kv.shape == (4, 8, 12) and c[1].kv.data_ptr() != c[2].kv.data_ptr()
    assert c[3].c.shape == (50, 24) and c[3].c.dtype == torch.bfloat16 and int(c[4].prev) == -1
    assert [len(x.carried()) for x in c] == [2, 2, 2, 0, 1]
    pool = scmx.engine.CachePool(lambda n: HM.make_prompt_cache(model, n), 50)
    c = pool.acquire()
    c[4].prev.fill_(7)
    c[0].kv.fill_(1.0)
    for x in c:
        x.offset = 3
    pool.release(c)
    c = pool.acquire()
    assert int(c[4].prev) == -1 and float(c[0].kv.abs().sum()) == 0.0 and all(x.offset == 0 for x in c)


def test_gated_weights_are_interleaved(scmx):
    gate, up = torch.arange(20.0)[:, None].repeat(1, 3), -torch.arange(20.0)[:, None].repeat(1, 3) - 100
    w = scmx.sc_mixers.GatedGELU.weight(gate, up)
    assert w.shape == (64, 3)
    for i in range(20):
        assert w[32 * (i // 16) + i % 16, 0] == gate[i, 0] and w[32 * (i // 16) + 16 + i % 16, 0] == up[i, 0]
    assert float(w[36:48].abs().sum() + w[52:].abs().sum()) == 0.0


# ---- the oracle against closed forms --------------------------------------------------------------------------------------

def test_oracle_delta_rule():
    r = np.random.default_rng(1)
    T, H, G, d, dv = 12, 4, 2, 5, 3
    q, k, v = r.standard_normal((T, G, d)), O.unit(r.standard_normal((T, G, d))), r.standard_normal((T, H, dv))
    one, zero = np.ones((T, H, d)), np.zeros((T, H))
    # beta = 1 without decay: the key just written returns its value; orthogonal keys add up
    _, S = O.delta_rule(q, k, v, one, zero + 1)
    for h in range(H):
        assert np.allclose(S[h].T @ k[-1, h // 2], v[-1, h], atol=1e-4)
    e = np.eye(d)[:, None, :].repeat(G, 1)
    o, S = O.delta_rule(e, e, v[:d], one[:d], zero[:d] + 0.5)
    assert np.allclose(S, 0.5 * v[:d].transpose(1, 0, 2)) and np.allclose(o, 0.5 * v[:d])
    # beta = 0: only the decay acts, per row
    g = r.random((T, H, d))
    S0 = r.standard_normal((H, d, dv))
    _, S = O.delta_rule(q, k, v, g, zero, S0)
    assert np.allclose(S, g.prod(0)[:, :, None] * S0)
    # matrix form of one step
    S1 = O.delta_rule(q[:1], k[:1], v[:1], g[:1], zero[:1] + 0.3, S0)[1]
    for h in range(H):
        kk = k[0, h // 2][:, None]
        want = (np.eye(d) - 0.3 * kk @ kk.T) @ (g[0, h][:, None] * S0[h]) + 0.3 * kk @ v[0, h][None]
        assert np.allclose(S1[h], want)


def test_oracle_decay_and_conv():
    r = np.random.default_rng(2)
    A, a, b = r.standard_normal(3), r.standard_normal((4, 3)), r.standard_normal(3)
    assert np.allclose(np.exp(O.log_decay(A, a, b)), (1 + np.exp(a + b)) ** -np.exp(A))
    x, w = r.standard_normal((9, 2)), r.standard_normal((2, 4))
    y = np.stack([np.convolve(x[:, c], w[c, ::-1])[:9] for c in range(2)], 1)
    assert np.allclose(O.short_conv(x, w), y / (1 + np.exp(-y)))
    assert np.allclose((O.unit(x) ** 2).sum(-1), 1, atol=1e-4)


def test_oracle_rotation_and_window():
    r = np.random.default_rng(3)
    a, b = r.standard_normal((1, 1, 6)), r.standard_normal((1, 1, 6))
    dot = lambda i, j: (O.rotate_pairs(a, 300.0, 4, [i]) * O.rotate_pairs(b, 300.0, 4, [j])).sum()      # noqa: E731
    assert np.isclose(dot(9, 4), dot(105, 100)) and not np.isclose(dot(9, 4), dot(9, 5))
    z = O.rotate_pairs(a, 300.0, 4, [17])[0, 0]
    w = (a[0, 0, 0] + 1j * a[0, 0, 1]) * np.exp(17j)
    assert np.allclose(z[:2], [w.real, w.imag]) and np.array_equal(z[4:], a[0, 0, 4:])
    q, k, v = r.standard_normal((8, 4)), r.standard_normal((8, 4)), r.standard_normal((8, 3))
    i = np.arange(8)
    for size in (1, 3, 8, None):
        dist = i[:, None] - i[None]
        s = np.where((dist >= 0) & (dist < (size or 99)), q @ k.T * 0.7, -np.inf)
        p = np.exp(s - s.max(1, keepdims=True))
        assert np.allclose(O.window_attention(q, k, v, 0.7, size), p / p.sum(1, keepdims=True) @ v)


def test_oracle_embedding_and_gelu():
    r = np.random.default_rng(4)
    cfg, W = small_config(), {"embed": r.standard_normal((40, 6)), "bigram": r.standard_normal((12, 6))}
    x = O.embedding(W, cfg, [3, 39, 3])
    assert np.allclose(x[0], 3 * W["embed"][3] + W["bigram"][11])
    assert np.allclose(x[1], 3 * W["embed"][39] + W["bigram"][(3 * 5 + 39 * 2) % 11])
    assert np.allclose(x[2], 3 * W["embed"][3] + W["bigram"][(39 * 5 + 3 * 2) % 11])
    z = torch.linspace(-4, 4, 9, dtype=torch.float64)
    assert np.allclose(O.gelu_tanh(z.numpy()), torch.nn.functional.gelu(z, approximate="tanh").numpy())
