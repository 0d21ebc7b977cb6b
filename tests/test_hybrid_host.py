"""CPU: configuration, tensor names, registry and bindings of the hybrid decoders; the plain oracle against closed forms; the
argument checks the mixer kernels make before a launch."""
import ctypes
import json
import os
import re

import numpy as np
import pytest
import torch

import hybrid_oracle as O

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def small_config():
    return {"architecture": "Sebesun", "vocab": 40, "width": 24, "norm": {"eps": 1e-6}, "layers": [
        {"type": "retention", "mixer": {"heads": 2, "dim": 8, "vdim": 12, "decay": [0.9, 0.75], "rot": {"base": 500.0, "dims": 4}},
         "mlp": {"kind": "dense", "ff": 20}},
        {"type": "mamba1", "mixer": {"inner": 28, "state": 5, "dt_rank": 3, "conv": 4}, "mlp": None},
        {"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 10, "scale": 0.3, "diff": 0.55}, "mlp": None}]}


def test_binding_matches_header(scmx):
    hdr = open(os.path.join(ROOT, "include", "scmx_mixers.h")).read()
    declared = set(re.findall(r"^(?:int|int64_t) (scmx_[a-z0-9_]+)\s*\(", hdr, re.M))
    assert declared == set(scmx._lib.MIXER_SIGNATURES) - {"scmx_last_error_string"}
    h = ctypes.CDLL(scmx._lib.MIXERS_PATH)
    assert all(hasattr(h, n) for n in declared)


def test_arguments_are_checked_before_a_launch(scmx):
    lib, p = scmx._lib.mixers(), ctypes.c_void_p(256)
    assert lib.scmx_embed(p, p, 2, 4, 4, 4, p, None, None) == -1 and b"dtype" in lib.scmx_last_error_string()
    assert lib.scmx_conv_silu(p, 8, 0, 4, 8, 4, p, p, None, p, 8, None) == -1              # taps without the carried inputs
    assert lib.scmx_selective_scan(p, 8, p, 8, p, 600, p, 8, 0, 4, 8, 300, p, p, p, p, p, 8, None) == -5
    assert lib.scmx_retention(p, 8, p, 8, p, 8, 0, 4, 1, 8, 8, p, 3, 1.0, p, p, p, None, 0, p, None) == -1   # odd rotation
    assert lib.scmx_retention_step(p, p, p, p, 1, 8, 8, p, 16, 8, 16, None, 1.0, p, 1e-5, p, p, None) == -1  # beyond the table
    assert lib.scmx_qk_norm_append(p, 8, p, 8, p, 8, 0, 0, 0, 4, 1, 1, 8, 8, p, p, 1e-5, 5, None, p, p, p, 8, None) == -1
    assert b"cache of 8" in lib.scmx_last_error_string()
    assert lib.scmx_diff_attn(p, p, p, 0, 4, 0, 8, 3, 2, 8, 8, 1.0, 0.5, 0.5, 1e-5, p, 0, p, None) == -1     # 3 heads over 2
    assert lib.scmx_diff_attn(p, p, p, 1, 4, 0, 8, 2, 2, 8, 8, 1.0, 0.5, 0.5, 1e-5, p, 2, p, None) == -5     # float32 on tensor cores
    assert lib.scmx_diff_decode(p, p, p, 0, 9, None, 8, 2, 2, 8, 8, 1.0, 0.5, 0.5, 1e-5, 4, p, p, p, None) == -1
    assert lib.scmx_gemm_bf16(p, 12, p, 16, 4, 8, 12, 0, 0.0, 0.0, p, 0, 8, 0, 1, None, p, None) == -1       # row pitch
    assert lib.scmx_gemm_bf16(p, 16, p, 16, 4, 8, 12, 0, 0.0, 0.0, p, 0, 8, 0, 2, p, p, None) == -1       # two ranges of one block
    assert lib.scmx_gemv_x(p, 12, 0, p, 4, 12, 0, 0.0, 0.0, None, None, None, 0, 0, p, None) == -1
    assert lib.scmx_retention_scratch(256, 2, 20, 64, 0, 128) == 0 and lib.scmx_retention_scratch(256, 2, 64, 64, 0, 128) > 0


def test_config_and_tensor_names(scmx):
    HM = scmx.host_model
    a = HM.HybridArgs.from_config(small_config())
    assert (a.vocab_size, a.hidden_size, a.rms_norm_eps, len(a.layers)) == (40, 24, 1e-6, 3)
    shapes = HM.HybridLM(a, "cpu", torch.float32).shapes()
    W = O.random_weights(small_config())
    assert {k: v.shape for k, v in W.items()} == shapes
    assert shapes["l0.mix.q"] == (16, 24) and shapes["l0.mix.g"] == (24, 24) and shapes["l2.mix.q"] == (48, 24) and shapes["l2.dwa"] == (4,)
    model = HM.HybridLM(a, "cpu", torch.float32).load_state_dict({k: torch.from_numpy(v) for k, v in W.items()})
    assert torch.equal(model.w["l1.mix.A_log"], torch.from_numpy(W["l1.mix.A_log"]))
    sd = {k: torch.from_numpy(v) for k, v in W.items()}
    sd.pop("l1.mix.D")
    with pytest.raises(ValueError, match="l1.mix.D"):
        HM.HybridLM(a, "cpu").load_state_dict(sd)
    sd = {k: torch.from_numpy(v) for k, v in W.items()}
    sd["head"] = sd["head"][:, :-1]
    with pytest.raises(ValueError, match="head"):
        HM.HybridLM(a, "cpu").load_state_dict(sd)


@pytest.mark.parametrize("change,word", [(("type", "window"), "mixer 'window'"), (("mlp", {"kind": "experts", "ff": 4}), "experts")])
def test_unknown_layers_are_refused(scmx, change, word):
    cfg = small_config()
    cfg["layers"][1][change[0]] = change[1]
    with pytest.raises(ValueError, match=word):
        scmx.host_model.HybridArgs.from_config(cfg)


def test_head_counts_are_checked(scmx):
    cfg = small_config()
    cfg["layers"][0]["mixer"]["decay"] = [0.9]
    with pytest.raises(ValueError, match="decays"):
        scmx.host_model.HybridArgs.from_config(cfg)
    cfg = small_config()
    cfg["layers"][2]["mixer"]["kv_heads"] = 3
    with pytest.raises(ValueError, match="key/value"):
        scmx.host_model.HybridArgs.from_config(cfg)


def test_registry_names(scmx, tmp_path):
    R = scmx.registry
    assert R.architecture(small_config()) == "sebesun" and R.architecture({"model_type": "qwen3"}) == "qwen3"
    with pytest.raises(KeyError, match="nosuch"):
        R.architecture({"architecture": "NoSuch"})
    (tmp_path / "config.json").write_text(json.dumps({"model_type": "qwen3"}))
    with pytest.raises(R.UnsupportedType):
        R.load(str(tmp_path), torch.float32)


def test_caches_and_pool(scmx):
    HM = scmx.host_model
    model = HM.HybridLM(HM.HybridArgs.from_config(small_config()), "cpu", torch.bfloat16)
    made = []

    def make(capacity):
        made.append(HM.make_prompt_cache(model, capacity))
        return made[-1]

    pool = scmx.engine.CachePool(make, 50)
    c = pool.acquire()
    assert [type(x).__name__ for x in c] == ["StateCache", "StateCache", "KVCache"]
    assert c[0].kv.shape == (2, 8, 12) and c[1].tail.shape == (28, 3) and c[1].ssm.shape == (28, 5)
    assert c[2].k.shape == (4, 50, 6) and c[2].v.shape == (2, 50, 10) and c[2].k.dtype == torch.bfloat16
    assert [len(x.carried()) for x in c] == [1, 2, 0]
    c[0].kv.fill_(3.0)
    c[1].ssm.fill_(1.0)
    for x in c:
        x.offset = 7
    pool.release(c)
    d = pool.acquire()
    assert d is c and len(made) == 1 and all(x.offset == 0 for x in d) and float(d[0].kv.abs().sum() + d[1].ssm.abs().sum()) == 0.0
    assert pool.acquire() is not d and len(made) == 2


# ---- the oracle against closed forms --------------------------------------------------------------------------------------

def test_oracle_retention_equals_its_quadratic_form():
    r = np.random.default_rng(1)
    T, H, d, dv = 20, 2, 5, 7
    q, k, v, dec = r.standard_normal((T, H, d)), r.standard_normal((T, H, d)), r.standard_normal((T, H, dv)), [0.8, 0.97]
    o, S = O.retention(q, k, v, dec)
    for h in range(H):
        i = np.arange(T)
        D = np.where(i[:, None] >= i[None], dec[h] ** np.maximum(i[:, None] - i[None], 0), 0.0)
        assert np.allclose(((q[:, h] @ k[:, h].T) * D) @ v[:, h], o[:, h])
        assert np.allclose(S[h], sum(dec[h] ** (T - 1 - t) * np.outer(k[t, h], v[t, h]) for t in range(T)))


def test_oracle_scan_conv_and_activations():
    r = np.random.default_rng(2)
    T, C, N = 15, 3, 4
    x, dt = r.standard_normal((T, C)), r.random((T, C))
    A, B, Cc, D = r.standard_normal((C, N)), r.standard_normal((T, N)), r.standard_normal((T, N)), r.standard_normal(C)
    y, _ = O.selective_scan(x, dt, A, B, Cc, D)
    for c in range(C):
        for t in range(T):
            s = sum(np.exp(-np.exp(A[c]) * dt[u + 1:t + 1, c].sum()) * dt[u, c] * x[u, c] * B[u] for u in range(t + 1))
            assert np.isclose(y[t, c], s @ Cc[t] + D[c] * x[t, c])
    w, b = r.standard_normal((C, 3)), r.standard_normal(C)
    full = np.stack([np.convolve(x[:, c], w[c, ::-1])[:T] for c in range(C)], 1) + b
    assert np.allclose(O.causal_conv(x, w, b), full)
    z = np.array([-3.0, -1e-4, 0.0, 2.0])
    sp = lambda v: np.log1p(np.exp(v))                                                   # noqa: E731
    want = [(0.5 + sp(0.7)) * (np.exp(v) - 1 - v) + v / 2 if v <= 0 else sp(-0.4) * v * v + v / 2 for v in z]
    assert np.allclose(O.xielu(z, -0.4, 0.7), want)


def test_oracle_rotation_preserves_relative_positions():
    r = np.random.default_rng(3)
    a, b = r.standard_normal((1, 1, 10)), r.standard_normal((1, 1, 10))
    dot = lambda i, j: (O.rotate_half(a, 300.0, 6, [i]) * O.rotate_half(b, 300.0, 6, [j])).sum()      # noqa: E731
    assert np.isclose(dot(9, 4), dot(105, 100)) and not np.isclose(dot(9, 4), dot(9, 5))
    assert np.array_equal(O.rotate_half(a, 300.0, 6, [17])[..., 6:], a[..., 6:])


def test_oracle_attention_maps():
    r = np.random.default_rng(4)
    q, k, v = r.standard_normal((6, 4)), r.standard_normal((6, 4)), r.standard_normal((6, 3))
    s = np.where(np.tri(6) > 0, q @ k.T * 0.7, -np.inf)
    p = np.exp(s - s.max(1, keepdims=True))
    assert np.allclose(O.causal_attention(q, k, v, 0.7), p / p.sum(1, keepdims=True) @ v)
    o = O.differential(r.standard_normal((6, 8)), r.standard_normal((6, 8)), 0.4, 0.3, 0.0)
    assert np.allclose(np.sqrt((o * o).mean(-1)), 0.7)
