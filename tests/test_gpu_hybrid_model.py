"""GPU: whole hybrid decoders against the plain float64 oracle, through the framework's prefill, decode, engine, registry and
command line: portions, token by token, requests among others, caches used again, long decoding, greedy generation."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import hybrid_oracle as O

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BF, F32 = torch.bfloat16, torch.float32


def ret(heads, dim, vdim, dims, decay, base=300.0):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay, "rot": {"base": base, "dims": dims}}}


def mam(inner, state, rank, conv):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": rank, "conv": conv}}


def att(heads, kv, dim, vdim, scale, diff):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}}


def config(vocab, width, eps, *layers):
    return {"architecture": "Sebesun", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": [{**ly, "mlp": {"kind": "dense", "ff": ff} if ff else None} for ly, ff in layers]}


CONFIGS = {
    "mixed": config(96, 64, 1e-5, (att(4, 2, 16, 24, 0.31, 0.2), None), (mam(80, 7, 5, 4), 48), (ret(3, 24, 40, 8, [0.6, 0.95, 0.999]), 72),
                    (att(2, 1, 40, 16, 0.12, 0.65), 56), (mam(48, 16, 8, 2), None)),
    "odd": config(51, 36, 1e-3, (ret(2, 6, 10, 4, [0.5, 1.0]), 20), (att(3, 1, 5, 7, 0.5, 0.4), 28), (mam(33, 3, 2, 1), 12)),
    "attention": config(64, 128, 1e-6, (att(2, 2, 64, 128, 0.125, 0.8), 96), (att(6, 2, 32, 64, 0.2, 0.05), None)),
    "recurrent": config(80, 96, 1e-5, (mam(192, 24, 6, 3), 64), (ret(4, 16, 64, 16, [0.9, 0.99, 0.7, 0.97], 10000.0), None), (ret(1, 128, 136, 64, [0.98]), None)),
    "one": config(33, 16, 1e-2, (mam(16, 1, 1, 5), 8)),
}


class Model:
    def __init__(self, scmx, cfg, dtype, capacity, seed=0):
        self.cfg = cfg
        HM = scmx.host_model
        self.W = {k: torch.from_numpy(v).to(dtype) for k, v in O.random_weights(cfg, seed, sharp=2.0).items()}
        model = HM.HybridLM(HM.HybridArgs.from_config(cfg), "cuda", dtype).load_state_dict(self.W)
        self.fused = scmx.fused_hybrid.FusedHybrid(model)
        self.decode = scmx.decode.DecodeHybrid(self.fused)
        self.bundle = scmx.registry.Bundle("hybrid", self.fused, self.decode, cfg["vocab"], scmx._lib.check_mixer_status)
        self.engine = scmx.engine.Engine(self.bundle, capacity)

    def oracle(self, tokens):
        return O.forward(self.cfg, {k: v.double().numpy() for k, v in self.W.items()}, tokens)[0]

    def run(self, tokens, cuts, rid="r", end=True):
        """Every position's logits with the sequence fed in portions of the given sizes."""
        out, lo = [], 0
        for n in cuts:
            part = tokens[lo:lo + n]
            lo += n
            out += self.engine.step([(rid, part, list(range(len(part))))], [rid] if end and lo == len(tokens) else [])
        return torch.cat(out).double().cpu().numpy()


def tokens(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def worst(got, want):
    """Largest root-mean-square difference of a position's logits, over the logits' own scale."""
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    return float(np.sqrt((d ** 2).mean(-1)).max() / want.std())


@pytest.fixture(autouse=True)
def _no_wait_ran_out(scmx):
    yield
    torch.cuda.synchronize()
    scmx._lib.check_mixer_status()


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("dtype,tol", [(F32, 2e-4), (BF, 8e-2)])
def test_prefill_portions_and_single_tokens(scmx, name, dtype, tol):
    cfg = CONFIGS[name]
    m, T = Model(scmx, cfg, dtype, 200), 150
    ids = tokens(cfg, T)
    want = m.oracle(ids)
    for cuts in ([T], [1] * T, [2] * 75, [63, 2, 1, 64, 20], [128, 22], [3, 100, 1, 1, 45]):
        e = worst(m.run(ids, cuts), want)
        assert e < tol, (cuts[:5], e)
    assert len(m.engine.pool.free) == 1            # one request at a time: one cache, used again


@pytest.mark.parametrize("dtype", [F32, BF])
def test_cuts_change_only_rounding(scmx, dtype):
    """Long sequence over retention chunks (256), attention tiles (128) and decode tiles (64); float32 agrees to rounding."""
    cfg = CONFIGS["mixed"]
    m, T = Model(scmx, cfg, dtype, 700), 640
    ids = tokens(cfg, T, 3)
    whole = m.run(ids, [T])
    for cuts in ([255, 2, 127, 129, 127], [300, 340], [513, 127], [600] + [1] * 40):
        assert worst(m.run(ids, cuts), whole) < (1e-4 if dtype == F32 else 8e-2), cuts


def test_long_decoding(scmx):
    cfg = CONFIGS["recurrent"]
    m, T = Model(scmx, cfg, F32, 500), 400
    ids = tokens(cfg, T, 4)
    assert worst(m.run(ids, [20] + [1] * 380), m.oracle(ids)) < 3e-4


def test_requests_among_others(scmx):
    """Interleaved requests of unequal lengths equal each alone; a finished request's cache serves the next without a trace of it."""
    cfg = CONFIGS["mixed"]
    m = Model(scmx, cfg, F32, 120)
    lens = {"a": 90, "b": 7, "c": 33}
    ids = {r: tokens(cfg, n, ord(r)) for r, n in lens.items()}
    alone = {r: m.run(t, [len(t)]) for r, t in ids.items()}
    pos, got = {r: 0 for r in ids}, {r: [] for r in ids}
    sizes = iter([5, 1, 11, 1, 1, 16, 2, 20, 3, 1, 30, 1, 8, 1, 40, 9] * 10)
    while any(pos[r] < lens[r] for r in ids):
        entries, end = [], []
        for r in ids:
            n = min(next(sizes), lens[r] - pos[r])
            if n:
                entries.append((r, ids[r][pos[r]:pos[r] + n], list(range(n))))
                pos[r] += n
                if pos[r] == lens[r]:
                    end.append(r)
        for (r, _, _), o in zip(entries, m.engine.step(entries, end)):
            got[r].append(o)
    for r in ids:
        assert worst(torch.cat(got[r]).double().cpu().numpy(), alone[r]) < 1e-4, r
    assert not m.engine.live and len(m.engine.pool.free) == 3
    for r in ids:                                  # all three caches once more
        m.engine.step([(r + "2", ids[r][:4], [])])
    for r in reversed(ids):
        assert worst(m.run(ids[r], [lens[r]], rid=r + "3"), alone[r]) < 1e-4


def test_wanted_places(scmx):
    cfg = CONFIGS["odd"]
    m = Model(scmx, cfg, F32, 40)
    ids = tokens(cfg, 12, 5)
    every = m.run(ids, [12])
    out = m.engine.step([("x", ids[:8], [6, 0, 3]), ("y", ids[:1], []), ("z", ids[:1], [0])])
    assert out[1] is None and np.allclose(out[0].cpu().numpy(), every[[6, 0, 3]], atol=1e-4)
    assert np.allclose(out[2].cpu().numpy(), every[:1], atol=1e-4)
    assert m.engine.step([("x", ids[8:12], [])])[0] is None and m.engine.live["x"][0].offset == 12
    with pytest.raises(AssertionError, match="capacity"):
        m.engine.step([("x", ids * 4, [])])


@pytest.mark.parametrize("name", ["mixed", "recurrent", "attention"])
@pytest.mark.parametrize("dtype", [F32, BF])
def test_greedy_generation(scmx, name, dtype):
    """Engine.generate (prompt in one step, then the captured graph): the continuation is the oracle's argmax at every position
    where the oracle's choice is clear, and a second request from the same engine repeats it."""
    cfg = CONFIGS[name]
    m, n = Model(scmx, cfg, dtype, 90), 40
    prompt = tokens(cfg, 30, 6)
    out = m.engine.generate(prompt, n)
    assert len(out) == n
    want = m.oracle(prompt + out)[len(prompt) - 1:-1]
    top = np.sort(want, -1)
    clear = top[:, -1] - top[:, -2] > (1e-3 if dtype == F32 else 0.3) * want.std()
    assert clear.sum() > n // 5 and (np.asarray(out)[clear] == want.argmax(-1)[clear]).all()
    assert m.engine.generate(prompt, n) == out
    stepped, lg = [], m.engine.step([("s", prompt, [29])])[0]
    for _ in range(n):                             # the same through single steps without the graph
        stepped.append(int(lg[0].argmax()))
        lg = m.engine.step([("s", [stepped[-1]], [0])])[0]
    assert stepped == out


def test_far_token_reaches_the_end(scmx):
    """Two prompts that differ in their first token only: the difference of the last position's logits equals the oracle's."""
    cfg = CONFIGS["attention"]
    m, T = Model(scmx, cfg, F32, 400), 300
    a = tokens(cfg, T, 7)
    b = [(a[0] + 1) % cfg["vocab"]] + a[1:]
    got = [m.run(x, [200, 99, 1])[-1] for x in (a, b)]
    want = [m.oracle(x)[-1] for x in (a, b)]
    delta = want[0] - want[1]
    assert np.abs(delta).max() > 1e-3 and np.abs(got[0] - got[1] - delta).max() < 0.05 * np.abs(delta).max() + 2e-4


def test_long_prompt_is_cut_into_portions(scmx):
    cfg = CONFIGS["mixed"]
    m = Model(scmx, cfg, F32, 300)
    ids = tokens(cfg, 250, 8)
    whole = m.run(ids, [250])
    m.fused.portion = 100
    assert worst(m.run(ids, [250]), whole) < 1e-4


def test_command_line_replay(scmx, tmp_path):
    from safetensors.torch import save_file
    cfg = CONFIGS["odd"]
    m = Model(scmx, cfg, F32, 30)
    model, out = tmp_path / "model", tmp_path / "out"
    model.mkdir(), out.mkdir()
    (model / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.to(BF).contiguous() for k, v in m.W.items()}, str(model / "model.safetensors"))
    m.W = {k: v.to(BF) for k, v in m.W.items()}
    ids = tokens(cfg, 20, 9)
    steps = [{"step": 0, "entries": [{"id": "q", "tokens": ids[:17], "want": [16, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "q", "tokens": ids[17:18], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "q", "tokens": ids[18:], "want": [1]}], "end": ["q"]}]
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(model), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "20"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = m.oracle(ids)
    assert sorted(os.listdir(out)) == ["0.f32", "2.f32"]
    got = [np.fromfile(out / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"]) for i in (0, 2)]
    assert worst(got[0], want[[16, 2]]) < 2e-4 and worst(got[1], want[[19]]) < 2e-4
