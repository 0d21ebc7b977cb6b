"""GPU: whole Fabezen decoders against the plain float64 oracle, through the framework's prefill, decode, engine, registry and command
line: portions down to two tokens, token by token, requests among others, caches used again, far keys, window borders, long decoding,
greedy generation."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import fabezen_oracle as O

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BF, F32 = torch.bfloat16, torch.float32


def delta(heads, kv, dim, vdim, conv, channel=False, ranks=None):
    mixer = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}
    if ranks:
        mixer["ranks"] = ranks
    return {"type": "channel_delta" if channel else "delta", "mixer": mixer}


def latent(heads, dim, rot, vdim, kv_rank, q_rank, size, base=700.0, scale=0.2):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale,
                                                  "mask": {"size": size}, "rot": {"base": base, "dims": rot}}}


def config(vocab, width, eps, mult, scale, bigram, *layers):
    """layers: (mixer entry, feed-forward width or 0), or the index of the layer whose weights are used again."""
    out = []
    for e in layers:
        if isinstance(e, int):
            out.append({**out[e], "weights_of": e})
        else:
            out.append({**e[0], "mlp": {"kind": "dense", "ff": e[1]} if e[1] else None})
    emb = {"scale": scale}
    if bigram:
        emb["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    return {"architecture": "Fabezen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "embedding": emb, "layers": out}


CONFIGS = {
    "mixed": config(90, 72, 1e-5, 0.6, 5.0, (101, 31, 3), (latent(3, 24, 8, 40, 48, 40, 37), 56), (delta(4, 2, 16, 24, 4), 0), (delta(2, 2, 40, 16, 3, True), 72),
                    0, (delta(6, 3, 8, 8, 2, True, (16, 8)), 40), 2, (latent(2, 64, 16, 32, 24, 56, 64, 9000.0, 0.3), 0), 1),
    "odd": config(51, 36, 1e-3, 1.0, 1.0, (7, 2, 5), (delta(3, 1, 5, 7, 1, False), 20), (latent(3, 5, 2, 7, 11, 9, 5), 28), (delta(2, 1, 6, 10, 5, True, (3, 5)), 12), 1),
    "delta": config(64, 96, 1e-6, 1.3, 2.0, (40, 11, 13), (delta(4, 2, 64, 128, 4), 64), (delta(2, 1, 128, 64, 4, True), 48), 1),
    "latent": config(70, 128, 1e-6, 0.5, 8.0, (33, 5, 17), (latent(4, 32, 16, 64, 64, 48, 130), 96), (latent(2, 128, 64, 128, 96, 64, 1000), 33)),
    "plain": config(40, 24, 1e-2, 0.8, 3.0, None, (delta(2, 2, 16, 16, 3, True), 0), (latent(1, 8, 0, 8, 16, 8, 12), 24)),
}


class Model:
    def __init__(self, scmx, cfg, dtype, capacity, seed=0, sharp=2.0, edit=None):
        self.cfg = cfg
        HM = scmx.host_model
        self.W = {k: torch.from_numpy(v).to(dtype) for k, v in O.random_weights(cfg, seed, sharp).items()}
        if edit:
            edit(self.W)
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


def test_residual_stream_after_every_layer(scmx):
    cfg = CONFIGS["mixed"]
    m = Model(scmx, cfg, F32, 80)
    ids = tokens(cfg, 70, 1)
    want = O.forward(cfg, {k: v.double().numpy() for k, v in m.W.items()}, ids)[1]
    m.fused.trace = []
    m.run(ids, [70])
    got = torch.stack(m.fused.trace).double().cpu().numpy()
    assert got.shape == want.shape and np.abs(got - want).max() < 2e-4 * np.abs(want).max()


@pytest.mark.parametrize("name", ["mixed", "delta", "latent"])
@pytest.mark.parametrize("dtype", [F32, BF])
def test_cuts_change_only_rounding(scmx, name, dtype):
    """Long sequence over chunks of the delta rule (64), attention tiles (128) and decode tiles (32); float32 agrees to rounding."""
    cfg = CONFIGS[name]
    m, T = Model(scmx, cfg, dtype, 700), 640
    ids = tokens(cfg, T, 3)
    whole = m.run(ids, [T])
    for cuts in ([255, 2, 127, 129, 127], [300, 340], [47, 48, 545], [513, 127], [600] + [1] * 40):
        assert worst(m.run(ids, cuts), whole) < (1e-4 if dtype == F32 else 8e-2), cuts


@pytest.mark.parametrize("name", ["mixed", "delta"])
def test_long_decoding(scmx, name):
    cfg = CONFIGS[name]
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


@pytest.mark.parametrize("decoded", [False, True])
def test_window_border(scmx, decoded):
    """One attention layer: changing one token changes exactly the positions whose window holds it."""
    size, T, at = 21, 90, 30
    cfg = config(48, 64, 1e-5, 0.9, 1.0, None, (latent(2, 16, 4, 16, 32, 24, size), 0))
    m = Model(scmx, cfg, F32, 100)
    a = tokens(cfg, T, 5)
    b = a[:at] + [(a[at] + 1) % 48] + a[at + 1:]
    cuts = [10] + [1] * 80 if decoded else [T]
    diff, want = m.run(a, cuts) - m.run(b, cuts), m.oracle(a) - m.oracle(b)
    seen = np.abs(want[at:at + size]).max(-1)
    assert seen.min() > 1e-4 and np.abs(diff - want).max() < 0.2 * seen.min()
    assert np.abs(diff[:at]).max() < 0.1 * seen.min() and np.abs(diff[at + size:]).max() < 0.1 * seen.min()


def test_first_and_previous_tokens(scmx):
    """The pair table's row changes with the previous token only, and the first token of every sequence uses the last row."""
    cfg = config(30, 32, 1e-5, 1.0, 1.0, (13, 3, 1), (delta(2, 2, 8, 8, 1), 0))

    def edit(W):
        W["l0.mix.o"].zero_()                      # nothing but the embedding reaches the logits
    m = Model(scmx, cfg, F32, 40, edit=edit)
    ids = tokens(cfg, 12, 6)
    want = m.oracle(ids)
    for cuts in ([12], [1] * 12, [1, 11], [5, 1, 6]):
        assert worst(m.run(ids, cuts), want) < 1e-4, cuts
    same = m.run([ids[3], ids[3], ids[3]], [1, 1, 1])
    assert np.abs(same[1] - same[2]).max() < 1e-5 < 1e-2 < np.abs(same[0] - same[1]).max()


def test_delta_remembers_a_far_token(scmx):
    """Two prompts that differ in one token 500 positions back, decays near one: the difference at the end is the oracle's."""
    cfg = config(60, 64, 1e-5, 0.7, 4.0, (19, 7, 3), (delta(2, 1, 32, 32, 2), 0), (delta(2, 2, 32, 16, 2, True), 32))

    def edit(W):
        W["l0.mix.A_log"].fill_(-9.0)
        W["l1.mix.A_log"].fill_(-9.0)
        for i in (0, 1):
            W[f"l{i}.mix.b"].mul_(0.05)
    m, T = Model(scmx, cfg, F32, 600, edit=edit), 520
    a = tokens(cfg, T, 7)
    b = a[:10] + [(a[10] + 1) % 60] + a[11:]
    want = m.oracle(a)[-1] - m.oracle(b)[-1]
    assert np.abs(want).max() > 0.01
    for cuts in ([T], [300, 2, 217, 1]):
        got = m.run(a, cuts)[-1] - m.run(b, cuts)[-1]
        assert np.abs(got - want).max() < 0.05 * np.abs(want).max(), cuts


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


@pytest.mark.parametrize("name", ["mixed", "delta", "latent", "plain"])
@pytest.mark.parametrize("dtype", [F32, BF])
def test_greedy_generation(scmx, name, dtype):
    """Engine.generate (prompt in one step, then the captured graph): the continuation is the oracle's argmax at every position
    where the oracle's choice is clear, and a second request from the same engine repeats it."""
    cfg = CONFIGS[name]
    m, n = Model(scmx, cfg, dtype, 120), 60
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


def test_long_prompt_is_cut_into_portions(scmx):
    cfg = CONFIGS["mixed"]
    m = Model(scmx, cfg, F32, 300)
    ids = tokens(cfg, 250, 8)
    whole = m.run(ids, [250])
    m.fused.portion = 100
    assert worst(m.run(ids, [250]), whole) < 1e-4


def test_shared_layers_hold_their_weights_once(scmx):
    cfg = CONFIGS["mixed"]
    m = Model(scmx, cfg, F32, 20)
    layers = m.fused.layers
    assert layers[3] is layers[0] and layers[5] is layers[2] and layers[7] is layers[1] and len(set(map(id, layers))) == 5
    cache = m.fused.make_cache(20)
    assert cache[3].c.data_ptr() != cache[0].c.data_ptr() and cache[5].kv.data_ptr() != cache[2].kv.data_ptr()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_command_line_replay(scmx, tmp_path, dtype):
    from safetensors.torch import save_file
    cfg = json.loads(json.dumps(CONFIGS["odd"]))
    for e in cfg["layers"]:
        e["mixer"].pop("ranks", None)              # inner sizes come from the tensors
    m = Model(scmx, CONFIGS["odd"], BF, 30)
    model, out = tmp_path / "model", tmp_path / "out"
    model.mkdir(), out.mkdir()
    (model / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in m.W.items()}, str(model / "model.safetensors"))
    ids = tokens(cfg, 20, 9)
    steps = [{"step": 0, "entries": [{"id": "q", "tokens": ids[:17], "want": [16, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "q", "tokens": ids[17:18], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "q", "tokens": ids[18:], "want": [1]}], "end": ["q"]}]
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(model), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "20"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    want, tol = m.oracle(ids), 2e-4 if dtype == "float32" else 8e-2
    assert sorted(os.listdir(out)) == ["0.f32", "2.f32"]
    got = [np.fromfile(out / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"]) for i in (0, 2)]
    assert worst(got[0], want[[16, 2]]) < tol and worst(got[1], want[[19]]) < tol
