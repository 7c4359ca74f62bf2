"""GPU: whole Pakalix models through the engine (prompt pass, token step, captured step, sequences, generate), against the
plain restatement of the equations in oracle/pakalix.py."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from llamatov_b200 import _lib, archs, dev_residency as dr, layered, llamatov_run as R, mixers, prefill as pf
from llamatov_b200.sequences import Sequences
from oracle import pakalix as O
from tests import layered_util as U
from tests import pakalix_util as K
from tests.test_gpu_layered import DTYPES, ROOT, TOL, _portions, _tokens

pytestmark = pytest.mark.gpu


@pytest.fixture(autouse=True)
def _clean():
    dr.reset_engine_state(); dr.apply_production_profile()
    yield
    assert _lib.device_status() == set()


MODELS = {
    "mixed": dict(),
    "odd-sizes": dict(width=52, vocab=77, residual_mult=1.0, layers=[
        K.layer("mamba2", K.mamba2(heads=5, groups=5, vdim=9, state=12, conv=3, norm_groups=9), 30),
        K.layer("attention", K.attention(heads=9, kv_heads=3, dim=11, vdim=13, rot=6), 41, 0.3),
        K.layer("attention", K.attention(heads=6, kv_heads=3, dim=10, vdim=13, rot=10, softcap=2.0), None),
        K.layer("mamba2", K.mamba2(heads=6, groups=2, vdim=20, state=7, conv=2, norm_groups=4), 17, 5.0)]),
    "ones": dict(width=24, vocab=50, layers=[
        K.layer("attention", K.attention(heads=1, kv_heads=1, dim=8, vdim=8, rot=2), None),
        K.layer("mamba2", K.mamba2(heads=1, groups=1, vdim=8, state=8, conv=1, norm_groups=1), 8),
        K.layer("mamba2", K.mamba2(heads=2, groups=1, vdim=1, state=1, conv=2, norm_groups=2), 16),
        K.layer("attention", K.attention(heads=4, kv_heads=4, dim=2, vdim=1, rot=2, v_mix=False), 16)]),
    "wide-heads": dict(width=136, vocab=120, residual_mult=0.3, layers=[
        K.layer("mamba2", K.mamba2(heads=4, groups=2, vdim=136, state=160, conv=4, norm_groups=2), 72),
        K.layer("attention", K.attention(heads=16, kv_heads=1, dim=64, vdim=136, rot=32), 200),
        K.layer("mamba2", K.mamba2(heads=8, groups=8, vdim=16, state=264, conv=5, norm_groups=8), 72)]),
    "attention-only": dict(layers=[K.layer("attention", K.attention(softcap=s)) for s in (1.0, 5.0, 50.0)]),
    "mamba-only": dict(layers=[K.layer("mamba2", K.mamba2(norm_groups=n)) for n in (1, 2, 6, 36)]),
    "no-cap-no-rotation": dict(layers=[K.layer("attention", {k: v for k, v in K.attention(rot=0).items() if k != "softcap"}),
                                       K.layer("mamba2", K.mamba2())]),
    "mixing-starts-late": dict(layers=[K.layer("attention", K.attention(v_mix=False, vdim=16)), K.layer("attention", K.attention()),
                                       K.layer("attention", K.attention(v_mix=False)), K.layer("attention", K.attention(heads=2))]),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(MODELS))
def test_models_whole_and_in_portions(name, dtype):
    cfg = K.config(**MODELS[name])
    t = K.random_tensors(cfg, seed=11)
    toks = _tokens(cfg, 150)
    want = K.oracle_logits(cfg, t, toks)
    c, w = U.product(cfg, t, dtype)
    S = Sequences(w, c, 160)
    for i, sizes in enumerate(([150], [1], [2], [97, 1], [5, 64, 1, 1, 2, 66, 3], [40, 41])):
        n = 60 if sizes[0] < 3 else 150
        got = _portions(S, i, toks[:n], sizes)
        assert U.rel_rms(got, want[:n]) < TOL[dtype], (name, sizes)
        S.end(i)


@pytest.mark.parametrize("dtype", DTYPES)
def test_layer_by_layer_against_the_oracle(dtype):
    cfg = K.config()
    t = K.random_tensors(cfg, seed=12)
    toks = _tokens(cfg, 70, 3)
    m = O.Model(cfg, U.as_numpy(t)); m.run(toks)
    c, w = U.product(cfg, t, dtype)
    seen = []

    def tap(run, x):
        seen.append(run.slot)
        assert U.rel_rms(x.cpu().numpy(), m.taps[run.slot]) < TOL[dtype], run
    pf.prefill_resident(w, c, torch.tensor(toks), [None] * archs.of(c).n_slots(c), want_rows=[], tap=tap)
    assert seen == list(range(5))


@pytest.mark.parametrize("block", [layered.SequentialBlock, layered.ParallelBlock])
@pytest.mark.parametrize("name", ["Nugusun", "Pakalix"])
def test_every_mixer_runs_in_every_block(monkeypatch, block, name):
    """Prompt pass and token steps agree (fp32) for all mixers under both kinds of block."""
    A = archs.by_name(name)
    monkeypatch.setattr(type(A), "block", block)
    kinds = [K.layer("mamba2", K.mamba2()), U.layer("gla", U.gla()), K.layer("attention", K.attention()),
             U.layer("latent_attention", U.latent()), U.layer("lightning", U.lightning(), None)]
    for k in kinds:
        if k["mlp"] is not None:
            k["mlp"] = {"kind": "dense", "ff": 40, "limit": 1.2}
    c1, c2 = U.config(layers=[k for k in kinds if k["type"] not in ("mamba2", "attention")], loop=None), \
        K.config(layers=[k for k in kinds if k["type"] in ("mamba2", "attention")])
    t1, t2 = U.random_tensors(c1, seed=1), K.random_tensors(c2, seed=2)
    js = {**U.config(layers=kinds, loop=None), **K.config(layers=kinds), "architecture": name}
    t = {**t1, **{k: v for k, v in t2.items() if not k[0] == "l"}}
    for i, (src, j) in enumerate(((t2, 0), (t1, 0), (t2, 1), (t1, 1), (t1, 2))):
        t.update({f"l{i}." + k[3:]: v for k, v in src.items() if k.startswith(f"l{j}.")})
        t.setdefault(f"l{i}.norm2", torch.ones(js["width"]).bfloat16())
    c, w = U.product(js, t, "float32")
    c["residual_mult"] = 0.5
    S = Sequences(w, c, 100)
    toks = _tokens(js, 90, 4)
    a = S.step("a", toks, range(90)).numpy()
    assert np.isfinite(a).all() and U.rel_rms(_portions(S, "b", toks, [3, 1]), a) < 1e-4


def test_chunked_and_scanned_prompts_agree(monkeypatch):
    cfg = K.config()
    c, w = U.product(cfg, K.random_tensors(cfg, seed=13), "bfloat16")
    toks = _tokens(cfg, 200)
    S = Sequences(w, c)
    a = S.step("a", toks, range(200)).numpy()
    monkeypatch.setattr(mixers, "CHUNKED_FROM", 10 ** 9)
    b = S.step("b", toks, range(200)).numpy()
    assert U.rel_rms(a, b) < TOL["bfloat16"]


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompts_and_long_decoding(dtype, monkeypatch):
    """Prompts of several passes, then some hundred single tokens."""
    monkeypatch.setattr(layered.Layered, "max_rows", 24)
    cfg = K.config(layers=[K.layer("mamba2", K.mamba2(heads=2, groups=1, norm_groups=1)), K.layer("attention", K.attention(heads=2, kv_heads=1))])
    t = K.random_tensors(cfg, seed=14)
    toks = _tokens(cfg, 400, 5)
    want = K.oracle_logits(cfg, t, toks)
    c, w = U.product(cfg, t, dtype)
    S = Sequences(w, c, 400)
    got = _portions(S, "a", toks, [101, 3, 50, 1])
    assert U.rel_rms(got, want) < TOL[dtype]
    assert S.length("a") == 400 and all(k.length == 400 for k in S.live["a"].kv)
    with pytest.raises(RuntimeError, match="overflow"):
        S.step("a", [1], [0])
    with pytest.raises(RuntimeError, match="overflow"):
        S.step("a", [1, 2], [0])


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_are_reused_and_sequences_do_not_touch(dtype):
    """Sequences of unequal lengths interleaved token by token, ended and followed by others in the same slots."""
    cfg = K.config()
    t = K.random_tensors(cfg, seed=15)
    c, w = U.product(cfg, t, dtype)
    S = Sequences(w, c)
    reqs = {i: _tokens(cfg, n, 20 + i) for i, n in enumerate((33, 5, 90, 1, 41))}
    alone = {i: _portions(Sequences(w, c), i, q, [max(1, len(q) - 6), 1]) for i, q in reqs.items()}
    out, at = {i: [] for i in reqs}, {i: 0 for i in reqs}
    active, waiting, kvs = [0, 1], [2, 3, 4], set()
    while active:
        for i in list(active):
            n = max(1, len(reqs[i]) - 6) if at[i] == 0 else 1
            out[i].append(S.step(i, reqs[i][at[i]:at[i] + n], list(range(n))).numpy())
            kvs.add(id(S.live[i]))
            at[i] += n
            if at[i] == len(reqs[i]):
                S.end(i)
                active.remove(i)
                if waiting:
                    active.append(waiting.pop(0))
    assert len(kvs) == 2 and len(S.free) == 2 and not S.live
    for i in reqs:
        assert np.array_equal(np.concatenate(out[i]), alone[i]), i       # the same kernels on other slots: the same bits
        assert U.rel_rms(alone[i], K.oracle_logits(cfg, t, reqs[i])) < TOL[dtype]


def test_freed_state_is_emptied():
    cfg = K.config()
    c, w = U.product(cfg, K.random_tensors(cfg, seed=16), "float32")
    S = Sequences(w, c)
    q = _tokens(cfg, 30)
    a = S.step("a", q, range(30)).numpy()
    S.step("a", q[:1]); S.step("a", q[:1])
    S.end("a")
    kv = S.free[0].kv
    assert all(k.length == 0 and int(k._len.item()) == 0 for k in kv)
    assert all(float(k.state.abs().sum()) == 0 for k in kv if isinstance(k, dr.DeviceSsdState))
    assert np.array_equal(S.step("b", q, range(30)).numpy(), a)
    S.end("b")
    first = S.step("c", q[:1], [0]).numpy()              # a sequence that starts with a captured single token
    assert U.rel_rms(first, a[:1]) < 1e-5


@pytest.mark.parametrize("dtype", DTYPES)
def test_captured_step_equals_eager_step(dtype):
    cfg = K.config()
    c, w = U.product(cfg, K.random_tensors(cfg, seed=17), dtype)
    toks = _tokens(cfg, 50)
    A = archs.of(c)
    A.ensure_buffers(w, c)
    kv = [None] * A.n_slots(c)
    eager = [dr.forward_pass_resident(w, c, torch.tensor([t]), torch.tensor([p]), kv).reshape(-1).numpy().copy() for p, t in enumerate(toks)]
    S = Sequences(w, c)
    for p, t in enumerate(toks):
        assert np.array_equal(S.step("a", [t], [0]).numpy()[0], eager[p]), p
    r = S.live["a"].runner
    assert r.captured and r.launches_per_token <= 3 * 5 + 4        # three launches a layer; embedding, logits, argmax


def test_unequal_sequences_in_one_prompt_pass():
    """Two sequences of one pass that stand at different positions."""
    cfg = K.config()
    t = K.random_tensors(cfg, seed=18)
    c, w = U.product(cfg, t, "bfloat16")
    A = archs.of(c)
    q = [_tokens(cfg, 100, 1), _tokens(cfg, 70, 2)]
    kvs = [[None] * A.n_slots(c) for _ in q]
    pf.prefill_resident(w, c, torch.tensor(q[0][:31]), kvs[0], want_rows=[])
    pf.prefill_resident(w, c, torch.tensor(q[1][:1]), kvs[1], want_rows=[])
    got = pf.prefill_resident(w, c, torch.tensor([q[0][31:100], q[1][1:70]]), kvs, want_rows=list(range(138))).numpy()
    for i, lo in enumerate((31, 1)):
        assert U.rel_rms(got[69 * i:69 * i + 69], K.oracle_logits(cfg, t, q[i])[lo:]) < TOL["bfloat16"]


def test_far_tokens_are_remembered():
    """One key of the first token stands out: changing it moves the last logits, and by what the oracle says."""
    cfg = K.config(layers=[K.layer("attention", K.attention(heads=2, kv_heads=1, scale=0.6, softcap=30.0)), K.layer("mamba2", K.mamba2())])
    t = K.random_tensors(cfg, seed=19)
    t["l0.mix.q.norm"] = t["l0.mix.q.norm"] * 2
    t["l1.mix.A_log"] = t["l1.mix.A_log"] * 0 - 12.0          # hardly any decay
    c, w = U.product(cfg, t, "float32")
    q = _tokens(cfg, 300, 7)
    r = [(q[0] + 1) % cfg["vocab"]] + q[1:]
    S = Sequences(w, c, 320)
    for lo in (300, 290):                                     # the last ten from a prompt, or decoded
        a, b = _portions(S, "q", q, [lo, 1])[-1], _portions(S, "r", r, [lo, 1])[-1]
        want = K.oracle_logits(cfg, t, q)[-1] - K.oracle_logits(cfg, t, r)[-1]
        assert np.abs(want).max() > 1e-3 and np.abs(a - b - want).max() < 0.02 * np.abs(want).max()
        S.end("q"); S.end("r")


# --------------------------------------------------------------------------- generation

def _greedy_oracle(cfg, t, prompt, n):
    m = O.Model(cfg, U.as_numpy(t))
    lg = m.run(prompt)[-1]
    out, gap = [], []
    for _ in range(n):
        s = np.sort(lg)
        gap.append(s[-1] - s[-2])
        out.append(int(np.argmax(lg)))
        lg = m.run([out[-1]])[-1]
    return out, min(gap)


@pytest.mark.parametrize("plen", [1, 2, 40])
def test_generate_from_a_folder_is_greedy(tmp_path, plen):
    cfg = K.config()
    t = K.random_tensors(cfg, seed=21)
    path = U.write_model(tmp_path / "m", cfg, t)
    prompt = _tokens(cfg, plen, 9)
    want, gap = _greedy_oracle(cfg, t, prompt, 25)
    assert gap > 1e-3                      # far above fp32 rounding: the tokens are decided
    assert R.generate(path, prompt, 25, verbose=False, dtype="float32") == prompt + want
    got = R.generate(path, prompt, 25, verbose=False)
    assert got[:plen] == prompt and len(got) == plen + 25


def test_device_token_loop_equals_host_loop():
    cfg = K.config()
    c, w = U.product(cfg, K.random_tensors(cfg, seed=22), "bfloat16")
    prompt = _tokens(cfg, 30)
    host = R.generate("", prompt, 20, preloaded=(c, w), verbose=False)
    kv = [None] * archs.of(c).n_slots(c)
    gr = dr.GraphRunner(w, c, kv)
    first = int(gr.seed(torch.tensor(prompt), torch.arange(len(prompt))).reshape(-1).argmax())
    gr.capture_device_loop(first)
    gr.replay_device(19)
    assert [first] + gr.device_tokens() == host[len(prompt):]


def test_command_line_generates(tmp_path):
    cfg = K.config()
    path = U.write_model(tmp_path / "m", cfg, K.random_tensors(cfg, seed=23))
    r = subprocess.run([sys.executable, "-m", "llamatov_b200.llamatov_run", path, "3,5,7", "6", "--dtype=float32"], cwd=ROOT,
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    want = R.generate(path, [3, 5, 7], 6, verbose=False, dtype="float32")
    assert f"GENERATED: {want[3:]}" in r.stdout


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_run_replays_portions(tmp_path, dtype):
    cfg = K.config()
    t = K.random_tensors(cfg, seed=24)
    path = U.write_model(tmp_path / "m", cfg, t)
    out = tmp_path / "out"
    out.mkdir()
    a, b = _tokens(cfg, 45, 1), _tokens(cfg, 12, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:40], "want": [39, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[40:41], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[41:], "want": [0, 3]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b, "want": [11]}], "end": ["b"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(out), "--max-tokens", "45"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    wa, wb = K.oracle_logits(cfg, t, a), K.oracle_logits(cfg, t, b)
    read = lambda i: np.fromfile(out / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"])
    assert U.rel_rms(read(0), wa[[39, 3]]) < TOL[dtype] and U.rel_rms(read(2), wa[[41, 44]]) < TOL[dtype]
    assert U.rel_rms(read(3), wb[[11]]) < TOL[dtype] and not (out / "1.f32").exists()


def test_impossible_models_are_refused():
    cfg = K.config(layers=[K.layer("attention", K.attention(heads=4, kv_heads=2))])
    t = K.random_tensors(cfg, seed=25)
    cfg["layers"][0]["mixer"]["kv_heads"] = 3
    c, w = U.product(cfg, t, "bfloat16")
    with pytest.raises(ValueError, match="key heads"):
        Sequences(w, c).step("a", [1, 2], [0])
    cfg = K.config(layers=[K.layer("mamba2", K.mamba2(conv=3))])
    t = K.random_tensors(cfg, seed=25)
    cfg["layers"][0]["mixer"]["conv"] = 4
    c, w = U.product(cfg, t, "bfloat16")
    with pytest.raises(ValueError, match="taps"):
        Sequences(w, c).step("a", [1, 2], [0])
