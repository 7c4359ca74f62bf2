"""GPU: whole mixer-layer models through the engine (prompt pass, token step, captured step, sequences, generate), against
the plain restatement of the equations in oracle/layered.py."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from llamatov_b200 import _lib, archs, dev_residency as dr, layered, llamatov_run as R, mixers, prefill as pf
from llamatov_b200.sequences import Sequences
from oracle import layered as L
from tests import layered_util as U

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = ["float32", "bfloat16"]
TOL = {"float32": 2e-4, "bfloat16": 8e-2}


@pytest.fixture(autouse=True)
def _clean():
    dr.reset_engine_state(); dr.apply_production_profile()
    yield
    assert _lib.device_status() == set()


def _tokens(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def _portions(S, sid, toks, sizes):
    """logits of every token, fed in portions of the given sizes (the last size repeats)"""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(sizes[min(i, len(sizes) - 1)], len(toks) - at)
        out.append(S.step(sid, toks[at:at + n], list(range(n))).numpy())
        at += n
        i += 1
    return np.concatenate(out)


MODELS = {
    "mixed": dict(),
    "no-loop": dict(loop=None),
    "loop-all-three-times": dict(loop={"start": 0, "stop": 4, "times": 3}),
    "loop-once": dict(loop={"start": 2, "stop": 4, "times": 1}),
    "odd-sizes": dict(width=52, vocab=77, layers=[
        U.layer("lightning", U.lightning(heads=5, dim=12, vdim=9), 30),
        U.layer("latent_attention", U.latent(heads=3, dim=11, rot_dim=6, vdim=13, kv_rank=20, window=9), 41),
        U.layer("gla", U.gla(heads=3, dim=10, vdim=7, tau=1.0), None)], loop={"start": 1, "stop": 3, "times": 2}),
    "ones": dict(width=24, vocab=50, layers=[
        U.layer("latent_attention", U.latent(heads=1, dim=8, rot_dim=2, vdim=8, kv_rank=8, window=1), None),
        U.layer("lightning", U.lightning(heads=1, dim=8, vdim=8, decay=[1.0]), 8),
        U.layer("gla", U.gla(heads=1, dim=8, vdim=8, tau=2.0), 16),
        U.layer("latent_attention", U.latent(heads=1, dim=8, rot_dim=8, vdim=16, kv_rank=16, window=2), 16)], loop=None),
    "wide-heads": dict(width=136, vocab=120, layers=[
        U.layer("gla", U.gla(heads=1, dim=136, vdim=160, tau=4.0), 72),
        U.layer("latent_attention", U.latent(heads=9, dim=64, rot_dim=32, vdim=136, kv_rank=264, window=40), 200),
        U.layer("lightning", U.lightning(heads=2, dim=96, vdim=56, decay=[0.0, 0.995]), 72)], loop={"start": 0, "stop": 1, "times": 2}),
    "window-beyond-the-sequence": dict(layers=[U.layer("latent_attention", U.latent(window=4000)), U.layer("gla", U.gla())], loop=None),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(MODELS))
def test_models_whole_and_in_portions(name, dtype):
    cfg = U.config(**MODELS[name])
    t = U.random_tensors(cfg, seed=11, rank_a=10)
    toks = _tokens(cfg, 150)
    want = U.oracle_logits(cfg, t, toks)
    c, w = U.product(cfg, t, dtype)
    S = Sequences(w, c)
    for i, sizes in enumerate(([150], [1], [2], [97, 1], [5, 64, 1, 1, 2, 66, 3], [40, 41])):
        n = 60 if sizes[0] < 3 else 150
        got = _portions(S, i, toks[:n], sizes)
        assert U.rel_rms(got, want[:n]) < TOL[dtype], (name, sizes)
        S.end(i)


@pytest.mark.parametrize("dtype", DTYPES)
def test_layer_by_layer_against_the_oracle(dtype):
    cfg = U.config()
    t = U.random_tensors(cfg, seed=12)
    toks = _tokens(cfg, 70, 3)
    m = L.Model(cfg, U.as_numpy(t)); m.run(toks)
    c, w = U.product(cfg, t, dtype)
    seen = []

    def tap(run, x):
        seen.append(run.slot)
        assert U.rel_rms(x.cpu().numpy(), m.taps[run.slot]) < TOL[dtype], run
    pf.prefill_resident(w, c, torch.tensor(toks), [None] * archs.of(c).n_slots(c), want_rows=[], tap=tap)
    assert seen == list(range(len(m.runs)))


def test_chunked_and_scanned_prompts_agree(monkeypatch):
    cfg = U.config()
    c, w = U.product(cfg, U.random_tensors(cfg, seed=13), "bfloat16")
    toks = _tokens(cfg, 200)
    S = Sequences(w, c)
    a = S.step("a", toks, range(200)).numpy()
    monkeypatch.setattr(mixers, "CHUNKED_FROM", 10 ** 9)
    b = S.step("b", toks, range(200)).numpy()
    assert U.rel_rms(a, b) < TOL["bfloat16"]


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompts_and_long_decoding_wrap_the_ring(dtype, monkeypatch):
    """Few rows per pass: a ring hardly longer than the window, passed around many times by prompts and by decoding."""
    monkeypatch.setattr(layered.Layered, "max_rows", 24)
    cfg = U.config()
    t = U.random_tensors(cfg, seed=14)
    toks = _tokens(cfg, 400, 5)
    want = U.oracle_logits(cfg, t, toks)
    c, w = U.product(cfg, t, dtype)
    S = Sequences(w, c)
    got = _portions(S, "a", toks, [101, 3, 50, 1])
    assert max(k.cap for k in S.live["a"].kv if isinstance(k, dr.DeviceLatentCache)) == 18 + 24
    assert U.rel_rms(got, want) < TOL[dtype]
    assert S.length("a") == 400 and all(k.length == 400 for k in S.live["a"].kv)


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_are_reused_and_sequences_do_not_touch(dtype):
    """Sequences of unequal lengths interleaved token by token, ended and followed by others in the same slots."""
    cfg = U.config()
    t = U.random_tensors(cfg, seed=15)
    c, w = U.product(cfg, t, dtype)
    S = Sequences(w, c)
    reqs = {i: _tokens(cfg, n, 20 + i) for i, n in enumerate((33, 5, 90, 1, 41))}
    alone = {}
    for i, q in reqs.items():
        T = Sequences(w, c)
        alone[i] = _portions(T, i, q, [max(1, len(q) - 6), 1])
    out = {i: [] for i in reqs}
    at = {i: 0 for i in reqs}
    rng = np.random.default_rng(0)
    active, waiting, kvs = [0, 1], [2, 3, 4], set()
    while active:
        for i in list(active):
            first = at[i] == 0
            n = max(1, len(reqs[i]) - 6) if first else 1
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
        assert U.rel_rms(alone[i], U.oracle_logits(cfg, t, reqs[i])) < TOL[dtype]


def test_freed_state_is_emptied():
    cfg = U.config()
    c, w = U.product(cfg, U.random_tensors(cfg, seed=16), "float32")
    S = Sequences(w, c)
    q = _tokens(cfg, 30)
    a = S.step("a", q, range(30)).numpy()
    S.end("a")
    kv = S.free[0].kv
    assert all(k.length == 0 for k in kv) and all(float(k.state.abs().sum()) == 0 for k in kv if isinstance(k, dr.DeviceRecurrentState))
    assert np.array_equal(S.step("b", q, range(30)).numpy(), a)


@pytest.mark.parametrize("dtype", DTYPES)
def test_captured_step_equals_eager_step(dtype):
    cfg = U.config()
    c, w = U.product(cfg, U.random_tensors(cfg, seed=17), dtype)
    toks = _tokens(cfg, 50)
    A = archs.of(c)
    A.ensure_buffers(w, c)
    kv = [None] * A.n_slots(c)
    eager = [dr.forward_pass_resident(w, c, torch.tensor([t]), torch.tensor([p]), kv).reshape(-1).numpy().copy() for p, t in enumerate(toks)]
    S = Sequences(w, c)
    for p, t in enumerate(toks):
        assert np.array_equal(S.step("a", [t], [0]).numpy()[0], eager[p]), p
    assert S.live["a"].runner.captured and S.live["a"].runner.launches_per_token > 0


def test_two_sequences_in_one_prompt_pass():
    cfg = U.config()
    t = U.random_tensors(cfg, seed=18)
    c, w = U.product(cfg, t, "bfloat16")
    A = archs.of(c)
    q = [_tokens(cfg, 80, 1), _tokens(cfg, 80, 2)]
    kvs = [[None] * A.n_slots(c) for _ in q]
    rows = list(range(160))
    a = pf.prefill_resident(w, c, torch.tensor([x[:50] for x in q]), kvs, want_rows=list(range(100))).numpy()
    b = pf.prefill_resident(w, c, torch.tensor([x[50:] for x in q]), kvs, want_rows=list(range(60))).numpy()
    for i in range(2):
        got = np.concatenate([a[50 * i:50 * i + 50], b[30 * i:30 * i + 30]])
        assert U.rel_rms(got, U.oracle_logits(cfg, t, q[i])) < TOL["bfloat16"]
    assert len(rows) == 160


def test_far_tokens_are_remembered():
    """Strong memory (decay 1 in one head): changing the first token moves the last logits, and by what the oracle says."""
    cfg = U.config(layers=[U.layer("lightning", U.lightning(heads=2, dim=16, vdim=16, decay=[1.0, 0.9])),
                           U.layer("latent_attention", U.latent(window=5))], loop={"start": 0, "stop": 2, "times": 2})
    t = U.random_tensors(cfg, seed=19)
    c, w = U.product(cfg, t, "float32")
    q = _tokens(cfg, 300, 7)
    r = [(q[0] + 1) % cfg["vocab"]] + q[1:]
    S = Sequences(w, c)
    d = S.step("q", q, [299]).numpy() - S.step("r", r, [299]).numpy()
    want = U.oracle_logits(cfg, t, q)[[299]] - U.oracle_logits(cfg, t, r)[[299]]
    assert np.abs(want).max() > 1e-3 and np.abs(d - want).max() < 0.02 * np.abs(want).max()


# --------------------------------------------------------------------------- generation

def _greedy_oracle(cfg, t, prompt, n):
    m = L.Model(cfg, U.as_numpy(t))
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
    cfg = U.config()
    t = U.random_tensors(cfg, seed=21)
    path = U.write_model(tmp_path / "m", cfg, t)
    prompt = _tokens(cfg, plen, 9)
    want, gap = _greedy_oracle(cfg, t, prompt, 25)
    assert gap > 1e-3                      # far above fp32 rounding: the tokens are decided
    assert R.generate(path, prompt, 25, verbose=False, dtype="float32") == prompt + want
    got = R.generate(path, prompt, 25, verbose=False)
    assert got[:plen] == prompt and len(got) == plen + 25


def test_eager_driver_generates_the_same(tmp_path):
    from llamatov_b200 import decode_fact
    cfg = U.config()
    path = U.write_model(tmp_path / "m", cfg, U.random_tensors(cfg, seed=26))
    prompt = _tokens(cfg, 12, 3)
    assert decode_fact.decode(path, prompt, 8) == R.generate(path, prompt, 8, verbose=False)


def test_device_token_loop_equals_host_loop():
    cfg = U.config()
    c, w = U.product(cfg, U.random_tensors(cfg, seed=22), "bfloat16")
    prompt = _tokens(cfg, 30)
    host = R.generate("", prompt, 20, preloaded=(c, w), verbose=False)
    kv = [None] * archs.of(c).n_slots(c)
    gr = dr.GraphRunner(w, c, kv)
    first = int(gr.seed(torch.tensor(prompt), torch.arange(len(prompt))).reshape(-1).argmax())
    gr.capture_device_loop(first)
    gr.replay_device(19)
    assert [first] + gr.device_tokens() == host[len(prompt):]


def test_command_line_generates(tmp_path):
    cfg = U.config()
    path = U.write_model(tmp_path / "m", cfg, U.random_tensors(cfg, seed=23))
    r = subprocess.run([sys.executable, "-m", "llamatov_b200.llamatov_run", path, "3,5,7", "6", "--dtype=float32"], cwd=ROOT,
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    want = R.generate(path, [3, 5, 7], 6, verbose=False, dtype="float32")
    assert f"GENERATED: {want[3:]}" in r.stdout


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_run_replays_portions(tmp_path, dtype):
    cfg = U.config()
    t = U.random_tensors(cfg, seed=24)
    path = U.write_model(tmp_path / "m", cfg, t)
    out = tmp_path / "out"
    out.mkdir()
    a, b = _tokens(cfg, 45, 1), _tokens(cfg, 12, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:40], "want": [39, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[40:41], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[41:], "want": [0, 3]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b, "want": [11]}], "end": ["b"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(out), "--max-tokens", "64"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    wa, wb = U.oracle_logits(cfg, t, a), U.oracle_logits(cfg, t, b)
    V = cfg["vocab"]
    read = lambda i: np.fromfile(out / f"{i}.f32", "<f4").reshape(-1, V)
    assert U.rel_rms(read(0), wa[[39, 3]]) < TOL[dtype] and U.rel_rms(read(2), wa[[41, 44]]) < TOL[dtype]
    assert U.rel_rms(read(3), wb[[11]]) < TOL[dtype] and not (out / "1.f32").exists()


def test_bad_requests_are_refused():
    cfg = U.config()
    c, w = U.product(cfg, U.random_tensors(cfg, seed=25), "bfloat16")
    S = Sequences(w, c)
    with pytest.raises(ValueError, match="vocabulary"):
        S.step("a", [cfg["vocab"]], [0])
    with pytest.raises(ValueError, match="wanted"):
        S.step("a", [1, 2], [2])
    cfg["layers"][0]["type"] = "nonesuch"
    c, w = U.product(cfg, U.random_tensors(U.config(), seed=25), "bfloat16")
    with pytest.raises(NotImplementedError, match="nonesuch"):
        Sequences(w, c).step("a", [1, 2], [0])
