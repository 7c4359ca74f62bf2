"""CPU: configuration, loading, packing and binding of the mixer-layer models, and the oracle's own consistency."""
import ctypes
import os
import re
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracle import layered as L
from tests import layered_util as U

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# --------------------------------------------------------------------------- library binding

def test_dense_header_symbols_exported_and_bound():
    from llamatov_b200 import _lib
    text = open(os.path.join(ROOT, "include", "llamatov_b200_dense.h")).read()
    text = re.sub(r"/\*.*?\*/", "", text, flags=re.S)
    names = sorted(set(re.findall(r"\b(lt_dn_[a-z0-9_]+)\s*\(", text)))
    lib = ctypes.CDLL(_lib.DENSE_PATH)
    for n in names:
        assert hasattr(lib, n), n
    assert set(names) == set(_lib.DENSE_SIGNATURES) | set(_lib._DENSE_QUERIES)


def test_dense_argument_validation_without_gpu():
    from llamatov_b200 import _lib
    lib = _lib.dense()
    one = ctypes.c_void_p(256)     # never dereferenced: validation fails first
    e = _lib.DnEpilogue()
    assert lib.lt_dn_linear(one, 12, one, 16, one, 8, 0, 8, 12, 4, ctypes.byref(e), 0, None) == 1
    assert "multiple of 8" in _lib.last_error()
    assert lib.lt_dn_linear(one, 16, one, 16, one, 4, 0, 8, 16, 4, ctypes.byref(e), 0, None) == 1
    e.kind = 7
    assert lib.lt_dn_linear(one, 16, one, 16, one, 8, 0, 8, 16, 4, ctypes.byref(e), 0, None) == 1
    assert "epilogue" in _lib.last_error()
    d = _lib.DnDecay()
    assert lib.lt_dn_recurrence(one, one, one, 64, one, one, 64, 0, 5, 2, 16, 16, ctypes.byref(d), None) == 1
    assert "one token" in _lib.last_error()
    lat = _lib.DnLatent(2, 16, 8, 16, 8, 16, 16, 40, 20, 1.0, 1e-6, 256, 256)
    assert lib.lt_dn_latent_step(one, one, one, one, one, one, 0, ctypes.byref(lat), 2, one, None) == 1
    assert "ring" in _lib.last_error()
    assert lib.lt_dn_latent_rows(one, 64, one, one, 15, 30, 0, 8, ctypes.byref(lat), None) == 1


# --------------------------------------------------------------------------- files and configuration

def test_safetensors_round_trip(tmp_path):
    from llamatov_b200.safetensors_io import read_safetensors, write_safetensors
    t = {"a": torch.randn(3, 5).bfloat16(), "b": torch.arange(7, dtype=torch.int32), "c": torch.randn(4), "d": torch.zeros(0, 2)}
    write_safetensors(tmp_path / "x.safetensors", t)
    r = read_safetensors(tmp_path / "x.safetensors")
    assert set(r) == set(t)
    for k in t:
        assert r[k].dtype == t[k].dtype and r[k].shape == t[k].shape and torch.equal(r[k], t[k])
    (tmp_path / "bad").write_bytes(b"\x08\0\0\0\0\0\0\0notjson!")
    with pytest.raises(ValueError):
        read_safetensors(tmp_path / "bad")
    raw = (tmp_path / "x.safetensors").read_bytes()
    (tmp_path / "cut").write_bytes(raw[:-4])
    with pytest.raises(ValueError, match="offsets"):
        read_safetensors(tmp_path / "cut")


def test_loader_chooses_the_architecture(tmp_path):
    from llamatov_b200 import llamatov_run as R
    cfg = U.config()
    path = U.write_model(tmp_path / "m", cfg, U.random_tensors(cfg))
    c, w = R.load_model(path, dtype="float32")
    assert c["arch"] == "Nugusun" and c["n_layers"] == 4 and c["dtype"] == "float32" and c["vocab"] == cfg["vocab"]
    assert w["l0.mix.q"].dtype == torch.bfloat16
    with pytest.raises(ValueError, match="dtype"):
        R.load_model(path, dtype="int8")
    cfg["architecture"] = "Nonesuch"
    with pytest.raises(NotImplementedError, match="Nonesuch"):
        R.load_model(U.write_model(tmp_path / "n", cfg, {}))
    cfg = U.config(loop={"start": 3, "stop": 9, "times": 2})
    with pytest.raises(ValueError, match="loop"):
        R.load_model(U.write_model(tmp_path / "o", cfg, {}))


@pytest.mark.parametrize("loop,want", [
    (None, [(0, None), (1, None), (2, None), (3, None)]),
    ({"start": 1, "stop": 3, "times": 3}, [(0, None), (1, 0), (2, 0), (1, 1), (2, 1), (1, 2), (2, 2), (3, None)]),
    ({"start": 0, "stop": 4, "times": 1}, [(0, 0), (1, 0), (2, 0), (3, 0)]),
    ({"start": 3, "stop": 4, "times": 2}, [(0, None), (1, None), (2, None), (3, 0), (3, 1)])])
def test_layer_runs(loop, want):
    from llamatov_b200 import archs
    cfg = U.config(loop=loop)
    A = archs.by_name("Nugusun")
    runs = A.runs(A.config_from_json(cfg, "bfloat16"))
    assert [(r.layer, r.loop_pass) for r in runs] == want == L.layer_runs(cfg)
    assert [r.slot for r in runs] == list(range(len(want)))
    assert [r.opens_pass for r in runs] == [t is not None and i == loop["start"] for i, t in want]


def test_packing_pads_heads_and_columns():
    from llamatov_b200 import dense_ops as P
    W = torch.arange(2 * 5 * 3, dtype=torch.float32).reshape(10, 3)
    R = P._head_rows(W, [(2, 8), (3, 8)], 2)
    assert R.shape == (32, 3)
    assert torch.equal(R[0:2], W[0:2]) and torch.equal(R[8:11], W[2:5]) and torch.equal(R[16:18], W[5:7])
    assert R[2:8].abs().sum() == 0 and R[11:16].abs().sum() == 0
    O = torch.randn(4, 2 * 5)
    C = P._head_cols(O, 5, 2)
    assert C.shape == (4, 16) and torch.equal(C[:, :5], O[:, :5]) and torch.equal(C[:, 8:13], O[:, 5:]) and C[:, 13:].abs().sum() == 0
    v = P._head_rows(torch.arange(6.0), [(3, 8)], 2)
    assert v.shape == (16,) and v[8:11].tolist() == [3.0, 4.0, 5.0]


def test_other_families_still_registered():
    from llamatov_b200 import archs, q8_block
    assert archs.of({"arch": "qwen2", "n_layers": 2}) is q8_block.ARCH and archs.of({"n_layers": 2}) is q8_block.ARCH
    assert archs.of({"arch": "llama"}).n_slots({"n_layers": 5}) == 5


def test_trace_run_refuses_an_unknown_model(tmp_path):
    cfg = U.config()
    cfg["architecture"] = "Nonesuch"
    path = U.write_model(tmp_path / "m", cfg, {})
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", "bfloat16", "--out", str(tmp_path)],
                       input="", capture_output=True, text=True, timeout=300)
    assert r.returncode != 0 and "Nonesuch" in r.stderr


# --------------------------------------------------------------------------- the oracle against its definitions

def test_oracle_recurrence_is_the_decayed_sum():
    rng = np.random.default_rng(0)
    T, H, d, dv = 9, 2, 3, 4
    q, k, a = rng.standard_normal((T, H, d)), rng.standard_normal((T, H, d)), rng.uniform(0.2, 1.0, (T, H, d))
    v = rng.standard_normal((T, H, dv))
    S = np.zeros((H, d, dv))
    o = L.decayed_outer_recurrence(q, k, v, a, S)
    for t in range(T):
        want = np.zeros((H, dv))
        for j in range(t + 1):
            w = np.prod(a[j + 1:t + 1], axis=0)
            want += np.sum(q[t] * k[j] * w, axis=1)[:, None] * v[j]
        assert np.allclose(o[t], want)


def test_oracle_rotation_depends_on_distance_only_and_leaves_the_rest():
    rng = np.random.default_rng(1)
    x, y = rng.standard_normal((1, 10)), rng.standard_normal((1, 10))
    f = lambda p, r: float((L.rotate_half(x, [p], 500.0, 6) @ L.rotate_half(y, [r], 500.0, 6).T)[0, 0])
    assert abs(f(3, 1) - f(40, 38)) < 1e-9 and abs(f(3, 1) - f(3, 2)) > 1e-3
    assert np.array_equal(L.rotate_half(x, [9], 500.0, 6)[:, 6:], x[:, 6:])
    z = np.zeros((1, 4)); z[0, 0] = 1.0
    assert np.allclose(L.rotate_half(z, [1], 1.0, 4)[0], [np.cos(1), 0, np.sin(1), 0])     # 0 is paired with 0 + 4/2


def test_oracle_window_edges():
    assert L.window_visible(10, 11, 4).tolist() == [7, 8, 9, 10]
    assert L.window_visible(2, 11, 4).tolist() == [0, 1, 2]
    assert L.window_visible(5, 11, 1).tolist() == [5]


def test_oracle_portions_equal_one_pass():
    cfg = U.config()
    t = U.as_numpy(U.random_tensors(cfg, seed=3))
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], 50).tolist()
    want = L.Model(cfg, t).run(toks)
    m = L.Model(cfg, t)
    got, at = [], 0
    for n in (7, 1, 2, 20, 1, 19):
        got.append(m.run(toks[at:at + n])); at += n
    assert np.allclose(np.concatenate(got), want, atol=1e-9)


def test_every_mechanism_reaches_the_logits():
    """Dropping any tensor's contribution (or changing a constant) moves the oracle's logits: random weights hide nothing."""
    cfg = U.config()
    t = U.as_numpy(U.random_tensors(cfg, seed=4))
    toks = np.random.default_rng(2).integers(0, cfg["vocab"], 40).tolist()
    base = L.Model(cfg, t).run(toks)
    for name in t:
        t2 = dict(t)
        t2[name] = t[name] * np.where(np.arange(t[name].shape[-1]) % 2, 0.7, 1.3)     # (a common factor may cancel in a norm)
        assert U.rel_rms(L.Model(cfg, t2).run(toks), base) > 1e-3, name
    import copy
    for path, f in ((("layers", 1, "mixer", "mask", "size"), lambda v: v + 1), (("layers", 1, "mixer", "scale"), lambda v: v * 1.3),
                    (("layers", 0, "mixer", "tau"), lambda v: v * 0.5), (("layers", 1, "mixer", "rot", "base"), lambda v: v * 0.1),
                    (("layers", 2, "mixer", "decay", 1), lambda v: v * 0.9), (("norm", "eps"), lambda v: 0.05),
                    (("embedding", "scale"), lambda v: v * 0.5)):
        c = copy.deepcopy(cfg)
        node = c
        for k in path[:-1]:
            node = node[k]
        node[path[-1]] = f(node[path[-1]])
        assert U.rel_rms(L.Model(c, t).run(toks), base) > 1e-3, path
