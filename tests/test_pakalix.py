"""CPU: configuration and packing of the Pakalix models, and the consistency of their plain restatement."""
import copy

import numpy as np
import pytest
import torch

from oracle import pakalix as O
from tests import layered_util as U
from tests import pakalix_util as K


def test_loader_reads_the_design(tmp_path):
    from llamatov_b200 import archs, layered
    from llamatov_b200 import llamatov_run as R
    cfg = K.config()
    c, w = R.load_model(U.write_model(tmp_path / "m", cfg, K.random_tensors(cfg)), dtype="float32")
    assert archs.of(c) is layered.PAKALIX
    assert (c["n_layers"], c["residual_mult"], c["norm_eps"], c["loop"], c["embed_scale"]) == (5, 0.6, 1e-5, None, 1.0)
    assert w["l1.mix.vmix"].shape == () and [r.slot for r in archs.of(c).runs(c)] == [0, 1, 2, 3, 4]
    assert layered.ARCH.norm_offset == 0.0 and not layered.ARCH.embed_norm          # the other design is as it was


def test_argument_validation_without_gpu():
    import ctypes
    from llamatov_b200 import _lib
    lib = _lib.dense()
    one = ctypes.c_void_p(256)     # never dereferenced: validation fails first
    a = _lib.DnGqa(6, 4, 16, 16, 8, 96, 64, 10, 1.0, 0.0, 1e-5, 0.0, 256, 256, 256)
    assert lib.lt_dn_gqa_rows(one, 256, one, one, None, 0, 0, 2, 0, ctypes.byref(a), None) == 1 and "heads" in _lib.last_error()
    a.G = 3
    assert lib.lt_dn_gqa_rows(one, 256, one, one, None, 0, 0, 5, 6, ctypes.byref(a), None) == 1 and "cache of 10" in _lib.last_error()
    assert lib.lt_dn_gqa_attn(one, 256, one, one, None, 0, one, 96, 0, 5, 6, ctypes.byref(a), None) == 1
    a.softcap = -1.0
    assert lib.lt_dn_gqa_step(one, one, one, None, 0, None, one, 0, one, ctypes.byref(a), 2, one, one, None) == 1
    assert "softcap" in _lib.last_error()
    s = _lib.DnSsd(6, 4, 16, 16, 3, 256, 256, 256, 256, 256)
    assert lib.lt_dn_ssd_step(one, one, one, one, one, 0, one, one, ctypes.byref(s), None) == 1
    e = _lib.DnEpilogue()
    e.kind = _lib.DN_STORE_GLU
    assert lib.lt_dn_linear(one, 16, one, 16, one, 8, 0, 8, 16, 4, ctypes.byref(e), 0, None) == 1
    d = _lib.DnDecay()
    d.hla, d.hdt, d.D, d.ldh, d.per = 256, 256, 256, 6, 4
    assert lib.lt_dn_recurrence(one, one, one, 64, one, one, 64, 0, 5, 6, 16, 16, ctypes.byref(d), None) == 1
    assert "groups of 4" in _lib.last_error()


# --------------------------------------------------------------------------- the oracle against its definitions

def test_causal_conv_carries_its_inputs():
    rng = np.random.default_rng(0)
    u, taps, b = rng.standard_normal((11, 3)), rng.standard_normal((3, 4)), rng.standard_normal(3)
    whole, _ = O.causal_conv(u, taps, b, np.zeros((3, 3)))
    for t in range(11):
        want = b + sum(taps[:, 3 - i] * u[t - i] for i in range(4) if t - i >= 0)
        assert np.allclose(whole[t], want)
    before, parts = np.zeros((3, 3)), []
    for lo, hi in ((0, 1), (1, 3), (3, 4), (4, 11)):
        y, before = O.causal_conv(u[lo:hi], taps, b, before)
        parts.append(y)
    assert np.allclose(np.concatenate(parts), whole)
    y, before = O.causal_conv(u, taps[:, :1], b, np.zeros((0, 3)))      # one tap: nothing to carry
    assert np.allclose(y, b + taps[:, 0] * u) and before.shape == (0, 3)


def test_ssd_recurrence_is_the_decayed_sum():
    rng = np.random.default_rng(1)
    T, H, G, N, P = 8, 4, 2, 3, 5
    x, B, C = rng.standard_normal((T, H, P)), rng.standard_normal((T, G, N)), rng.standard_normal((T, G, N))
    dt, A, D = rng.uniform(0.1, 2.0, (T, H)), -rng.uniform(0.1, 2.0, H), rng.standard_normal(H)
    y = O.ssd_recurrence(x, B, C, dt, A, D, np.zeros((H, N, P)))
    for t in range(T):
        for h in range(H):
            want = D[h] * x[t, h]
            for j in range(t + 1):
                want = want + np.exp(A[h] * dt[j + 1:t + 1, h].sum()) * dt[j, h] * (C[t, h // 2] @ B[j, h // 2]) * x[j, h]
            assert np.allclose(y[t, h], want)


def test_norm_in_parts_and_softplus():
    y = np.arange(1.0, 13.0).reshape(1, 12)
    o = O.rms_in_parts(y, np.ones(12), 3, 0.0)
    assert np.allclose((o.reshape(3, 4) ** 2).mean(axis=1), 1.0)
    assert np.allclose(O.softplus([-800.0, 0.0, 800.0]), [0.0, np.log(2), 800.0])


def test_capped_scores_and_clamped_feed_forward():
    assert abs(O.capped(1e-3, 5.0) - 1e-3) < 1e-9 and O.capped(1e3, 5.0) == pytest.approx(5.0)
    w = {"gate": np.eye(2), "up": np.eye(2), "down": np.eye(2)}
    y = O.clamped_feed_forward(np.array([[9.0, -9.0]]), lambda n: w[n], 0.5)
    sg = lambda z: 1 / (1 + np.exp(-z))
    assert np.allclose(y, [[0.5 * sg(1.702 * 0.5) * 1.5, -9 * sg(-1.702 * 9) * 0.5]])       # the gate has no lower bound


def test_first_value_mixing_layer_keeps_its_own_values():
    cfg = K.config()
    t = U.as_numpy(K.random_tensors(cfg, seed=2))
    toks = list(range(9))
    base = O.Model(cfg, t).run(toks)
    for name, moves in (("l1.mix.vmix", False), ("l3.mix.vmix", True)):
        t2 = dict(t)
        t2[name] = t[name] * 0 + 0.9
        assert (U.rel_rms(O.Model(cfg, t2).run(toks), base) > 1e-3) == moves, name


def test_portions_equal_one_pass():
    cfg = K.config()
    t = U.as_numpy(K.random_tensors(cfg, seed=3))
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], 40).tolist()
    want = O.Model(cfg, t).run(toks)
    m, got, at = O.Model(cfg, t), [], 0
    for n in (7, 1, 2, 20, 1, 9):
        got.append(m.run(toks[at:at + n])); at += n
    assert np.allclose(np.concatenate(got), want, atol=1e-9)


def test_every_mechanism_reaches_the_logits():
    """Changing any tensor or constant moves the oracle's logits: the random weights hide nothing."""
    cfg = K.config()
    t = U.as_numpy(K.random_tensors(cfg, seed=4))
    toks = np.random.default_rng(2).integers(0, cfg["vocab"], 30).tolist()
    base = O.Model(cfg, t).run(toks)
    for name in t:
        if name == "l1.mix.vmix":
            continue                          # of the first mixing layer: unused
        t2 = dict(t)
        n = t[name].shape[-1] if t[name].ndim else 1
        f = np.where(np.arange(n) % 2, 0.6, 1.4)
        t2[name] = t[name] * (f if t[name].ndim else 1.4) + (0.05 if name.endswith(("norm", "norm1")) else 0.0)
        assert U.rel_rms(O.Model(cfg, t2).run(toks), base) > 5e-4, name
    for path, f in ((("layers", 1, "mixer", "scale"), lambda v: v * 1.3), (("layers", 1, "mixer", "softcap"), lambda v: v * 0.3),
                    (("layers", 1, "mixer", "rot", "base"), lambda v: v * 0.1), (("layers", 1, "mixer", "rot", "dims"), lambda v: v - 4),
                    (("layers", 0, "mixer", "norm_groups"), lambda v: 1), (("layers", 0, "mlp", "limit"), lambda v: v * 0.7),
                    (("layers", 3, "mixer", "v_mix"), lambda v: False), (("norm", "eps"), lambda v: 0.05), (("residual_mult",), lambda v: v * 0.8)):
        c = copy.deepcopy(cfg)
        node = c
        for k in path[:-1]:
            node = node[k]
        node[path[-1]] = f(node[path[-1]])
        assert U.rel_rms(O.Model(c, t).run(toks), base) > 5e-4, path


def test_frequencies_as_two_floats():
    """hi + lo is the frequency to far below fp32 rounding, so that angles at far positions keep their fraction."""
    f = 7000.0 ** (-2.0 * torch.arange(12, dtype=torch.float64) / 24)
    hi = f.float()
    lo = (f - hi.double()).float()
    assert ((hi.double() + lo.double() - f).abs() / f).max() < 2.0 ** -46
