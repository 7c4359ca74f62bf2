"""GPU: every kernel of the mixer-layer models alone, against plain fp64 arithmetic, at ragged sizes."""
import ctypes

import numpy as np
import pytest
import torch

from llamatov_b200 import _lib, dense_ops as P
from oracle import layered as L
from tests.gpu_util import stream

pytestmark = pytest.mark.gpu
DT = {0: torch.bfloat16, 1: torch.float32}


@pytest.fixture(autouse=True)
def _clean_status():
    yield
    assert _lib.device_status() == set()


def _t(shape, seed, f32, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(shape, generator=g) * scale).to(DT[f32]).cuda()


def _np(t):
    return t.double().cpu().numpy()


def _close(got, want, tol, floor=0.0, rel=0.0):
    """tol relative to the root mean square of the wanted values, rel to each value (a rounded store)"""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    assert np.isfinite(got).all()
    rms = np.sqrt(np.mean(want * want)) + floor
    worst = float((np.abs(got - want) - rel * np.abs(want)).max() / rms)
    assert worst <= tol, worst


# --------------------------------------------------------------------------- linears

def _epi_ref(v, kind, act=None, scale=1.0, bias=None):
    if bias is not None:
        v = v + bias
    if act == "silu":
        v = L.silu(v)
    elif act == "sigmoid":
        v = L.sigmoid(v)
    elif act == "logsigmoid":
        v = np.log(L.sigmoid(v))
    return v * scale


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("M,K,T,variant", [(40, 24, 2, 0), (203, 80, 33, 0), (128, 64, 65, 32), (256, 200, 130, 64), (300, 136, 257, 128),
                                           (136, 520, 300, 256), (1000, 328, 700, 0)])
def test_linear_store_with_segments(f32, M, K, T, variant):
    W, X = _t((M, K), 1, f32, K ** -0.5), _t((T, K + 8), 2, f32)      # x rows lie in wider rows
    bias = torch.randn(M).cuda()
    s1, s2 = M // 3, M // 2
    e = P.epilogue(segs=[(s1, "silu", 1.0), (s2, None, 0.25), (M, "sigmoid", 1.0)], bias=bias)
    Y = torch.full((T, M + 4), 7.0, dtype=DT[f32], device="cuda")
    _lib.call("lt_dn_linear", W.data_ptr(), K, X.data_ptr(), K + 8, Y.data_ptr(), M + 4, f32, M, K, T, ctypes.byref(e), variant, stream())
    v = _np(X)[:, :K] @ _np(W).T + _np(bias)
    want = np.concatenate([L.silu(v[:, :s1]), v[:, s1:s2] * 0.25, L.sigmoid(v[:, s2:])], axis=1)
    _close(_np(Y)[:, :M], want, 2e-6 * K ** 0.5 if f32 else 1e-3, rel=0 if f32 else 2 ** -8)
    assert (_np(Y)[:, M:] == 7.0).all()


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("M,K,T", [(48, 40, 3), (200, 264, 129), (520, 128, 600)])
def test_linear_residual_logsigmoid_and_gated(f32, M, K, T):
    W, X = _t((M, K), 3, f32, K ** -0.5), _t((T, K), 4, f32)
    ls = torch.randn(M).cuda()
    Y = torch.randn(T, M).cuda()
    y0 = _np(Y)
    e = P.epilogue(_lib.DN_RESID, ls=ls)
    _lib.call("lt_dn_linear", W.data_ptr(), K, X.data_ptr(), K, Y.data_ptr(), M, f32, M, K, T, ctypes.byref(e), 0, stream())
    v = _np(X) @ _np(W).T
    _close(_np(Y), y0 + v * _np(ls), 1e-5)          # fp32 in both types: operands are exact
    e = P.epilogue(segs=[(M, "logsigmoid", 0.5)], out_f32=True)
    Z = torch.empty(T, M, device="cuda")
    _lib.call("lt_dn_linear", W.data_ptr(), K, X.data_ptr(), K, Z.data_ptr(), M, f32, M, K, T, ctypes.byref(e), 0, stream())
    _close(_np(Z), np.log(L.sigmoid(v)) * 0.5, 1e-5)
    U = _t((2 * M, K), 5, f32, K ** -0.5)
    e = P.epilogue(_lib.DN_GLU, out_f32=True)
    for variant in (0, 32, 64, 128):
        Z.zero_()
        _lib.call("lt_dn_linear", U.data_ptr(), K, X.data_ptr(), K, Z.data_ptr(), M, f32, M, K, T, ctypes.byref(e), variant, stream())
        u = _np(X) @ _np(U).T
        _close(_np(Z), L.gelu_tanh(u[:, :M]) * u[:, M:], 1e-5)


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("M,K", [(1, 8), (40, 24), (203, 80), (600, 1032), (97, 4104)])
def test_gemv_prologues(f32, M, K):
    W = _t((M, K), 6, f32, K ** -0.5)
    x, x2 = torch.randn(K).cuda(), torch.randn(K).cuda()
    w = torch.rand(K).cuda() + 0.5
    gate = _t((K,), 7, f32)
    Y = torch.empty(M, device="cuda")
    e = P.epilogue(out_f32=True)
    tol = 2e-6 * K ** 0.5 if f32 else 3e-2
    run = lambda pro: (_lib.call("lt_dn_gemv", W.data_ptr(), K, Y.data_ptr(), f32, M, K, ctypes.byref(pro), ctypes.byref(e), stream()), _np(Y))[1]
    xt = _t((K,), 8, f32)
    _close(run(P.typed_input(xt.data_ptr())), _np(W) @ _np(xt), 1e-5)
    n1 = 4 * (K // 8)
    cat = np.concatenate([_np(x)[:n1], _np(x2)[:K - n1]])
    _close(run(P.cast_input(x.data_ptr(), n1, x2.data_ptr())), _np(W) @ cat, tol, 0.1)
    count = K - 3           # as with three padding elements: the mean counts the real ones
    n = P.Norm(w.cpu(), count, K, 1e-5)
    nx = _np(x) / np.sqrt((_np(x) ** 2).sum() / count + 1e-5) * _np(w)
    _close(run(n.prologue(x.data_ptr())), _np(W) @ nx, tol, 0.1)
    _close(run(n.prologue(x.data_ptr(), gate.data_ptr())), _np(W) @ (nx * _np(gate)), tol, 0.1)
    n = P.Norm(w[:8].cpu(), 7, 8, 1e-5)
    g = _np(x).reshape(-1, 8)
    gx = (g / np.sqrt((g ** 2).sum(1, keepdims=True) / 7 + 1e-5) * _np(w)[:8]).reshape(-1)
    _close(run(n.prologue(x.data_ptr(), gate.data_ptr())), _np(W) @ (gx * _np(gate)), tol, 0.1)
    # residual and gated epilogues
    r = torch.randn(M).cuda(); r0 = _np(r); ls = torch.randn(M).cuda()
    e2 = P.epilogue(_lib.DN_RESID, ls=ls)
    pro = P.typed_input(xt.data_ptr())
    _lib.call("lt_dn_gemv", W.data_ptr(), K, r.data_ptr(), f32, M, K, ctypes.byref(pro), ctypes.byref(e2), stream())
    _close(_np(r), r0 + _np(ls) * (_np(W) @ _np(xt)), 1e-5, 0.1)
    U = _t((2 * M, K), 9, f32, K ** -0.5)
    e3 = P.epilogue(_lib.DN_GLU, out_f32=True)
    _lib.call("lt_dn_gemv", U.data_ptr(), K, Y.data_ptr(), f32, M, K, ctypes.byref(pro), ctypes.byref(e3), stream())
    u = _np(U) @ _np(xt)
    _close(_np(Y), L.gelu_tanh(u[:M]) * u[M:], 1e-5, 0.1)


@pytest.mark.parametrize("f32", [0, 1])
def test_row_operators(f32):
    T, N = 5, 72
    x = torch.randn(T, N).cuda()
    w = torch.rand(N).cuda() + 0.5
    y = torch.empty(3, N, dtype=DT[f32], device="cuda")
    idx = torch.tensor([4, 0, 2], dtype=torch.int32).cuda()
    P.Norm(w.cpu(), N, N, 1e-6).rows(x.data_ptr(), N, y.data_ptr(), N, f32, 3, N, index=idx.data_ptr())
    _close(_np(y), L.rms(_np(x), _np(w), 1e-6)[[4, 0, 2]], 1e-6 if f32 else 2e-2)
    gate = _t((T, N + 8), 3, f32)
    y = torch.empty(T, N, dtype=DT[f32], device="cuda")
    P.Norm(w[:24].cpu(), 20, 24, 1e-6).rows(x.data_ptr(), N, y.data_ptr(), N, f32, T, N, gate=gate.data_ptr(), ldg=N + 8)
    g = _np(x).reshape(T, 3, 24)
    want = (g / np.sqrt((g ** 2).sum(-1, keepdims=True) / 20 + 1e-6) * _np(w)[:24]).reshape(T, N) * _np(gate)[:, :N]
    _close(_np(y), want, 2e-6 if f32 else 2e-2)
    tab = _t((9, 13), 4, f32)
    tok = torch.tensor([8, 0, 3], dtype=torch.int32).cuda()
    a, b = torch.full((3, 16), 5.0).cuda(), torch.full((3, 16), 5.0).cuda()
    _lib.call("lt_dn_embed", tab.data_ptr(), f32, 13, tok.data_ptr(), 3.5, None, 0.0, a.data_ptr(), b.data_ptr(), 13, 16, 9, 3, stream())
    _close(_np(a)[:, :13], _np(tab)[[8, 0, 3]] * 3.5, 1e-6)
    assert torch.equal(a, b) and (a[:, 13:] == 0).all()
    _lib.call("lt_dn_embed", tab.data_ptr(), f32, 13, torch.tensor([9], dtype=torch.int32).cuda().data_ptr(), 1.0, None, 0.0, a.data_ptr(), None, 13, 16,
              9, 1, stream())
    assert _lib.device_status() == {"bad_token"}
    y = torch.empty(3, 40, dtype=DT[f32], device="cuda")
    _lib.call("lt_dn_concat_rows", a.data_ptr(), 16, 16, x.data_ptr(), N, 24, y.data_ptr(), 40, f32, 3, stream())
    _close(_np(y), np.concatenate([_np(a), _np(x)[:3, :24]], axis=1), 1e-2)


# --------------------------------------------------------------------------- recurrence

def _recur_case(T, H, dp, dvp, f32, kind, seed=0, strong=1.0):
    """inputs and the fp64 answer; kind: const | log"""
    ld = H * (2 * dp + dvp) + 8
    y = _t((T, ld), seed, f32, dp ** -0.25)
    S = torch.randn(H, dvp, dp, generator=torch.Generator().manual_seed(seed + 1)).cuda()
    dec = _lib.DnDecay()
    keep = [y]
    if kind == "const":
        lam = torch.tensor(np.concatenate([[0.0, 1.0, 0.999], np.random.default_rng(seed).uniform(0.3, 0.99, 16)])[:H], dtype=torch.float32).cuda()
        dec.decay = lam.data_ptr()
        a = np.broadcast_to(_np(lam)[None, :, None], (T, H, dp))
        keep.append(lam)
    else:
        la = -(torch.rand(T, H * dp, generator=torch.Generator().manual_seed(seed + 2)) ** 4) * strong
        la = la.cuda()
        dec.la, dec.ldla = la.data_ptr(), H * dp
        a = np.exp(_np(la)).reshape(T, H, dp)
        keep.append(la)
    yn = _np(y)
    q, k = yn[:, :H * dp].reshape(T, H, dp), yn[:, H * dp:2 * H * dp].reshape(T, H, dp)
    v = yn[:, 2 * H * dp:2 * H * dp + H * dvp].reshape(T, H, dvp)
    Sn = np.transpose(_np(S), (0, 2, 1)).copy()
    o = L.decayed_outer_recurrence(q, k, v, a, Sn)
    return y, ld, S, dec, keep, o.reshape(T, H * dvp), np.transpose(Sn, (0, 2, 1))


def _ptrs(y, H, dp):
    e = y.element_size()
    return y.data_ptr(), y.data_ptr() + H * dp * e, y.data_ptr() + 2 * H * dp * e


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("kind", ["const", "log"])
@pytest.mark.parametrize("T,H,dp,dvp", [(1, 3, 16, 24), (2, 2, 48, 40), (17, 1, 8, 8), (40, 3, 128, 72), (33, 2, 136, 16), (20, 1, 264, 40)])
def test_recurrence_scan(f32, kind, T, H, dp, dvp):
    y, ld, S, dec, keep, o, Sn = _recur_case(T, H, dp, dvp, f32, kind, strong=5.0)
    out = torch.full((T, H * dvp + 4), 9.0, device="cuda")
    q, k, v = _ptrs(y, H, dp)
    _lib.call("lt_dn_recurrence", q, k, v, ld, S.data_ptr(), out.data_ptr(), H * dvp + 4, f32, T, H, dp, dvp, ctypes.byref(dec), stream())
    _close(_np(out)[:, :H * dvp], o, 1e-5)
    assert (_np(out)[:, H * dvp:] == 9.0).all()
    _close(_np(S), Sn, 1e-5)


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("rank,tau", [(8, 16.0), (24, 1.0)])
def test_recurrence_low_rank_decay(f32, rank, tau):
    H, dp, dvp = 2, 40, 16
    y, ld, S, dec, keep, _o, _s = _recur_case(1, H, dp, dvp, f32, "const")
    S0 = np.transpose(_np(S), (0, 2, 1)).copy()
    a1, a2, b = _t((rank,), 5, f32), _t((H * dp, rank), 6, f32), torch.randn(H * dp).cuda()
    dec = _lib.DnDecay()
    dec.a1, dec.a2, dec.lda2, dec.rank, dec.bias, dec.inv_tau = a1.data_ptr(), a2.data_ptr(), rank, rank, b.data_ptr(), 1.0 / tau
    out = torch.empty(1, H * dvp, device="cuda")
    q, k, v = _ptrs(y, H, dp)
    _lib.call("lt_dn_recurrence", q, k, v, ld, S.data_ptr(), out.data_ptr(), H * dvp, f32, 1, H, dp, dvp, ctypes.byref(dec), stream())
    alpha = (L.sigmoid(_np(a2) @ _np(a1) + _np(b)) ** (1.0 / tau)).reshape(1, H, dp)
    yn = _np(y)[0]
    o = L.decayed_outer_recurrence(yn[:H * dp].reshape(1, H, dp), yn[H * dp:2 * H * dp].reshape(1, H, dp),
                                   yn[2 * H * dp:2 * H * dp + H * dvp].reshape(1, H, dvp), alpha, S0)
    _close(_np(out), o.reshape(1, -1), 2e-5)
    _close(_np(S), np.transpose(S0, (0, 2, 1)), 2e-5)


@pytest.mark.parametrize("kind,strong", [("const", 0), ("log", 0.05), ("log", 1.0), ("log", 12.0), ("log", 90.0)])
@pytest.mark.parametrize("T,H,dp,dvp", [(64, 2, 64, 64), (65, 3, 48, 32), (130, 2, 128, 128), (200, 1, 24, 40), (16, 2, 8, 8), (150, 2, 200, 136),
                                        (96, 1, 256, 256), (321, 4, 40, 24)])
def test_recurrence_chunked(kind, strong, T, H, dp, dvp):
    """Gentle and violent decays: with strong ones a block's exponents leave the safe range and are summed pair by pair."""
    y, ld, S, dec, keep, o, Sn = _recur_case(T, H, dp, dvp, 0, kind, strong=strong)
    out = torch.full((T, H * dvp + 4), 9.0, device="cuda")
    ws = torch.full((_lib.dense().lt_dn_recurrence_chunked_ws(T, H, dp, dvp),), float("nan"), device="cuda")
    q, k, v = _ptrs(y, H, dp)
    _lib.call("lt_dn_recurrence_chunked", q, k, v, ld, S.data_ptr(), out.data_ptr(), H * dvp + 4, T, H, dp, dvp, ctypes.byref(dec),
              ws.data_ptr(), stream())
    _close(_np(out)[:, :H * dvp], o, 1e-4)
    assert (_np(out)[:, H * dvp:] == 9.0).all()
    _close(_np(S), Sn, 1e-4)


def test_recurrence_chunked_recalls_one_far_key():
    """A value stored at token 3 under its own key channel is read back 200 tokens later with the decay it should have."""
    T, H, dp, dvp = 256, 1, 32, 16
    ld = 2 * dp + dvp
    y = torch.zeros(T, ld)
    y[3, dp + 5] = 1.0                       # k_3 = e_5
    y[3, 2 * dp:] = torch.arange(dvp) + 1.0
    y[203, 5] = 1.0                          # q_203 = e_5
    y = y.bfloat16().cuda()
    la = torch.full((T, dp), -0.01).cuda()
    dec = _lib.DnDecay(); dec.la, dec.ldla = la.data_ptr(), dp
    S = torch.zeros(H, dvp, dp).cuda()
    o = torch.empty(T, dvp, device="cuda")
    ws = torch.empty(_lib.dense().lt_dn_recurrence_chunked_ws(T, H, dp, dvp), device="cuda")
    q, k, v = _ptrs(y, H, dp)
    _lib.call("lt_dn_recurrence_chunked", q, k, v, ld, S.data_ptr(), o.data_ptr(), dvp, T, H, dp, dvp, ctypes.byref(dec), ws.data_ptr(), stream())
    want = np.zeros((T, dvp)); want[203] = (np.arange(dvp) + 1) * np.exp(-2.0)
    assert np.abs(_np(o) - want).max() < 1e-4


# --------------------------------------------------------------------------- latent attention

class _Latent:
    def __init__(self, f32, H=3, d=24, r=16, dv=40, rank=32, window=19, cap=64, base=1000.0, scale=0.3, seed=0):
        self.f32, self.H, self.d, self.r, self.dv, self.rank, self.window, self.cap = f32, H, d, r, dv, rank, window, cap
        self.base, self.scale = base, scale
        dt = DT[f32]
        g = torch.Generator().manual_seed(seed)
        self.freq = (base ** (-2.0 * torch.arange(r // 2, dtype=torch.float64) / r)).float().cuda()
        self.cnorm = (torch.rand(rank, generator=g) + 0.5).cuda()
        self.uk = (torch.randn(H * d, rank, generator=g) * rank ** -0.5).to(dt).cuda()
        self.uv = (torch.randn(H * dv, rank, generator=g) * rank ** -0.5).to(dt).cuda()
        self.ukT = self.uk.reshape(H, d, rank).transpose(1, 2).contiguous()
        self.expand = torch.cat([self.uk, self.uv]).contiguous()
        self.desc = _lib.DnLatent(H, d, r, dv, r, rank, rank, window, cap, scale, 1e-6, self.freq.data_ptr(), self.cnorm.data_ptr())
        self.width = H * (d + r) + rank + r
        self.ring = torch.full((cap, rank + r), float("nan"), dtype=dt, device="cuda")
        self.len = torch.zeros(1, dtype=torch.int32, device="cuda")
        self.pos = 0
        self.cache = {"c": [], "kr": []}

    def rows(self, y):
        """a portion: y [T, width] (rotated in place); returns the heads' outputs"""
        T, np_ = y.shape[0], min(self.window - 1, self.pos)
        nk, wr, dt = np_ + T, self.rank + self.r, DT[self.f32]
        keys = torch.empty(nk, wr, dtype=dt, device="cuda")
        nkv = self.H * (self.d + self.dv)
        kv = torch.empty(nk, nkv, dtype=dt, device="cuda")
        out = torch.empty(T, self.H * self.dv, dtype=dt, device="cuda")
        e = y.element_size()
        d = ctypes.byref(self.desc)
        _lib.call("lt_dn_latent_rows", y.data_ptr(), self.width, self.ring.data_ptr(), keys.data_ptr(), np_, self.pos, self.f32, T, d, stream())
        ep = P.epilogue()
        _lib.call("lt_dn_linear", self.expand.data_ptr(), self.rank, keys.data_ptr(), wr, kv.data_ptr(), nkv, self.f32, nkv, self.rank, nk,
                  ctypes.byref(ep), 0, stream())
        _lib.call("lt_dn_window_attn", y.data_ptr(), self.width, kv.data_ptr(), nkv, keys.data_ptr() + self.rank * e, wr,
                  kv.data_ptr() + self.H * self.d * e, nkv, out.data_ptr(), self.H * self.dv, self.f32, T, np_, d, stream())
        self.pos += T
        self.len.fill_(self.pos)
        return _np(out)

    def step(self, y, splits):
        out = torch.empty(self.H * self.dv, dtype=DT[self.f32], device="cuda")
        ws = torch.full((_lib.dense().lt_dn_latent_step_ws(self.H, self.rank, self.r, splits),), float("nan"), device="cuda")
        _lib.call("lt_dn_latent_step", y.data_ptr(), self.ring.data_ptr(), self.len.data_ptr(), self.ukT.data_ptr(), self.uv.data_ptr(),
                  out.data_ptr(), self.f32, ctypes.byref(self.desc), splits, ws.data_ptr(), stream())
        self.pos += 1
        assert int(self.len.item()) == self.pos
        return _np(out).reshape(1, -1)

    def oracle(self, y, pos0):
        """the same from the untouched projections, through the oracle's mechanism with identity projections"""
        eye = np.eye(self.width)
        nq = self.H * (self.d + self.r)
        w = {"q": eye[:nq], "dkv": eye[nq:], "dkv.norm": _np(self.cnorm), "uk": _np(self.uk), "uv": _np(self.uv), "o": np.eye(self.H * self.dv)}
        m = {"heads": self.H, "dim": self.d, "rot_dim": self.r, "vdim": self.dv, "kv_rank": self.rank, "mask": {"size": self.window},
             "rot": {"base": self.base, "dims": self.r}, "scale": self.scale}
        return L.latent_attention(y, m, lambda n: w[n], 1e-6, self.cache, pos0)


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("kw", [dict(), dict(window=1), dict(window=2, H=1, d=8, r=8, dv=8, rank=8), dict(window=64, cap=120, dv=136, d=64, r=32),
                                dict(window=33, cap=80, H=11, d=16, r=8, dv=64, rank=264), dict(window=500, cap=600, rank=520, H=2, dv=24),
                                dict(window=70, cap=140, d=128, r=64, dv=128, rank=128, H=2)])
def test_latent_portions_and_single_tokens(f32, kw):
    """Portions of many sizes and single tokens through a small ring that wraps several times."""
    A = _Latent(f32, **kw)
    rng = np.random.default_rng(5)
    cap_T = A.cap - A.window + 1
    sizes = [min(cap_T, s) for s in (3, 1, 2, 37, 1, 1, 64, 65, 1, 5, 2)]
    for n, T in enumerate(sizes):
        y = _t((T, A.width), 100 + n, f32)
        want = A.oracle(_np(y), A.pos)
        splits = int(rng.integers(1, 12))
        got = A.step(y, splits) if T == 1 else A.rows(y)
        if f32:
            _close(got, want, 5e-5)
        else:       # the rounded latents, keys, values and queries add up: small on average, never far off
            _close(got, want, 0.1)
            assert np.sqrt(np.mean((got - want) ** 2)) < 1e-2 * np.sqrt(np.mean(want ** 2))


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("T", [1, 30])
def test_window_edge_shows(f32, T):
    """One key outshines all others.  The query at exactly window - 1 tokens' distance returns its value, the next query
    does not see it."""
    W = 21
    A = _Latent(f32, H=2, d=16, r=8, dv=16, rank=16, window=W, cap=96, scale=1.0)
    A.uk.zero_(); A.uv.zero_()
    for h in range(2):
        A.uk[h * 16:(h + 1) * 16] = torch.eye(16); A.uv[h * 16:(h + 1) * 16] = torch.eye(16)
    A.ukT.copy_(A.uk.reshape(2, 16, 16).transpose(1, 2)); A.expand.copy_(torch.cat([A.uk, A.uv]))
    A.cnorm.fill_(1.0)
    n, star = 70, 25
    y = torch.zeros(n, A.width)
    for t in range(n):
        for h in range(2):
            y[t, h * 24 + 3] = 20.0                # every query asks for channel 3
        y[t, 48 + (3 if t == star else 7)] = 1.0   # only the star's latent has it (normed: 4 in one channel)
    y = y.to(DT[f32]).cuda()
    outs, at = [], 0
    while at < n:
        c = 1 if T == 1 else min(T, n - at)
        outs.append(A.step(y[at:at + 1].clone(), 3) if T == 1 else A.rows(y[at:at + c].clone()))
        at += c
    o = np.concatenate(outs)
    for t in range(n):
        sees = 0 <= t - star < W
        assert abs(o[t, 3] - (4.0 if sees else 0.0)) < 0.05, (t, o[t, 3])
        assert abs(o[t, 16 + 7] - (0.0 if sees else 4.0)) < 0.05, (t, o[t, 23])
