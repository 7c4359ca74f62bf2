"""GPU: every kernel that the Pakalix models add or extend, alone, against plain fp64 arithmetic, at ragged sizes."""
import ctypes

import numpy as np
import pytest
import torch

from llamatov_b200 import _lib, dense_ops as P
from oracle import layered as L
from oracle import pakalix as O
from tests.gpu_util import stream
from tests.test_gpu_layered_kernels import DT, _close, _np, _t

pytestmark = pytest.mark.gpu


@pytest.fixture(autouse=True)
def _clean_status():
    yield
    assert _lib.device_status() == set()


def _glu(g, u, limit):
    return O.clamped_feed_forward(np.concatenate([g, u], axis=1),
                                  lambda n: {"gate": np.eye(2 * g.shape[1])[:g.shape[1]], "up": np.eye(2 * g.shape[1])[g.shape[1]:],
                                             "down": np.eye(g.shape[1])}[n], limit)


# --------------------------------------------------------------------------- linears

@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("M,tail,K,T,variant", [(40, 3, 24, 2, 0), (200, 17, 80, 70, 0), (128, 128, 64, 65, 32), (256, 5, 200, 130, 128),
                                                (8, 1, 8, 300, 256)])
def test_linear_with_an_fp32_tail(f32, M, tail, K, T, variant):
    W, X = _t((M + tail, K), 1, f32, K ** -0.5), _t((T, K), 2, f32)
    e = P.with_tail(P.epilogue(segs=[(8, "silu", 1.0), (M, None, 1.0), (M + tail, "sigmoid", 1.0)], tail_from=M), None, 1)
    Y = torch.full((T, M + 8), 7.0, dtype=DT[f32], device="cuda")
    Z = torch.full((T, tail + 2), 7.0, device="cuda")
    e = P.with_tail(e, Z.data_ptr(), tail + 2)
    _lib.call("lt_dn_linear", W.data_ptr(), K, X.data_ptr(), K, Y.data_ptr(), M + 8, f32, M + tail, K, T, ctypes.byref(e), variant, stream())
    v = _np(X) @ _np(W).T
    _close(_np(Y)[:, :M], np.concatenate([L.silu(v[:, :8]), v[:, 8:M]], axis=1), 2e-6 * K ** 0.5 if f32 else 1e-3, rel=0 if f32 else 2 ** -8)
    _close(_np(Z)[:, :tail], L.sigmoid(v[:, M:]), 1e-5)          # fp32 in both types
    assert (_np(Y)[:, M:] == 7.0).all() and (_np(Z)[:, tail:] == 7.0).all()


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("M,K,T", [(48, 40, 1), (200, 264, 129)])
def test_clamped_gate(f32, M, K, T):
    U, X = _t((2 * M, K), 5, f32, 2 * K ** -0.5), _t((T, K), 4, f32)
    u = _np(X) @ _np(U).T
    for limit in (0.4, 1.0, 7.0):
        want = _glu(u[:, :M], u[:, M:], limit)
        e = P.epilogue(_lib.DN_GLU, glu=(_lib.DN_GLU_CLAMPED, 1.702, limit))
        Y = torch.empty(T, M, dtype=DT[f32], device="cuda")
        for variant in (0, 32, 128):
            _lib.call("lt_dn_linear", U.data_ptr(), K, X.data_ptr(), K, Y.data_ptr(), M, f32, M, K, T, ctypes.byref(e), variant, stream())
            _close(_np(Y), want, 2e-5 if f32 else 2e-3, rel=0 if f32 else 2 ** -8)
        pro = P.typed_input(X.data_ptr())
        _lib.call("lt_dn_gemv", U.data_ptr(), K, Y.data_ptr(), f32, M, K, ctypes.byref(pro), ctypes.byref(e), stream())
        _close(_np(Y)[0], want[0], 2e-5 if f32 else 2e-3, rel=0 if f32 else 2 ** -8)


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("M,tail,F,K", [(40, 3, 24, 80), (16, 4, 8, 24), (203, 1, 120, 1032), (8, 0, 300, 64), (9, 0, 16, 64)])
def test_gemv_stored_and_gated_rows_in_one_launch(f32, M, tail, F, K):
    W = _t((M + tail + 2 * F, K), 6, f32, 1.5 * K ** -0.5)
    x = torch.randn(K).cuda()
    nm = P.Norm(torch.ones(K), K, K, 1e-5)
    e = P.epilogue(_lib.DN_STORE_GLU, segs=[(M, None, 1.0), (M + tail, "sigmoid", 1.0)], glu=(_lib.DN_GLU_CLAMPED, 1.702, 1.1),
                   tail_from=M if tail else None)
    Y, Z = torch.full((M + 3,), 7.0, dtype=DT[f32], device="cuda"), torch.full((tail + 1,), 7.0, device="cuda")
    G = torch.full((F + 3,), 7.0, dtype=DT[f32], device="cuda")
    if tail:
        e = P.with_tail(e, Z.data_ptr(), tail)
    e.glu_from, e.y2 = M + tail, G.data_ptr()
    pro = nm.prologue(x.data_ptr())
    _lib.call("lt_dn_gemv", W.data_ptr(), K, Y.data_ptr(), f32, M + tail + F, K, ctypes.byref(pro), ctypes.byref(e), stream())
    xn = _np(torch.from_numpy(L.rms(_np(x), 1.0, 1e-5)).to(DT[f32]))
    v = _np(W) @ xn
    _close(_np(Y)[:M], v[:M], 1e-2 if not f32 else 1e-5, rel=0 if f32 else 2 ** -8)
    if tail:
        _close(_np(Z)[:tail], L.sigmoid(v[M:M + tail]), 1e-5 if f32 else 5e-3)
    g, u = v[M + tail:M + tail + F], v[M + tail + F:]
    _close(_np(G)[:F], _glu(g[None], u[None], 1.1)[0], 1e-2 if not f32 else 3e-5, rel=0 if f32 else 2 ** -8)
    assert (_np(Y)[M:] == 7.0).all() and (_np(Z)[tail:] == 7.0).all() and (_np(G)[F:] == 7.0).all()


# heads of `P` (padded to Pp), `parts` norm groups over all of them
PARTS = [(4, 16, 1), (4, 16, 4), (4, 16, 2), (6, 20, 3), (6, 20, 4), (3, 5, 5), (8, 8, 16), (5, 12, 1), (2, 6, 3)]


def _gated(H, Pn, parts, f32, T, seed):
    Pp, n = P.pad8(Pn), H * Pn
    mask = np.zeros((H, Pp), bool); mask[:, :Pn] = True
    mask = mask.reshape(-1)
    o, z = torch.randn(T, H * Pp, generator=torch.Generator().manual_seed(seed)), _t((T, H * Pp + 8), seed + 1, f32)
    o[:, ~torch.from_numpy(mask)] = 0
    w = torch.rand(n, generator=torch.Generator().manual_seed(seed + 2)) + 0.5
    count = n // parts
    wp = P._head_rows(w, [(Pn, Pp)], H)
    if count % Pn == 0:
        nm = P.Norm(wp, count, count // Pn * Pp, 1e-5, gate_first=True)
    elif Pn == Pp and count % 4 == 0:
        nm = P.Norm(wp, count, count, 1e-5, gate_first=True)
    else:
        nm = P.Norm(wp, count, 0, 1e-5, gate_first=True, seg=(Pn, Pp))
    o, z = o.cuda(), z
    want = np.zeros((T, H * Pp))
    want[:, mask] = O.rms_in_parts((_np(o) * _np(z)[:, :H * Pp])[:, mask], _np(w), parts, 1e-5)
    return nm, o, z, want, H * Pp


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("H,Pn,parts", PARTS)
def test_gate_ahead_of_a_norm_in_parts(f32, H, Pn, parts):
    T = 3
    nm, o, z, want, N = _gated(H, Pn, parts, f32, T, 3)
    y = torch.full((T, N + 16), 7.0, dtype=DT[f32], device="cuda")
    nm.rows(o.data_ptr(), N, y.data_ptr(), N + 16, f32, T, N, gate=z.data_ptr(), ldg=N + 8)
    _close(_np(y)[:, :N], want, 3e-6 if f32 else 1e-5, rel=0 if f32 else 2 ** -8)
    assert (_np(y)[:, N:] == 7.0).all()
    # the same as the input of a one-token linear, with more inputs behind it
    F, M = 24, 37
    W, f = _t((M, N + F), 5, f32, N ** -0.5), _t((F,), 6, f32)
    pro = nm.prologue(o.data_ptr(), z.data_ptr())
    pro.n1, pro.x2 = N, f.data_ptr()
    r = torch.randn(M).cuda(); r0 = _np(r)
    ls = torch.full((M,), 0.3).cuda()
    e = P.epilogue(_lib.DN_RESID, ls=ls)
    _lib.call("lt_dn_gemv", W.data_ptr(), N + F, r.data_ptr(), f32, M, N + F, ctypes.byref(pro), ctypes.byref(e), stream())
    x = np.concatenate([_np(y)[0, :N], _np(f)])
    _close(_np(r), r0 + 0.3 * (_np(W) @ x), 1e-5 if f32 else 1e-2)


@pytest.mark.parametrize("f32", [0, 1])
def test_embedding_row_is_normed(f32):
    tab = _t((9, 13), 4, f32)
    w = torch.randn(13).cuda()
    tok = torch.tensor([8, 0, 3], dtype=torch.int32).cuda()
    a = torch.full((3, 16), 5.0).cuda()
    _lib.call("lt_dn_embed", tab.data_ptr(), f32, 13, tok.data_ptr(), 2.0, w.data_ptr(), 0.3, a.data_ptr(), None, 13, 16, 9, 3, stream())
    _close(_np(a)[:, :13], L.rms(2 * _np(tab)[[8, 0, 3]], _np(w), 0.3), 1e-6)
    assert (_np(a)[:, 13:] == 0).all()


# --------------------------------------------------------------------------- state-space recurrence

def _ssd_case(T, H, G, dp, dvp, f32, strong, seed=0):
    """rows [x | k | q], step sizes and decays, and the fp64 answer"""
    ld = H * dvp + 2 * G * dp + 8
    u = _t((T, ld), seed, f32, 0.7)
    rng = np.random.default_rng(seed)
    hdt = torch.from_numpy(rng.uniform(0.01, 1.5, (T, H))).float().cuda()
    A = torch.from_numpy(-strong * rng.uniform(0.0, 1.0, H) ** 2).float().cuda()
    hla = (hdt * A).contiguous()
    D = torch.randn(H, generator=torch.Generator().manual_seed(seed)).cuda()
    S = torch.randn(H, dvp, dp, generator=torch.Generator().manual_seed(seed + 1)).cuda()
    dec = _lib.DnDecay()
    dec.hla, dec.hdt, dec.D, dec.ldh, dec.per = hla.data_ptr(), hdt.data_ptr(), D.data_ptr(), H, H // G
    un, nv, ng = _np(u), H * dvp, G * dp
    x, k, q = un[:, :nv].reshape(T, H, dvp), un[:, nv:nv + ng].reshape(T, G, dp), un[:, nv + ng:nv + 2 * ng].reshape(T, G, dp)
    Sn = np.transpose(_np(S), (0, 2, 1)).copy()
    o = np.zeros((T, H, dvp))
    for t in range(T):               # with the rounded log decays the kernels are given
        for h in range(H):
            g = h // (H // G)
            Sn[h] = np.exp(_np(hla)[t, h]) * Sn[h] + _np(hdt)[t, h] * np.outer(k[t, g], x[t, h])
            o[t, h] = Sn[h].T @ q[t, g] + _np(D)[h] * x[t, h]
    ptr = lambda off: u.data_ptr() + off * u.element_size()
    return u, ld, S, dec, (hdt, hla, D, A), (ptr(nv + ng), ptr(nv), ptr(0)), o.reshape(T, nv), np.transpose(Sn, (0, 2, 1))


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("T,H,G,dp,dvp", [(1, 4, 2, 16, 24), (2, 3, 3, 48, 40), (17, 2, 1, 8, 8), (40, 6, 2, 128, 72), (20, 2, 1, 264, 40)])
def test_ssd_recurrence_in_token_order(f32, T, H, G, dp, dvp):
    u, ld, S, dec, keep, (q, k, v), o, Sn = _ssd_case(T, H, G, dp, dvp, f32, 2.0)
    out = torch.full((T, H * dvp + 4), 9.0, device="cuda")
    _lib.call("lt_dn_recurrence", q, k, v, ld, S.data_ptr(), out.data_ptr(), H * dvp + 4, f32, T, H, dp, dvp, ctypes.byref(dec), stream())
    _close(_np(out)[:, :H * dvp], o, 1e-5)
    assert (_np(out)[:, H * dvp:] == 9.0).all()
    _close(_np(S), Sn, 1e-5)


@pytest.mark.parametrize("strong", [0.02, 1.0, 60.0])
@pytest.mark.parametrize("T,H,G,dp,dvp", [(64, 2, 1, 64, 64), (65, 3, 3, 48, 32), (130, 4, 2, 128, 128), (200, 1, 1, 24, 40), (16, 2, 2, 8, 8),
                                          (150, 4, 1, 200, 136), (96, 2, 1, 256, 256), (321, 6, 2, 40, 24)])
def test_ssd_recurrence_in_chunks(strong, T, H, G, dp, dvp):
    u, ld, S, dec, keep, (q, k, v), o, Sn = _ssd_case(T, H, G, dp, dvp, 0, strong)
    out = torch.full((T, H * dvp + 4), 9.0, device="cuda")
    ws = torch.full((_lib.dense().lt_dn_recurrence_chunked_ws(T, H, dp, dvp),), float("nan"), device="cuda")
    _lib.call("lt_dn_recurrence_chunked", q, k, v, ld, S.data_ptr(), out.data_ptr(), H * dvp + 4, T, H, dp, dvp, ctypes.byref(dec),
              ws.data_ptr(), stream())
    _close(_np(out)[:, :H * dvp], o, 1e-4)
    assert (_np(out)[:, H * dvp:] == 9.0).all()
    _close(_np(S), Sn, 1e-4)


def test_ssd_chunks_recall_one_far_token():
    """One token is written under a key of its own and read back 190 tokens later with the decay it should have, across chunk
    borders and not; everything else is silent."""
    T, H, dp, dvp = 256, 2, 32, 16
    for star, ask in ((3, 193), (63, 64), (64, 127), (0, 255)):
        u = torch.zeros(T, H * dvp + 2 * dp)
        u[star, :dvp] = torch.arange(dvp) + 1.0
        u[star, H * dvp + 5] = 1.0
        u[ask, H * dvp + dp + 5] = 1.0
        u = u.bfloat16().cuda()
        hdt = torch.full((T, H), 0.5).cuda()
        hla = torch.full((T, H), -0.01).cuda()
        D = torch.zeros(H).cuda()
        dec = _lib.DnDecay()
        dec.hla, dec.hdt, dec.D, dec.ldh, dec.per = hla.data_ptr(), hdt.data_ptr(), D.data_ptr(), H, H
        S, o = torch.zeros(H, dvp, dp).cuda(), torch.empty(T, H * dvp, device="cuda")
        ws = torch.empty(_lib.dense().lt_dn_recurrence_chunked_ws(T, H, dp, dvp), device="cuda")
        p, e = u.data_ptr(), 2
        _lib.call("lt_dn_recurrence_chunked", p + (H * dvp + dp) * e, p + H * dvp * e, p, u.shape[1], S.data_ptr(), o.data_ptr(), H * dvp, T, H, dp,
                  dvp, ctypes.byref(dec), ws.data_ptr(), stream())
        want = np.zeros((T, H * dvp)); want[ask, :dvp] = (np.arange(dvp) + 1) * 0.5 * np.exp(-0.01 * (ask - star))
        assert np.abs(_np(o) - want).max() < 1e-3, (star, ask)


class _Ssd:
    """A state-space layer behind its projections, fed in portions."""

    def __init__(self, f32, H, G, dp, dvp, taps, seed=0):
        self.f32, self.H, self.G, self.dp, self.dvp, self.taps = f32, H, G, dp, dvp, taps
        self.C = H * dvp + 2 * G * dp
        g = torch.Generator().manual_seed(seed)
        r = lambda *s: torch.randn(*s, generator=g).cuda()
        self.conv, self.cb, self.dtb, self.A, self.D = r(taps, self.C), r(self.C) * 0.2, r(H), -torch.rand(H, generator=g).cuda(), r(H)
        self.desc = _lib.DnSsd(H, G, dp, dvp, taps, *[t.data_ptr() for t in (self.conv, self.cb, self.dtb, self.A, self.D)])
        self.ring = torch.full((taps, self.C), float("nan"), dtype=DT[f32], device="cuda")
        self.S = torch.zeros(H, dvp, dp, device="cuda")
        self.len, self.ticket = torch.zeros(1, dtype=torch.int32, device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
        self.pos = 0
        self.before, self.So = np.zeros((taps - 1, self.C)), np.zeros((H, dp, dvp))

    def rows(self, u, dt):
        T, ld = u.shape
        out = torch.empty(T, self.C, dtype=DT[self.f32], device="cuda")
        hla, hdt, o = [torch.empty(T, n, device="cuda") for n in (self.H, self.H, self.H * self.dvp)]
        _lib.call("lt_dn_ssd_rows", u.data_ptr(), ld, dt.data_ptr(), self.H, self.ring.data_ptr(), out.data_ptr(), self.C, hla.data_ptr(),
                  hdt.data_ptr(), self.f32, T, self.pos, ctypes.byref(self.desc), stream())
        dec = _lib.DnDecay()
        dec.hla, dec.hdt, dec.D, dec.ldh, dec.per = hla.data_ptr(), hdt.data_ptr(), self.D.data_ptr(), self.H, self.H // self.G
        e, nv, ng = out.element_size(), self.H * self.dvp, self.G * self.dp
        p = out.data_ptr()
        _lib.call("lt_dn_recurrence", p + (nv + ng) * e, p + nv * e, p, self.C, self.S.data_ptr(), o.data_ptr(), nv, self.f32, T, self.H, self.dp,
                  self.dvp, ctypes.byref(dec), stream())
        self.pos += T
        self.len.fill_(self.pos)
        return _np(o)

    def step(self, u, dt):
        o = torch.empty(1, self.H * self.dvp, device="cuda")
        _lib.call("lt_dn_ssd_step", u.data_ptr(), dt.data_ptr(), self.ring.data_ptr(), self.S.data_ptr(), o.data_ptr(), self.f32,
                  self.len.data_ptr(), self.ticket.data_ptr(), ctypes.byref(self.desc), stream())
        self.pos += 1
        assert int(self.len.item()) == self.pos and int(self.ticket.item()) == 0
        return _np(o)

    def oracle(self, u, dt):
        T, nv, ng = u.shape[0], self.H * self.dvp, self.G * self.dp
        y, self.before = O.causal_conv(u[:, :self.C], _np(self.conv).T, _np(self.cb), self.before)
        x, k, q = np.split(L.silu(y), [nv, nv + ng], axis=1)
        return O.ssd_recurrence(x.reshape(T, self.H, self.dvp), k.reshape(T, self.G, self.dp), q.reshape(T, self.G, self.dp),
                                O.softplus(dt + _np(self.dtb)), _np(self.A), _np(self.D), self.So).reshape(T, nv)


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("H,G,dp,dvp,taps", [(4, 2, 16, 24, 4), (3, 1, 40, 8, 3), (2, 2, 8, 40, 2), (4, 1, 24, 16, 1), (2, 1, 16, 8, 7),
                                             (2, 1, 264, 72, 4)])
def test_convolution_and_state_across_portions_and_single_tokens(f32, H, G, dp, dvp, taps):
    A = _Ssd(f32, H, G, dp, dvp, taps)
    for n, T in enumerate((1, 1, 2, 1, 3, 9, 1, 1, 20, 2, 2, 1, 1, 1, 1, 8, 1)):
        u, dt = _t((T, A.C + 8), 100 + n, f32), torch.randn(T, H, generator=torch.Generator().manual_seed(n)).cuda() * 3
        want = A.oracle(_np(u), _np(dt))
        got = A.step(u, dt) if T == 1 else A.rows(u, dt)
        if f32:
            _close(got, want, 3e-5)
        else:
            _close(got, want, 6e-2)
            assert np.sqrt(np.mean((got - want) ** 2)) < 1.5e-2 * np.sqrt(np.mean(want ** 2))


# --------------------------------------------------------------------------- grouped-query attention

class _Gqa:
    def __init__(self, f32, H=6, G=2, d=24, dv=40, rot=16, cap=300, base=1000.0, scale=0.4, softcap=8.0, vmix=0.0, vstore=None, seed=0):
        self.f32, self.H, self.G, self.d, self.dv, self.rot, self.cap = f32, H, G, d, dv, rot, cap
        self.base, self.scale, self.softcap, self.vmix, self.vstore = base, scale, softcap, vmix, vstore
        g = torch.Generator().manual_seed(seed)
        f = base ** (-2.0 * torch.arange(rot // 2, dtype=torch.float64) / max(rot, 1))
        hi = f.float()
        self.freq = torch.stack([hi, (f - hi.double()).float()], dim=1).contiguous().cuda()
        self.qn, self.kn = (torch.rand(H * d, generator=g) + 0.5).cuda(), (torch.rand(G * d, generator=g) + 0.5).cuda()
        self.desc = _lib.DnGqa(H, G, d, dv, rot, H * d, G * d, cap, scale, softcap, 1e-5, vmix, self.freq.data_ptr(), self.qn.data_ptr(),
                               self.kn.data_ptr())
        self.width = (H + G) * d + G * dv
        self.k = torch.full((cap, G * d), float("nan"), dtype=DT[f32], device="cuda")
        self.v = torch.full((cap, G * dv), float("nan"), dtype=DT[f32], device="cuda")
        self.len = torch.zeros(1, dtype=torch.int32, device="cuda")
        self.tickets = torch.zeros(_lib.dense().lt_dn_gqa_step_tickets(H, G), dtype=torch.int32, device="cuda")
        self.pos = 0
        self.cache = {"k": [], "v": []}

    def rows(self, y, gate, vf=None):
        T = y.shape[0]
        d, e = ctypes.byref(self.desc), y.element_size()
        out = torch.empty(T, self.H * self.dv, dtype=DT[self.f32], device="cuda")
        _lib.call("lt_dn_gqa_rows", y.data_ptr(), self.width, self.k.data_ptr(), self.v.data_ptr(), None if vf is None else vf.data_ptr(),
                  int(self.vstore or 0), self.f32, T, self.pos, d, stream())
        _lib.call("lt_dn_gqa_attn", y.data_ptr(), self.width, self.k.data_ptr(), self.v.data_ptr(), None if gate is None else gate.data_ptr(),
                  self.H, out.data_ptr(), self.H * self.dv, self.f32, T, self.pos, d, stream())
        self.pos += T
        self.len.fill_(self.pos)
        return _np(out)

    def step(self, y, gate, splits, vf=None):
        out = torch.empty(self.H * self.dv, dtype=DT[self.f32], device="cuda")
        ws = torch.full((_lib.dense().lt_dn_gqa_step_ws(self.H, self.dv, splits),), float("nan"), device="cuda")
        _lib.call("lt_dn_gqa_step", y.data_ptr(), self.k.data_ptr(), self.v.data_ptr(), None if vf is None else vf.data_ptr(),
                  int(self.vstore or 0), None if gate is None else gate.data_ptr(), out.data_ptr(), self.f32, self.len.data_ptr(),
                  ctypes.byref(self.desc), splits, ws.data_ptr(), self.tickets.data_ptr(), stream())
        self.pos += 1
        assert int(self.len.item()) == self.pos and int(self.tickets.abs().sum().item()) == 0
        return _np(out).reshape(1, -1)

    def oracle(self, y, gate, pos0, vf=None):
        """the same from the untouched rows, through the oracle's mechanism with identity projections"""
        eye = np.eye(self.width)
        nq, nk = self.H * self.d, self.G * self.d
        w = {"q": eye[:nq], "k": eye[nq:nq + nk], "v": eye[nq + nk:], "q.norm": _np(self.qn), "k.norm": _np(self.kn), "vmix": np.array(self.vmix),
             "g": np.zeros((self.H, self.width)), "o": 2.0 * np.eye(self.H * self.dv)}        # gates of a zero matrix are 1/2
        m = {"heads": self.H, "kv_heads": self.G, "dim": self.d, "vdim": self.dv, "rot": {"base": self.base, "dims": self.rot},
             "scale": self.scale, "softcap": self.softcap, "v_mix": vf is not None and not self.vstore}
        o = O.grouped_attention(y, m, lambda n: w[n], 1e-5, self.cache, pos0, {} if vf is None else {"v": vf})
        return o if gate is None else (o.reshape(len(y), self.H, self.dv) * gate[:, :, None]).reshape(len(y), -1)


GQA = [dict(), dict(H=1, G=1, d=8, dv=8, rot=0, softcap=0.0), dict(H=12, G=1, d=16, dv=8, rot=2), dict(H=3, G=3, d=64, dv=136, rot=64, softcap=3.0),
       dict(H=10, G=2, d=40, dv=24, rot=24, softcap=30.0), dict(H=4, G=2, d=128, dv=128, rot=128), dict(H=2, G=1, d=72, dv=264, rot=40, softcap=0.0),
       dict(H=34, G=2, d=8, dv=16, rot=8), dict(H=2, G=2, d=264, dv=512, rot=264)]


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("kw", GQA)
def test_grouped_attention_portions_and_single_tokens(f32, kw):
    A = _Gqa(f32, **kw)
    rng = np.random.default_rng(5)
    for n, T in enumerate((3, 1, 2, 37, 1, 1, 64, 65, 1, 5, 2, 1)):
        y = _t((T, A.width), 100 + n, f32)
        gate = torch.rand(T, A.H, generator=torch.Generator().manual_seed(n)).cuda()
        want = A.oracle(_np(y), _np(gate), A.pos)
        got = A.step(y, gate, int(rng.integers(1, 20))) if T == 1 else A.rows(y, gate)
        if f32:
            _close(got, want, 5e-5)
        else:
            _close(got, want, 0.15)
            assert np.sqrt(np.mean((got - want) ** 2)) < 1e-2 * np.sqrt(np.mean(want ** 2))


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("lam", [0.0, 0.3, 1.0])
def test_values_mixed_with_an_earlier_layer(f32, lam):
    A, B = _Gqa(f32, vstore=1), _Gqa(f32, vmix=lam, vstore=0, seed=9)
    for n, T in enumerate((5, 1, 1, 20, 2, 1)):
        ya, yb = _t((T, A.width), 10 + n, f32), _t((T, A.width), 50 + n, f32)
        vf = torch.full((T, A.G * A.dv), float("nan"), dtype=DT[f32], device="cuda")
        first = _np(ya)[:, (A.H + A.G) * A.d:]
        wa, wb = A.oracle(_np(ya), None, A.pos), B.oracle(_np(yb), None, B.pos, first)
        ga, gb = (A.step(ya, None, 3, vf), B.step(yb, None, 3, vf)) if T == 1 else (A.rows(ya, None, vf), B.rows(yb, None, vf))
        assert np.array_equal(_np(vf), first)
        for got, want in ((ga, wa), (gb, wb)):
            _close(got, want, 5e-5 if f32 else 0.15)


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("star", [0, 15, 16, 63, 64, 127, 128, 200])
def test_one_outstanding_key_is_found_from_everywhere(f32, star):
    """Every query asks for one channel, one position has it: its value comes back from any distance, in prompts, short
    portions and single tokens with several numbers of ranges; before the position nothing of it is seen."""
    A = _Gqa(f32, H=4, G=2, d=16, dv=16, rot=0, scale=1.0, softcap=40.0, cap=420)
    A.qn.fill_(1.0); A.kn.fill_(1.0)
    n = 420
    y = torch.zeros(n, A.width)
    for h in range(A.H):
        y[:, h * 16 + 3] = 1.0                        # normed: 4 in one channel
    for g in range(A.G):
        y[:, (A.H + g) * 16 + 7] = 1.0
        y[star, (A.H + g) * 16 + 7] = 0.0
        y[star, (A.H + g) * 16 + 3] = 1.0
        y[:, (A.H + A.G + g) * 16 + 1] = 1.0
        y[star, (A.H + A.G + g) * 16 + 1] = 0.0
        y[star, (A.H + A.G + g) * 16 + 2 + g] = 1.0
    y = y.to(DT[f32]).cuda()
    outs, at, i = [], 0, 0
    for c in (130, 1, 2, 1, 66, 1, 1, 1, 150):
        s = y[at:at + c].clone()
        outs.append(A.step(s, None, (1, 3, 7, 26)[i % 4]) if c == 1 else A.rows(s, None))
        at += c; i += 1
    while at < n:
        outs.append(A.step(y[at:at + 1].clone(), None, (1, 3, 7, 26)[at % 4])); at += 1
    o = np.concatenate(outs)
    cap = lambda s: 40 * np.tanh(s / 40)
    for t in range(n):
        w = np.exp(cap(16.0)) / (np.exp(cap(16.0)) + t) if t >= star else 0.0
        for h in range(A.H):
            assert abs(o[t, h * 16 + 2 + h // 2] - w) < 5e-3, (t, h, o[t, h * 16:h * 16 + 8])
            assert abs(o[t, h * 16 + 1] - (1 - w)) < 5e-3


@pytest.mark.parametrize("f32", [0, 1])
def test_rotation_of_far_positions(f32):
    """Scores depend on the distance alone, also far from the start (fp32 products of position and frequency would not do)."""
    import math
    d = 32
    A = _Gqa(f32, H=1, G=1, d=d, dv=8, rot=d, cap=40000, scale=1.0, softcap=0.0)
    A.qn.fill_(1.0); A.kn.fill_(1.0)
    y = _t((2, A.width), 1, f32)
    q = {}
    for pos in (5, 39990):
        s = y.clone()
        A.pos = pos
        _lib.call("lt_dn_gqa_rows", s.data_ptr(), A.width, A.k.data_ptr(), A.v.data_ptr(), None, 0, f32, 2, pos, ctypes.byref(A.desc), stream())
        q[pos] = float(_np(s)[1, :d] @ _np(A.k)[pos])
        want = L.rotate_half(L.rms(_np(y)[1:, :d], 1.0, 1e-5), [pos + 1], A.base, d)
        _close(_np(s)[1:, :d], want, 2e-6 if f32 else 1e-2)
    assert math.isclose(q[5], q[39990], abs_tol=2e-5 * d if f32 else 0.2)


def test_a_full_cache_is_reported():
    A = _Gqa(0, cap=4)
    y = _t((1, A.width), 1, 0)
    for _ in range(4):
        A.step(y, None, 2)
    assert _lib.device_status() == set()
    A.pos = 3
    A.step(y, None, 2)
    assert _lib.device_status() == {"kv_overflow"}
