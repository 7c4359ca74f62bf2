"""Token mixers and feed-forwards of the decoders in `layered`: classes of one interface, registered by the type name a
config uses.  What a mixer needs of a model (sizes, constants) it reads from its own config entry, so another design can
list the same mixers with other numbers:

  RecurrentMixer         linear attention with a decaying fp32 state; two parameterisations of it are registered, "gla"
                         (a decay per key channel from a low-rank projection, norm per head) and "lightning" (a constant
                         decay per head, activations on q, k, v, norm over all heads)
  Mamba2Mixer            state-space recurrence with step sizes per token and head behind a short convolution
  LatentAttentionMixer   attention over a sliding window with keys and values projected from a cached latent
  GroupedAttentionMixer  grouped-query attention over all positions: normed and rotated queries and keys, capped scores,
                         values mixed with an earlier layer's, a gate per head

A mixer is an input projection, a core and an output projection.  It hands the two matrices to the block that it is part of
(`layered.SequentialBlock`, `layered.ParallelBlock`), which may stack them with the feed-forward's:

  w_in, segs, tail_from   input matrix, activations of its outputs, first output that stays fp32 (or None)
  width, ntail            elements of a stored row without the tail; outputs of the tail
  w_out, nin              output matrix, its inputs
  step_core(pk, y, tail, out, cache)            one token: from the projected row to a prologue that makes the nin inputs of the
                                                output projection (`out` holds nin elements for a core that stores them)
  rows_core(pk, st, y, tail, X, ldx, caches)    token rows: from y [R, width] and tail [R, ntail] to rows of X
"""
import ctypes

import torch

from . import _lib
from . import dev_residency as dr
from .dense_ops import (DTYPES, Linear, Norm, _head_cols, _head_rows, _pad_cols, _pad_rows, epilogue, pad8, typed_input)

# bf16 portions of at least this many tokens take the chunked form of the recurrence, for head sizes up to the limit
CHUNKED_FROM = 64
CHUNKED_MAX_DIM = 256


def recurrence(pk, q, k, v, ld, state, o, ldo, T, H, dp, dvp, dec, st):
    """The recurrence over T tokens: chunks on the tensor cores for long bf16 portions, else in token order."""
    if not pk.f32 and T >= CHUNKED_FROM and max(dp, dvp) <= CHUNKED_MAX_DIM:
        ws = st.buf("chunk_ws", _lib.dense().lt_dn_recurrence_chunked_ws(T, H, dp, dvp), torch.float32)
        _lib.call("lt_dn_recurrence_chunked", q, k, v, ld, state, o, ldo, T, H, dp, dvp, ctypes.byref(dec), ws, dr._stream())
        return
    _lib.call("lt_dn_recurrence", q, k, v, ld, state, o, ldo, pk.f32, T, H, dp, dvp, ctypes.byref(dec), dr._stream())


class RecurrentMixer:
    """S <- diag(a_t) S + k_t v_t^T, o_t = S^T q_t per head; the output is W_o of norm(o) * gate.

    Parameters: activations of q, k and v, the scale on q, the gate's activation, whether the norm is per head, and
    the decay (constants per head, or low-rank per key channel with temperature tau)."""
    tail_from, ntail = None, 0

    def __init__(self, pk, cfg, m, tensor, act=None, q_scale=1.0, gate="sigmoid", head_norm=False, decay=None, tau=None):
        dt, E, eps = pk.dtype, cfg["n_embd"], cfg["norm_eps"]
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        self.H, self.dp, self.dvp = H, pad8(d), pad8(dv)
        nk, nv = H * self.dp, H * self.dvp
        parts = [_head_rows(tensor("q"), [(d, self.dp)], H), _head_rows(tensor("k"), [(d, self.dp)], H),
                 _head_rows(tensor("v"), [(dv, self.dvp)], H), _head_rows(tensor("g"), [(dv, self.dvp)], H)]
        self.off_k, self.off_v, self.off_g = nk, 2 * nk, 2 * nk + nv
        self.off_a = 2 * nk + 2 * nv
        self.segs = [(nk, act, q_scale), (2 * nk, act, 1.0), (2 * nk + nv, act, 1.0), (2 * nk + 2 * nv, gate, 1.0)]
        self.decay = self.a2 = None
        if decay is not None:
            if len(decay) != H:
                raise ValueError(f"{len(decay)} decays for {H} heads")
            self.decay = torch.tensor(decay, dtype=torch.float32).cuda()
        else:
            a1 = tensor("a1")
            self.rank = pad8(a1.shape[0])
            parts.append(_pad_rows(a1, self.rank))
            self.segs.append((self.off_a + self.rank, None, 1.0))
            self.a2 = Linear(_head_rows(tensor("a2"), [(d, self.dp)], H), dt)
            self.a2b = _head_rows(tensor("a2.b").float(), [(d, self.dp)], H).cuda()
            self.inv_tau = 1.0 / float(tau)
            self.epi_la = epilogue(segs=[(nk, "logsigmoid", self.inv_tau)], bias=self.a2b, out_f32=True)
        self.w_in = torch.cat([_pad_cols(p, pad8(E)) for p in parts])
        self.width = self.w_in.shape[0]
        if head_norm:
            self.norm = Norm(_pad_rows(tensor("norm").float(), self.dvp), dv, self.dvp, eps)
        else:
            self.norm = Norm(_head_rows(tensor("norm").float(), [(dv, self.dvp)], H), H * dv, nv, eps)
        self.w_out = _pad_rows(_head_cols(tensor("o"), dv, H), pad8(E))
        self.nin = self.nv = nv
        self.nk = nk
        pk.want(o=nv)

    def new_cache(self, cfg, max_rows):
        return dr.DeviceRecurrentState(self.H, self.dvp, self.dp)

    def _recur(self, pk, y, ld, o, ldo, cache, T, dec, st=None):
        e = pk.esize
        cache.length += T
        recurrence(pk, y, y + self.off_k * e, y + self.off_v * e, ld, cache.state.data_ptr(), o, ldo, T, self.H, self.dp,
                   self.dvp, dec, st)

    def step_core(self, pk, y, tail, out, cache):
        e = pk.esize
        dec = _lib.DnDecay()
        if self.decay is not None:
            dec.decay = self.decay.data_ptr()
        else:
            dec.a1, dec.a2, dec.lda2, dec.rank = y + self.off_a * e, self.a2.ptr, self.a2.K, self.rank
            dec.bias, dec.inv_tau = self.a2b.data_ptr(), self.inv_tau
        o = pk.step.o.data_ptr()
        self._recur(pk, y, self.width, o, self.nv, cache, 1, dec)
        return self.norm.prologue(o, y + self.off_g * e)

    def rows_core(self, pk, st, y, tail, X, ldx, caches):
        e, T, R, w = pk.esize, st.T, st.R, self.width
        o = st.buf("o", R * self.nv, torch.float32)
        la = None
        if self.a2 is not None:
            la = st.buf("la", R * self.nk, torch.float32)
            self.a2.rows(y + self.off_a * e, w, la, self.nk, R, self.epi_la)
        for b, c in enumerate(caches):
            dec = _lib.DnDecay()
            if la is None:
                dec.decay = self.decay.data_ptr()
            else:
                dec.la, dec.ldla = la + b * T * self.nk * 4, self.nk
            self._recur(pk, y + b * T * w * e, w, o + b * T * self.nv * 4, self.nv, c, T, dec, st)
        self.norm.rows(o, self.nv, X, ldx, pk.f32, R, self.nv, gate=y + self.off_g * e, ldg=w)


class Mamba2Mixer:
    """S <- exp(A dt_t) S + dt_t B_t x_t^T, y_t = S^T C_t + D x_t per head, B and C shared by the heads of a group; x, B and
    C pass a causal convolution and silu, dt is softplus(dt + bias).  The output is W_o of norm(y * silu(z)), the norm in
    `norm_groups` equal parts."""

    def __init__(self, pk, cfg, m, tensor):
        E, eps = cfg["n_embd"], cfg["norm_eps"]
        H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
        parts, taps = m["norm_groups"], m["conv"]
        inner = H * P
        if H % G or inner % parts:
            raise ValueError(f"{H} heads in {G} groups, {inner} channels in {parts} norm groups")
        if tuple(tensor("conv").shape) != (inner + 2 * G * N, taps):
            raise ValueError(f"convolution {tuple(tensor('conv').shape)} for {inner + 2 * G * N} channels and {taps} taps")
        self.H, self.G, self.dp, self.dvp, self.taps = H, G, pad8(N), pad8(P), taps
        nv, ng = H * self.dvp, G * self.dp

        def split(W):           # x | B | C, head by head
            x, b, c = W.split([inner, G * N, G * N])
            return torch.cat([_head_rows(x, [(P, self.dvp)], H), _head_rows(b, [(N, self.dp)], G), _head_rows(c, [(N, self.dp)], G)])
        z, xbc, dt = tensor("in").split([inner, inner + 2 * G * N, H])
        self.w_in = _pad_cols(torch.cat([_head_rows(z, [(P, self.dvp)], H), split(xbc), dt]), pad8(E))
        self.off_x, self.channels = nv, nv + 2 * ng
        self.tail_from = self.width = nv + self.channels
        self.ntail = H
        self.segs = [(nv, "silu", 1.0)]
        conv = split(tensor("conv").float()).T.contiguous().cuda()
        f32 = lambda n: tensor(n).float().cuda().contiguous()
        A = (-torch.exp(tensor("A_log").double())).float().cuda()
        self.keep = [conv, split(tensor("conv.b").float()).cuda(), f32("dt_bias"), A, f32("D")]
        self.D = self.keep[4]
        self.desc = _lib.DnSsd(H, G, self.dp, self.dvp, taps, *[t.data_ptr() for t in self.keep])
        w, count = _head_rows(tensor("norm").float(), [(P, self.dvp)], H), inner // parts
        if count % P == 0:
            self.norm = Norm(w, count, count // P * self.dvp, eps, gate_first=True)
        elif P == self.dvp and count % 4 == 0:
            self.norm = Norm(w, count, count, eps, gate_first=True)
        else:
            self.norm = Norm(w, count, 0, eps, gate_first=True, seg=(P, self.dvp))
        self.w_out = _pad_rows(_head_cols(tensor("o"), P, H), pad8(E))
        self.nin = self.nv = nv
        pk.want(o=nv, tickets=1)

    def new_cache(self, cfg, max_rows):
        return dr.DeviceSsdState(self.H, self.dvp, self.dp, self.taps, self.channels, DTYPES[cfg["dtype"]])

    def step_core(self, pk, y, tail, out, cache):
        b = pk.step
        o = b.o.data_ptr()
        lp = cache._ensure_len_ptr(seed=not dr._capturing())
        _lib.call("lt_dn_ssd_step", y + self.off_x * pk.esize, tail, cache.ring.data_ptr(), cache.state.data_ptr(), o, pk.f32, lp,
                  b.tickets.data_ptr(), ctypes.byref(self.desc), dr._stream())
        cache.length += 1
        return self.norm.prologue(o, y)

    def rows_core(self, pk, st, y, tail, X, ldx, caches):
        e, T, R, w, H, C = pk.esize, st.T, st.R, self.width, self.H, self.channels
        u = st.buf("conv", R * C, pk.dtype)
        o = st.buf("o", R * self.nv, torch.float32)
        hla, hdt = st.buf("hla", R * H, torch.float32), st.buf("hdt", R * H, torch.float32)
        for b, c in enumerate(caches):
            ub, la, hd = u + b * T * C * e, hla + b * T * H * 4, hdt + b * T * H * 4
            _lib.call("lt_dn_ssd_rows", y + (b * T * w + self.off_x) * e, w, tail + b * T * H * 4, H, c.ring.data_ptr(), ub, C, la, hd,
                      pk.f32, T, c.length, ctypes.byref(self.desc), dr._stream())
            dec = _lib.DnDecay()
            dec.hla, dec.hdt, dec.D, dec.ldh, dec.per = la, hd, self.D.data_ptr(), H, H // self.G
            kb = ub + self.nv * e
            recurrence(pk, kb + self.G * self.dp * e, kb, ub, C, c.state.data_ptr(), o + b * T * self.nv * 4, self.nv, T, H, self.dp,
                       self.dvp, dec, st)
            c.length += T
            c._ensure_len_ptr()
        self.norm.rows(o, self.nv, X, ldx, pk.f32, R, self.nv, gate=y, ldg=w)


class LatentAttentionMixer:
    """Softmax attention over a sliding window.  A head's query and key have `dim` plain and `rot_dim` rotated components;
    plain keys and values are projections of a cached, normed latent, the rotated key part is shared by the heads."""
    tail_from, ntail, segs = None, 0, ()

    def __init__(self, pk, cfg, m, tensor):
        dt, E, eps = pk.dtype, cfg["n_embd"], cfg["norm_eps"]
        H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        rot, base = m["rot"]["dims"], float(m["rot"]["base"])
        if rot > r or rot % 2:
            raise ValueError(f"{rot} rotated dimensions of {r}")
        self.H, self.dp, self.rtp, self.dvp, self.rp = H, pad8(d), pad8(r), pad8(dv), pad8(rank)
        self.window = int(m["mask"]["size"])
        if self.window < 1:
            raise ValueError(f"window of {self.window}")
        self.nq = H * (self.dp + self.rtp)
        q = _head_rows(tensor("q"), [(d, self.dp), (r, self.rtp)], H)
        dkv = _head_rows(tensor("dkv"), [(rank, self.rp), (r, self.rtp)], 1)
        self.w_in = torch.cat([_pad_cols(q, pad8(E)), _pad_cols(dkv, pad8(E))])
        self.width = self.w_in.shape[0]
        self.epi_expand = epilogue()
        uk = _pad_cols(_head_rows(tensor("uk"), [(d, self.dp)], H), self.rp)
        uv = _pad_cols(_head_rows(tensor("uv"), [(dv, self.dvp)], H), self.rp)
        self.expand = Linear(torch.cat([uk, uv]), dt)                 # latent rows -> plain keys and values of all heads
        self.uv = self.expand.ptr + H * self.dp * self.rp * pk.esize
        self.ukT = uk.reshape(H, self.dp, self.rp).transpose(1, 2).to(dt).contiguous().cuda()
        self.w_out = _pad_rows(_head_cols(tensor("o"), dv, H), pad8(E))
        self.nin = self.nv = H * self.dvp
        i = torch.arange(rot // 2, dtype=torch.float64)
        self.freq = (base ** (-2.0 * i / max(rot, 1))).float().cuda()
        self.cnorm = _pad_rows(tensor("dkv.norm").float(), self.rp).cuda()
        self.desc = _lib.DnLatent(H, self.dp, self.rtp, self.dvp, rot, self.rp, rank, self.window, 0, float(m["scale"]),
                                  float(eps), self.freq.data_ptr(), self.cnorm.data_ptr())
        groups = (H + 7) // 8
        self.splits = max(1, min((self.window + 31) // 32, 148 // groups))
        pk.want(ws=_lib.dense().lt_dn_latent_step_ws(H, self.rp, self.rtp, self.splits))

    def new_cache(self, cfg, max_rows):
        return dr.DeviceLatentCache(self.window - 1 + max_rows, self.rp + self.rtp, DTYPES[cfg["dtype"]])

    def _desc(self, cache):
        d = _lib.DnLatent.from_buffer_copy(self.desc)
        d.cap = cache.cap
        return d

    def step_core(self, pk, y, tail, out, cache):
        b = pk.step
        lp = cache._ensure_len_ptr(seed=not dr._capturing())
        _lib.call("lt_dn_latent_step", y, cache.rows.data_ptr(), lp, self.ukT.data_ptr(), self.uv, out, pk.f32,
                  ctypes.byref(self._desc(cache)), self.splits, b.ws.data_ptr(), dr._stream())
        cache.length += 1
        return typed_input(out)

    def rows_core(self, pk, st, y, tail, X, ldx, caches):
        e, T, w, s = pk.esize, st.T, self.width, dr._stream
        wr, nkv = self.rp + self.rtp, self.H * self.dp + self.nv
        for b, c in enumerate(caches):
            np_ = min(self.window - 1, c.length)          # earlier rows the portion's queries can see
            nk = np_ + T
            keys = st.buf("keys", nk * wr, pk.dtype)
            kv = st.buf("kv", nk * nkv, pk.dtype)
            yb = y + b * T * w * e
            d = self._desc(c)
            _lib.call("lt_dn_latent_rows", yb, w, c.rows.data_ptr(), keys, np_, c.length, pk.f32, T, ctypes.byref(d), s())
            self.expand.rows(keys, wr, kv, nkv, nk, self.epi_expand)
            _lib.call("lt_dn_window_attn", yb, w, kv, nkv, keys + self.rp * e, wr, kv + self.H * self.dp * e, nkv,
                      X + b * T * ldx * e, ldx, pk.f32, T, np_, ctypes.byref(d), s())
            c.length += T
            c._ensure_len_ptr()


class GroupedAttentionMixer:
    """Softmax attention over all earlier positions, H query heads on G key/value heads.  Queries and keys are RMS-normed over
    the whole projection and rotated; scores pass softcap * tanh(score / softcap) if a softcap is given; with v_mix the
    values are mixed with those of the first such layer; a head's output is scaled by a gate of its own."""
    SMS = 148

    def __init__(self, pk, cfg, m, tensor):
        E = cfg["n_embd"]
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        rot = m.get("rot") or {"dims": 0, "base": 1.0}
        if H % G:
            raise ValueError(f"{H} query heads on {G} key heads")
        if rot["dims"] > d or rot["dims"] % 2:
            raise ValueError(f"{rot['dims']} rotated dimensions of {d}")
        self.H, self.G, self.dp, self.dvp = H, G, pad8(d), pad8(dv)
        nq, nk, nv = H * self.dp, G * self.dp, G * self.dvp
        self.w_in = _pad_cols(torch.cat([_head_rows(tensor("q"), [(d, self.dp)], H), _head_rows(tensor("k"), [(d, self.dp)], G),
                                         _head_rows(tensor("v"), [(dv, self.dvp)], G), tensor("g")]), pad8(E))
        self.tail_from = self.width = nq + nk + nv
        self.ntail = H
        self.segs = [(self.width, None, 1.0), (self.width + H, "sigmoid", 1.0)]
        self.w_out = _pad_rows(_head_cols(tensor("o"), dv, H), pad8(E))
        self.nin = H * self.dvp
        self.kw, self.vw = nk, nv
        f = float(rot["base"]) ** (-2.0 * torch.arange(rot["dims"] // 2, dtype=torch.float64) / max(rot["dims"], 1))
        hi = f.float()
        freq = torch.stack([hi, (f - hi.double()).float()], dim=1).contiguous().cuda()
        self.keep = [freq, _head_rows(tensor("q.norm").float(), [(d, self.dp)], H).cuda(),
                     _head_rows(tensor("k.norm").float(), [(d, self.dp)], G).cuda()]
        self.mix = self.mix_first = False
        vmix = 0.0
        if m.get("v_mix"):
            self.mix = True
            self.mix_first = pk.first_values is None
            if self.mix_first:
                pk.first_values = (G, dv)
            else:
                if pk.first_values != (G, dv) and not (pk.first_values[0] * pk.first_values[1] == G * dv and
                                                       pk.first_values[1] % 8 == dv % 8 == 0):
                    raise NotImplementedError(f"values of {G} x {dv} mixed with {pk.first_values[0]} x {pk.first_values[1]}")
                vmix = float(tensor("vmix").reshape(()))
        self.desc = _lib.DnGqa(H, G, self.dp, self.dvp, rot["dims"], H * d, G * d, 0, float(m["scale"]), float(m.get("softcap") or 0.0),
                               cfg["norm_eps"], vmix, *[t.data_ptr() for t in self.keep])
        self.tickets = _lib.dense().lt_dn_gqa_step_tickets(H, G)
        self.splits = max(1, min(74, 2 * self.SMS // (self.tickets - 1)))
        pk.want(ws=_lib.dense().lt_dn_gqa_step_ws(H, self.dvp, self.splits), tickets=self.tickets, vfirst=nv if self.mix else 0)

    def new_cache(self, cfg, max_rows):
        return dr.DeviceGroupedKV(dr._KV_MAX_SEQ, self.kw, self.vw, DTYPES[cfg["dtype"]])

    def _desc(self, cache):
        d = _lib.DnGqa.from_buffer_copy(self.desc)
        d.cap = cache.cap
        return d

    def step_core(self, pk, y, tail, out, cache):
        b = pk.step
        lp = cache._ensure_len_ptr(seed=not dr._capturing())
        splits = min(self.splits, (cache.cap + 15) // 16)
        _lib.call("lt_dn_gqa_step", y, cache.k.data_ptr(), cache.v.data_ptr(), b.vfirst.data_ptr() if self.mix else None,
                  int(self.mix_first), tail, out, pk.f32, lp, ctypes.byref(self._desc(cache)), splits, b.ws.data_ptr(),
                  b.tickets.data_ptr(), dr._stream())
        cache.length += 1
        return typed_input(out)

    def rows_core(self, pk, st, y, tail, X, ldx, caches):
        e, T, w = pk.esize, st.T, self.width
        vf = st.buf("vfirst", st.R * self.vw, pk.dtype) if self.mix else None
        for b, c in enumerate(caches):
            c.require(T)
            d = self._desc(c)
            yb, k, v = y + b * T * w * e, c.k.data_ptr(), c.v.data_ptr()
            _lib.call("lt_dn_gqa_rows", yb, w, k, v, None if vf is None else vf + b * T * self.vw * e, int(self.mix_first), pk.f32, T,
                      c.length, ctypes.byref(d), dr._stream())
            _lib.call("lt_dn_gqa_attn", yb, w, k, v, tail + b * T * self.ntail * 4, self.ntail, X + b * T * ldx * e, ldx, pk.f32, T,
                      c.length, ctypes.byref(d), dr._stream())
            c.length += T
            c._ensure_len_ptr()


def _gla(pk, cfg, m, tensor):
    return RecurrentMixer(pk, cfg, m, tensor, q_scale=float(m["dim"]) ** -0.5, gate="silu", head_norm=True, tau=m["tau"])


def _lightning(pk, cfg, m, tensor):
    return RecurrentMixer(pk, cfg, m, tensor, act="silu", gate="sigmoid", decay=m["decay"])


MIXERS = {"gla": _gla, "lightning": _lightning, "latent_attention": LatentAttentionMixer, "mamba2": Mamba2Mixer,
          "attention": GroupedAttentionMixer}


class GatedFeedForward:
    """W_down glu(W_gate h, W_up h); gate and up are one launch that stores the product.  `glu` is the gated activation as the
    epilogue takes it: (kind, alpha, limit)."""

    def __init__(self, pk, cfg, m, tensor, glu):
        E = pad8(cfg["n_embd"])
        F = self.F = pad8(m["ff"])
        self.glu = glu
        self.w_gu = torch.cat([_pad_cols(_pad_rows(tensor(n), F), E) for n in ("gate", "up")])
        self.w_down = _pad_rows(_pad_cols(tensor("down"), F), E)


def gelu_feed_forward(pk, cfg, m, tensor):
    """glu(g, u) = gelu_tanh(g) * u"""
    return GatedFeedForward(pk, cfg, m, tensor, (_lib.DN_GLU_GELU, 0.0, 0.0))


def clamped_feed_forward(pk, cfg, m, tensor):
    """glu(g, u) = g' sigmoid(1.702 g') (u' + 1) with g' = min(g, limit) and u' = u clamped to [-limit, limit]"""
    return GatedFeedForward(pk, cfg, m, tensor, (_lib.DN_GLU_CLAMPED, 1.702, float(m["limit"])))
