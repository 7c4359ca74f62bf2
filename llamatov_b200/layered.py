"""Decoders whose layers are mixers chosen per layer, with dense bf16 or fp32 weights (libllamatov_b200_dense.so).

A layer is x <- x + ls1 * mixer(norm1(x)), x <- x + ls2 * ff(norm2(x)), the residual stream in fp32.  The mixers are
classes of one interface, registered by the type name a config uses; what a mixer needs of a model (sizes, constants)
it reads from its own config entry, so another design can list the same mixers with other numbers:

  RecurrentMixer        linear attention with a decaying fp32 state; two parameterisations of it are registered, "gla"
                        (a decay per key channel from a low-rank projection, norm per head) and "lightning" (a constant
                        decay per head, activations on q, k, v, norm over all heads)
  LatentAttentionMixer  attention over a sliding window with keys and values projected from a cached latent

A range of layers may run several times (config "loop"); every pass has its own cache slot.

Weights are packed once per model (`packed`): projections that read the same input are stacked into one matrix, head
sizes and row lengths are padded to multiples of 8 with zeros, so kernels need no ragged edges.
"""
import ctypes

import torch

from . import _lib, archs
from . import dev_residency as dr

# bf16 portions of at least this many tokens take the chunked form of the recurrence, for head sizes up to the limit
CHUNKED_FROM = 64
CHUNKED_MAX_DIM = 256

DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


def pad8(n):
    return (n + 7) // 8 * 8


class DenseWeights(dict):
    """Tensor name -> CPU tensor, as loaded; the packed device form is made on first use."""
    packed = None


# --------------------------------------------------------------------------- packing helpers

def _head_rows(W, sizes, heads):
    """Rows of a projection laid out head by head, each head `sizes` = [(n, padded n), ...] consecutive pieces."""
    per = sum(n for n, _ in sizes)
    W = W.reshape(heads, per, *W.shape[1:])
    parts, r = [], 0
    for n, p in sizes:
        piece = W[:, r:r + n]
        r += n
        if p > n:
            piece = torch.cat([piece, piece.new_zeros((heads, p - n) + tuple(W.shape[2:]))], dim=1)
        parts.append(piece)
    out = torch.cat(parts, dim=1)
    return out.reshape(-1, *W.shape[2:])


def _head_cols(W, n, heads):
    """Columns of an output projection, each head's n padded to a multiple of 8."""
    return _head_rows(W.T.contiguous(), [(n, pad8(n))], heads).T.contiguous()


def _pad_cols(W, k):
    return W if W.shape[1] == k else torch.cat([W, W.new_zeros(W.shape[0], k - W.shape[1])], dim=1)


def _pad_rows(W, n):
    return W if W.shape[0] == n else torch.cat([W, W.new_zeros((n - W.shape[0],) + tuple(W.shape[1:]))], dim=0)


# --------------------------------------------------------------------------- launch helpers

class Linear:
    """A packed matrix on the device: rows() over token rows, row() for one token with the input made in the kernel."""

    def __init__(self, W, dtype):
        W = _pad_cols(W.to(dtype), pad8(W.shape[1])).contiguous()
        self.M, self.K = W.shape
        self.f32 = int(dtype == torch.float32)
        self.W = W.cuda()
        self.ptr = self.W.data_ptr()

    def rows(self, x, ldx, y, ldy, T, epi, M=None):
        _lib.call("lt_dn_linear", self.ptr, self.K, x, ldx, y, ldy, self.f32, self.M if M is None else M, self.K, T,
                  ctypes.byref(epi), 0, dr._stream())

    def row(self, pro, y, epi, M=None):
        _lib.call("lt_dn_gemv", self.ptr, self.K, y, self.f32, self.M if M is None else M, self.K, ctypes.byref(pro),
                  ctypes.byref(epi), dr._stream())


def epilogue(kind=_lib.DN_STORE, segs=(), bias=None, ls=None, out_f32=False):
    """segs: (end, activation name or None, scale) per output segment."""
    e = _lib.DnEpilogue()
    e.kind, e.out_f32, e.nseg = kind, int(out_f32), len(segs)
    for i, (end, act, scale) in enumerate(segs):
        e.seg_end[i], e.seg_act[i], e.seg_scale[i] = end, _lib.DN_ACT[act], scale
    e.bias = None if bias is None else bias.data_ptr()
    e.ls = None if ls is None else ls.data_ptr()
    return e


class Norm:
    """RMS norm over groups of `group` (padded) elements of which `count` are real; weight repeats every w_period."""

    def __init__(self, w, count, group, eps):
        self.w = w.float().cuda().contiguous()
        self.count, self.group, self.eps = int(count), int(group), float(eps)

    def prologue(self, x, gate=None):
        return _lib.DnPrologue(_lib.DN_IN_NORM, 0, self.group, self.count, self.eps, x, None, self.w.data_ptr(),
                               self.w.numel(), gate)

    def rows(self, x, ldx, y, ldy, f32, T, N, gate=None, ldg=0, index=None):
        _lib.call("lt_dn_norm_rows", x, ldx, index, self.w.data_ptr(), self.w.numel(), gate, ldg, y, ldy, f32, T, N,
                  self.group, self.count, self.eps, dr._stream())


def typed_input(x):
    return _lib.DnPrologue(_lib.DN_IN_TYPED, 0, 0, 0, 0.0, x, None, None, 0, None)


def cast_input(x, n1, x2=None):
    return _lib.DnPrologue(_lib.DN_IN_CAST, n1, 0, 0, 0.0, x, x2, None, 0, None)


# --------------------------------------------------------------------------- mixers

class RecurrentMixer:
    """S <- diag(a_t) S + k_t v_t^T, o_t = S^T q_t per head; the output is W_o of norm(o) * gate.

    Parameters: activations of q, k and v, the scale on q, the gate's activation, whether the norm is per head, and
    the decay (constants per head, or low-rank per key channel with temperature tau)."""

    def __init__(self, pk, cfg, m, tensor, ls, act=None, q_scale=1.0, gate="sigmoid", head_norm=False, decay=None, tau=None):
        dt, E, eps = pk.dtype, cfg["n_embd"], cfg["norm_eps"]
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        self.H, self.dp, self.dvp = H, pad8(d), pad8(dv)
        nk, nv = H * self.dp, H * self.dvp
        parts = [_head_rows(tensor("q"), [(d, self.dp)], H), _head_rows(tensor("k"), [(d, self.dp)], H),
                 _head_rows(tensor("v"), [(dv, self.dvp)], H), _head_rows(tensor("g"), [(dv, self.dvp)], H)]
        self.off_k, self.off_v, self.off_g = nk, 2 * nk, 2 * nk + nv
        self.off_a = 2 * nk + 2 * nv
        segs = [(nk, act, q_scale), (2 * nk, act, 1.0), (2 * nk + nv, act, 1.0), (2 * nk + 2 * nv, gate, 1.0)]
        self.decay = self.a2 = None
        if decay is not None:
            if len(decay) != H:
                raise ValueError(f"{len(decay)} decays for {H} heads")
            self.decay = torch.tensor(decay, dtype=torch.float32).cuda()
        else:
            a1 = tensor("a1")
            self.rank = pad8(a1.shape[0])
            parts.append(_pad_rows(a1, self.rank))
            segs.append((self.off_a + self.rank, None, 1.0))
            self.a2 = Linear(_head_rows(tensor("a2"), [(d, self.dp)], H), dt)
            self.a2b = _head_rows(tensor("a2.b").float(), [(d, self.dp)], H).cuda()
            self.inv_tau = 1.0 / float(tau)
            self.epi_la = epilogue(segs=[(nk, "logsigmoid", self.inv_tau)], bias=self.a2b, out_f32=True)
        self.inp = Linear(torch.cat([_pad_cols(p, pad8(E)) for p in parts]), dt)
        self.width = self.inp.M
        self.epi_in = epilogue(segs=segs)
        if head_norm:
            self.norm = Norm(_pad_rows(tensor("norm").float(), self.dvp), dv, self.dvp, eps)
        else:
            self.norm = Norm(_head_rows(tensor("norm").float(), [(dv, self.dvp)], H), H * dv, nv, eps)
        self.out = Linear(_pad_rows(_head_cols(tensor("o"), dv, H), pad8(E)), dt)
        self.nv, self.nk = nv, nk
        self.epi_out = epilogue(_lib.DN_RESID, ls=ls)
        pk.want(y=self.width, o=nv)

    def new_cache(self, cfg, max_rows):
        return dr.DeviceRecurrentState(self.H, self.dvp, self.dp)

    def _recur(self, pk, y, ld, o, ldo, cache, T, dec, st=None):
        e = pk.esize
        cache.length += T
        if not pk.f32 and T >= CHUNKED_FROM and max(self.dp, self.dvp) <= CHUNKED_MAX_DIM:
            ws = st.buf("chunk_ws", _lib.dense().lt_dn_recurrence_chunked_ws(T, self.H, self.dp, self.dvp), torch.float32)
            _lib.call("lt_dn_recurrence_chunked", y, y + self.off_k * e, y + self.off_v * e, ld, cache.state.data_ptr(), o, ldo,
                      T, self.H, self.dp, self.dvp, ctypes.byref(dec), ws, dr._stream())
            return
        _lib.call("lt_dn_recurrence", y, y + self.off_k * e, y + self.off_v * e, ld, cache.state.data_ptr(), o, ldo, pk.f32,
                  T, self.H, self.dp, self.dvp, ctypes.byref(dec), dr._stream())

    def step(self, pk, x, norm1, cache):
        b, e = pk.step, pk.esize
        y = b.y.data_ptr()
        self.inp.row(norm1.prologue(x), y, self.epi_in)
        dec = _lib.DnDecay()
        if self.decay is not None:
            dec.decay = self.decay.data_ptr()
        else:
            dec.a1, dec.a2, dec.lda2, dec.rank = y + self.off_a * e, self.a2.ptr, self.a2.K, self.rank
            dec.bias, dec.inv_tau = self.a2b.data_ptr(), self.inv_tau
        o = b.o.data_ptr()
        self._recur(pk, y, self.width, o, self.nv, cache, 1, dec)
        self.out.row(self.norm.prologue(o, y + self.off_g * e), x, self.epi_out)

    def rows(self, pk, st, h, ldh, caches):
        e, T, R, w = pk.esize, st.T, st.R, self.width
        y = st.buf("y", R * w, pk.dtype)
        o = st.buf("o", R * self.nv, torch.float32)
        on = st.buf("on", R * self.nv, pk.dtype)
        self.inp.rows(h, ldh, y, w, R, self.epi_in)
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
        self.norm.rows(o, self.nv, on, self.nv, pk.f32, R, self.nv, gate=y + self.off_g * e, ldg=w)
        self.out.rows(on, self.nv, st.x, st.ldx, R, self.epi_out)


class LatentAttentionMixer:
    """Softmax attention over a sliding window.  A head's query and key have `dim` plain and `rot_dim` rotated components;
    plain keys and values are projections of a cached, normed latent, the rotated key part is shared by the heads."""

    def __init__(self, pk, cfg, m, tensor, ls):
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
        self.inp = Linear(torch.cat([_pad_cols(q, pad8(E)), _pad_cols(dkv, pad8(E))]), dt)
        self.width = self.inp.M
        self.epi_in = epilogue()
        uk = _pad_cols(_head_rows(tensor("uk"), [(d, self.dp)], H), self.rp)
        uv = _pad_cols(_head_rows(tensor("uv"), [(dv, self.dvp)], H), self.rp)
        self.expand = Linear(torch.cat([uk, uv]), dt)                 # latent rows -> plain keys and values of all heads
        self.uv = self.expand.ptr + H * self.dp * self.rp * pk.esize
        self.ukT = uk.reshape(H, self.dp, self.rp).transpose(1, 2).to(dt).contiguous().cuda()
        self.out = Linear(_pad_rows(_head_cols(tensor("o"), dv, H), pad8(E)), dt)
        self.nv = H * self.dvp
        self.epi_out = epilogue(_lib.DN_RESID, ls=ls)
        i = torch.arange(rot // 2, dtype=torch.float64)
        self.freq = (base ** (-2.0 * i / max(rot, 1))).float().cuda()
        self.cnorm = _pad_rows(tensor("dkv.norm").float(), self.rp).cuda()
        self.desc = _lib.DnLatent(H, self.dp, self.rtp, self.dvp, rot, self.rp, rank, self.window, 0, float(m["scale"]),
                                  float(eps), self.freq.data_ptr(), self.cnorm.data_ptr())
        groups = (H + 7) // 8
        self.splits = max(1, min((self.window + 31) // 32, 148 // groups))
        pk.want(y=self.width, att=self.nv, ws=_lib.dense().lt_dn_latent_step_ws(H, self.rp, self.rtp, self.splits))

    def new_cache(self, cfg, max_rows):
        return dr.DeviceLatentCache(self.window - 1 + max_rows, self.rp + self.rtp, DTYPES[cfg["dtype"]])

    def _desc(self, cache):
        d = _lib.DnLatent.from_buffer_copy(self.desc)
        d.cap = cache.cap
        return d

    def step(self, pk, x, norm1, cache):
        b = pk.step
        y, att = b.y.data_ptr(), b.att.data_ptr()
        self.inp.row(norm1.prologue(x), y, self.epi_in)
        lp = cache._ensure_len_ptr(seed=not dr._capturing())
        _lib.call("lt_dn_latent_step", y, cache.rows.data_ptr(), lp, self.ukT.data_ptr(), self.uv, att, pk.f32,
                  ctypes.byref(self._desc(cache)), self.splits, b.ws.data_ptr(), dr._stream())
        cache.length += 1
        self.out.row(typed_input(att), x, self.epi_out)

    def rows(self, pk, st, h, ldh, caches):
        e, T, R, w, s = pk.esize, st.T, st.R, self.width, dr._stream
        y = st.buf("y", R * w, pk.dtype)
        att = st.buf("att", R * self.nv, pk.dtype)
        self.inp.rows(h, ldh, y, w, R, self.epi_in)
        wr, nkv = self.rp + self.rtp, self.H * self.dp + self.nv
        for b, c in enumerate(caches):
            np_ = min(self.window - 1, c.length)          # earlier rows the portion's queries can see
            nk = np_ + T
            keys = st.buf("keys", nk * wr, pk.dtype)
            kv = st.buf("kv", nk * nkv, pk.dtype)
            yb = y + b * T * w * e
            d = self._desc(c)
            _lib.call("lt_dn_latent_rows", yb, w, c.rows.data_ptr(), keys, np_, c.length, pk.f32, T, ctypes.byref(d), s())
            self.expand.rows(keys, wr, kv, nkv, nk, self.epi_in)
            _lib.call("lt_dn_window_attn", yb, w, kv, nkv, keys + self.rp * e, wr, kv + self.H * self.dp * e, nkv,
                      att + b * T * self.nv * e, self.nv, pk.f32, T, np_, ctypes.byref(d), s())
            c.length += T
            c._ensure_len_ptr()
        self.out.rows(att, self.nv, st.x, st.ldx, R, self.epi_out)


def _gla(pk, cfg, m, tensor, ls):
    return RecurrentMixer(pk, cfg, m, tensor, ls, q_scale=float(m["dim"]) ** -0.5, gate="silu", head_norm=True, tau=m["tau"])


def _lightning(pk, cfg, m, tensor, ls):
    return RecurrentMixer(pk, cfg, m, tensor, ls, act="silu", gate="sigmoid", decay=m["decay"])


MIXERS = {"gla": _gla, "lightning": _lightning, "latent_attention": LatentAttentionMixer}


class GatedFeedForward:
    """W_down(gelu_tanh(W_gate h) * W_up h); gate and up are one launch that stores the product."""

    def __init__(self, pk, cfg, m, tensor, ls):
        E = pad8(cfg["n_embd"])
        F = self.F = pad8(m["ff"])
        self.gu = Linear(torch.cat([_pad_cols(_pad_rows(tensor(n), F), E) for n in ("gate", "up")]), pk.dtype)
        self.down = Linear(_pad_rows(_pad_cols(tensor("down"), F), E), pk.dtype)
        self.epi_glu = epilogue(_lib.DN_GLU)
        self.epi_out = epilogue(_lib.DN_RESID, ls=ls)
        pk.want(f=F)

    def step(self, pk, x, norm2):
        f = pk.step.f.data_ptr()
        self.gu.row(norm2.prologue(x), f, self.epi_glu, M=self.F)
        self.down.row(typed_input(f), x, self.epi_out)

    def rows(self, pk, st, h, ldh):
        f = st.buf("f", st.R * self.F, pk.dtype)
        self.gu.rows(h, ldh, f, self.F, st.R, self.epi_glu, M=self.F)
        self.down.rows(f, self.F, st.x, st.ldx, st.R, self.epi_out)


FEED_FORWARDS = {"dense": GatedFeedForward}


# --------------------------------------------------------------------------- a model's packed weights

class _Bufs:
    pass


class _Layer:
    pass


class Packed:
    """Device weights of one model and the fixed buffers of its token step."""

    def __init__(self, w, cfg):
        self.dtype = DTYPES[cfg["dtype"]]
        self.f32 = int(self.dtype == torch.float32)
        self.esize = self.dtype.itemsize
        self._sizes = {}
        E = cfg["n_embd"]
        Ep = self.Ep = pad8(E)
        eps = cfg["norm_eps"]

        def norm(name):
            return Norm(_pad_rows(w[name].float(), Ep), E, Ep, eps)

        def scale(name):
            return _pad_rows(w[name].float(), Ep).cuda() if name in w else None
        self.keep = []
        self.layers = []
        for i, ly in enumerate(cfg["layers"]):
            L = _Layer()
            if ly["type"] not in MIXERS:
                raise NotImplementedError(f"layer {i}: mixer {ly['type']!r}; known are {', '.join(sorted(MIXERS))}")
            ls1, ls2 = scale(f"l{i}.ls1"), scale(f"l{i}.ls2")
            self.keep += [ls1, ls2]
            L.norm1 = norm(f"l{i}.norm1")
            L.mixer = MIXERS[ly["type"]](self, cfg, ly["mixer"], lambda n, p=f"l{i}.mix.": w[p + n], ls1)
            L.ff = None
            if ly.get("mlp") is not None:
                kind = ly["mlp"].get("kind", "dense")
                if kind not in FEED_FORWARDS:
                    raise NotImplementedError(f"layer {i}: feed-forward {kind!r}; known are {', '.join(sorted(FEED_FORWARDS))}")
                L.norm2 = norm(f"l{i}.norm2")
                L.ff = FEED_FORWARDS[kind](self, cfg, ly["mlp"], lambda n, p=f"l{i}.mlp.": w[p + n], ls2)
            self.layers.append(L)
        if cfg.get("loop"):
            W = w["loop.in"]
            self.loop_in = Linear(_pad_rows(torch.cat([_pad_cols(W[:, :E], Ep), _pad_cols(W[:, E:], Ep)], dim=1), Ep), self.dtype)
            self.loop_step = _pad_cols(w["loop.step"].float(), Ep).cuda().contiguous()
            self.epi_loop = [epilogue(bias=self.loop_step[t], out_f32=True) for t in range(self.loop_step.shape[0])]
        self.embed = w["embed"].to(self.dtype).cuda().contiguous()
        self.final_norm = norm("final.norm")
        self.head = Linear(_pad_cols(w["head"], Ep), self.dtype)
        self.epi_head = epilogue(out_f32=True)

        # buffers of the token step: residual streams in turn (a loop entry reads one and writes the other)
        n = self._sizes
        b = self.step = _Bufs()
        f32 = dict(dtype=torch.float32, device="cuda")
        b.x = [torch.zeros(Ep, **f32), torch.zeros(Ep, **f32)]
        b.x0 = torch.zeros(Ep, **f32)
        b.y = torch.zeros(n.get("y", 8), dtype=self.dtype, device="cuda")
        b.att = torch.zeros(n.get("att", 8), dtype=self.dtype, device="cuda")
        b.f = torch.zeros(n.get("f", 8), dtype=self.dtype, device="cuda")
        b.o = torch.zeros(n.get("o", 8), **f32)
        b.ws = torch.zeros(n.get("ws", 8), **f32)
        b.tok = torch.zeros(1, dtype=torch.int32, device="cuda")
        b.cur = 0

    def want(self, **sizes):
        """A step buffer must hold at least this many elements."""
        for k, v in sizes.items():
            self._sizes[k] = max(self._sizes.get(k, 0), int(v))


def packed(w, cfg):
    if w.packed is None:
        if dr._capturing():
            raise RuntimeError("weight upload during graph capture: run a step first")
        w.packed = Packed(w, cfg)
    return w.packed


# --------------------------------------------------------------------------- the architecture

class _Rows:
    """State of a prompt pass: residual stream and work buffers, grown on demand and shared by the layers."""

    def __init__(self, w, cfg, toks):
        self.w, self.cfg = w, cfg
        self.pk = packed(w, cfg)
        self.B, self.T = int(toks.shape[0]), int(toks.shape[1])
        self.R = self.B * self.T
        self.ldx = self.pk.Ep
        self._bufs = {}
        f32 = dict(dtype=torch.float32, device="cuda")
        self._x = torch.empty((self.R, self.ldx), **f32)
        self._x0 = torch.empty((self.R, self.ldx), **f32) if cfg.get("loop") else None
        self.x = self._x.data_ptr()

    def buf(self, name, n, dtype):
        t = self._bufs.get(name)
        if t is None or t.numel() < n or t.dtype != dtype:
            t = self._bufs[name] = torch.empty(n, dtype=dtype, device="cuda")
        return t.data_ptr()


class Layered(archs.Architecture):
    device_token = True
    max_rows = 2048

    # ------------------------------------------------------------------ configuration and weights
    def config_from_json(self, js, dtype):
        if dtype not in DTYPES:
            raise ValueError(f"dtype {dtype!r}: known are {', '.join(sorted(DTYPES))}")
        cfg = {"arch": js["architecture"], "dtype": dtype, "n_layers": len(js["layers"]), "n_embd": int(js["width"]),
               "vocab": int(js["vocab"]), "norm_eps": float(js["norm"]["eps"]), "layers": js["layers"],
               "loop": js.get("loop"), "embed_scale": float(js["embedding"]["scale"])}
        lp = cfg["loop"]
        if lp is not None:
            if not (0 <= lp["start"] < lp["stop"] <= cfg["n_layers"] and lp["times"] >= 1):
                raise ValueError(f"loop {lp} over {cfg['n_layers']} layers")
        return cfg

    def weights_from_safetensors(self, tensors, cfg):
        return DenseWeights(tensors)

    def runs(self, cfg):
        n, lp = cfg["n_layers"], cfg["loop"]
        order = [(i, None) for i in range(n)]
        if lp is not None:
            order = (order[:lp["start"]] + [(i, t) for t in range(lp["times"]) for i in range(lp["start"], lp["stop"])] +
                     order[lp["stop"]:])
        return [archs.Run(i, s, t, t is not None and i == lp["start"]) for s, (i, t) in enumerate(order)]

    def new_cache(self, w, cfg, run):
        return packed(w, cfg).layers[run.layer].mixer.new_cache(cfg, self.max_rows)

    # ------------------------------------------------------------------ one token
    def ensure_buffers(self, w, cfg):
        packed(w, cfg)
        dr._ensure_logits_n(cfg["vocab"])

    def embed_step(self, w, cfg, tok):
        pk = packed(w, cfg)
        b = pk.step
        if dr._DEVICE_EMBED is not None:
            tok_ptr = dr._DEVICE_EMBED[2]
        else:
            b.tok.fill_(int(tok.reshape(-1)[0]))
            tok_ptr = b.tok.data_ptr()
        b.cur = 0
        _lib.call("lt_dn_embed", pk.embed.data_ptr(), pk.f32, cfg["n_embd"], tok_ptr, cfg["embed_scale"], b.x[0].data_ptr(),
                  b.x0.data_ptr() if cfg["loop"] else None, cfg["n_embd"], pk.Ep, cfg["vocab"], 1, dr._stream())
        return b.x[0].data_ptr()

    def layer_step(self, w, cfg, run, x, cache):
        pk = packed(w, cfg)
        L, b = pk.layers[run.layer], pk.step
        if run.opens_pass:
            b.cur ^= 1
            nxt = b.x[b.cur].data_ptr()
            pk.loop_in.row(cast_input(x, pk.Ep, b.x0.data_ptr()), nxt, pk.epi_loop[run.loop_pass])
            x = nxt
        L.mixer.step(pk, x, L.norm1, cache)
        if L.ff is not None:
            L.ff.step(pk, x, L.norm2)
        return x

    def logits_step(self, w, cfg, x):
        pk = packed(w, cfg)
        pk.head.row(pk.final_norm.prologue(x), dr._addr(dr._ensure_logits_n(cfg["vocab"]).ptr), pk.epi_head)

    # ------------------------------------------------------------------ rows
    def rows_supported(self, w, cfg):
        return True

    def rows_begin(self, w, cfg, toks):
        st = _Rows(w, cfg, toks)
        pk = st.pk
        ids = toks.reshape(-1).to(device="cuda", dtype=torch.int32)
        _lib.call("lt_dn_embed", pk.embed.data_ptr(), pk.f32, cfg["n_embd"], ids.data_ptr(), cfg["embed_scale"], st.x,
                  None if st._x0 is None else st._x0.data_ptr(), cfg["n_embd"], pk.Ep, cfg["vocab"], st.R, dr._stream())
        st.ids = ids
        return st

    def layer_rows(self, st, run, caches):
        pk, R, Ep = st.pk, st.R, st.ldx
        L = pk.layers[run.layer]
        if run.opens_pass:
            xx = st.buf("xx", R * 2 * Ep, pk.dtype)
            _lib.call("lt_dn_concat_rows", st.x, Ep, Ep, st._x0.data_ptr(), Ep, Ep, xx, 2 * Ep, pk.f32, R, dr._stream())
            pk.loop_in.rows(xx, 2 * Ep, st.x, Ep, R, pk.epi_loop[run.loop_pass])
        h = st.buf("h", R * Ep, pk.dtype)
        L.norm1.rows(st.x, Ep, h, Ep, pk.f32, R, Ep)
        L.mixer.rows(pk, st, h, Ep, caches)
        if L.ff is not None:
            L.norm2.rows(st.x, Ep, h, Ep, pk.f32, R, Ep)
            L.ff.rows(pk, st, h, Ep)

    def rows_residual(self, st):
        return st._x[:, :st.cfg["n_embd"]]

    def rows_logits(self, st, rows):
        pk, V, n = st.pk, st.cfg["vocab"], len(rows)
        idx = torch.tensor(rows, dtype=torch.int32, device="cuda")
        h = st.buf("hl", n * st.ldx, pk.dtype)
        out = torch.empty((n, V), dtype=torch.float32, device="cuda")
        pk.final_norm.rows(st.x, st.ldx, h, st.ldx, pk.f32, n, st.ldx, index=idx.data_ptr())
        pk.head.rows(h, st.ldx, out.data_ptr(), V, n, pk.epi_head)
        return out.cpu()


ARCH = Layered()
