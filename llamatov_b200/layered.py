"""Decoders whose layers are mixers chosen per layer, with dense bf16 or fp32 weights (libllamatov_b200_dense.so), the
residual stream in fp32.  Mixers and feed-forwards are in `mixers`; a block puts them together:

  SequentialBlock   x <- x + ls1 * mixer(norm1(x)), x <- x + ls2 * ff(norm2(x))
  ParallelBlock     h = norm1(x), x <- x + m * (mixer(h) + ff(h)).  The projections of h are one stacked matrix, and so are the
                    two output projections: a token's layer is one launch into the block, the mixer's core, one out of it

A design (`Layered` and its subclasses) says which block, mixers and feed-forwards it has, and how its config is read:

  Nugusun   sequential blocks with layer scale, embedding scale, a range of layers that may run several times (config
            "loop"; every pass has its own cache slot)
  Pakalix   parallel blocks, norm weights stored around zero, a norm behind the embedding

Weights are packed once per model (`packed`).
"""
import torch

from . import _lib, archs
from . import dev_residency as dr
from .dense_ops import (DTYPES, Linear, Norm, _pad_cols, _pad_rows, cast_input, epilogue, pad8, typed_input, with_tail)
from .mixers import MIXERS, clamped_feed_forward, gelu_feed_forward


class DenseWeights(dict):
    """Tensor name -> CPU tensor, as loaded; the packed device form is made on first use."""
    packed = None


# --------------------------------------------------------------------------- blocks

class Block:
    """A layer.  `norm(name)` makes one of its norms, `scale(name)` a vector that scales a branch."""

    def __init__(self, pk, cfg, mixer, ff, norm, scale):
        raise NotImplementedError

    def step(self, pk, x, cache):
        raise NotImplementedError

    def rows(self, pk, st, caches):
        raise NotImplementedError

    def _input(self, pk, mixer):
        self.mixer = mixer
        self.epi_in = epilogue(segs=mixer.segs, tail_from=mixer.tail_from)
        pk.want(y=mixer.width, tail=mixer.ntail)

    def _project_rows(self, pk, st, inp, h, ldh):
        """The mixer's input projection over the rows: (y, tail)."""
        m = self.mixer
        y = st.buf("y", st.R * m.width, pk.dtype)
        tail = st.buf("tail", st.R * m.ntail, torch.float32) if m.ntail else None
        inp.rows(h, ldh, y, m.width, st.R, with_tail(self.epi_in, tail, m.ntail) if m.ntail else self.epi_in, M=m.width + m.ntail)
        return y, tail


class SequentialBlock(Block):
    def __init__(self, pk, cfg, mixer, ff, norm, scale):
        self.norm1, self.ls1, self.ff = norm("norm1"), scale("ls1"), ff
        self._input(pk, mixer)
        self.inp, self.out = Linear(mixer.w_in, pk.dtype), Linear(mixer.w_out, pk.dtype)
        self.epi_out = epilogue(_lib.DN_RESID, ls=self.ls1)
        pk.want(mid=mixer.nin)
        del mixer.w_in, mixer.w_out
        if ff is not None:
            self.norm2, self.ls2 = norm("norm2"), scale("ls2")
            self.gu, self.down = Linear(ff.w_gu, pk.dtype), Linear(ff.w_down, pk.dtype)
            self.epi_glu = epilogue(_lib.DN_GLU, glu=ff.glu)
            self.epi_down = epilogue(_lib.DN_RESID, ls=self.ls2)
            pk.want(mid=ff.F)
            del ff.w_gu, ff.w_down

    def step(self, pk, x, cache):
        b, m = pk.step, self.mixer
        y, mid, tail = b.y.data_ptr(), b.mid.data_ptr(), b.tail.data_ptr()
        self.inp.row(self.norm1.prologue(x), y, with_tail(self.epi_in, tail, m.ntail) if m.ntail else self.epi_in)
        self.out.row(m.step_core(pk, y, tail, mid, cache), x, self.epi_out)
        if self.ff is not None:
            self.gu.row(self.norm2.prologue(x), mid, self.epi_glu, M=self.ff.F)
            self.down.row(typed_input(mid), x, self.epi_down)

    def rows(self, pk, st, caches):
        R, Ep, m = st.R, st.ldx, self.mixer
        h = st.buf("h", R * Ep, pk.dtype)
        self.norm1.rows(st.x, Ep, h, Ep, pk.f32, R, Ep)
        y, tail = self._project_rows(pk, st, self.inp, h, Ep)
        X = st.buf("mid", R * m.nin, pk.dtype)
        m.rows_core(pk, st, y, tail, X, m.nin, caches)
        self.out.rows(X, m.nin, st.x, Ep, R, self.epi_out)
        if self.ff is not None:
            F = self.ff.F
            self.norm2.rows(st.x, Ep, h, Ep, pk.f32, R, Ep)
            f = st.buf("f", R * F, pk.dtype)
            self.gu.rows(h, Ep, f, F, R, self.epi_glu, M=F)
            self.down.rows(f, F, st.x, Ep, R, self.epi_down)


class ParallelBlock(Block):
    def __init__(self, pk, cfg, mixer, ff, norm, scale):
        self.norm1 = norm("norm1")
        self._input(pk, mixer)
        F = self.F = 0 if ff is None else ff.F
        self.nm = mixer.width + mixer.ntail                 # matrix rows of the mixer; gate and up rows follow
        w_in, w_out = mixer.w_in, mixer.w_out
        del mixer.w_in, mixer.w_out
        if F:
            w_in, w_out = torch.cat([w_in, ff.w_gu]), torch.cat([w_out, ff.w_down], dim=1)
            del ff.w_gu, ff.w_down
            self.epi_glu = epilogue(_lib.DN_GLU, glu=ff.glu)
        self.inp, self.out = Linear(w_in, pk.dtype), Linear(w_out, pk.dtype)
        self.mult = torch.full((pk.Ep,), float(cfg["residual_mult"]), dtype=torch.float32, device="cuda")
        self.epi_out = epilogue(_lib.DN_RESID, ls=self.mult)
        pk.want(mid=mixer.nin + F)

    def step(self, pk, x, cache):
        b, m, F = pk.step, self.mixer, self.F
        y, mid, tail = b.y.data_ptr(), b.mid.data_ptr(), b.tail.data_ptr()
        f = mid + m.nin * pk.esize
        e = with_tail(self.epi_in, tail, m.ntail) if m.ntail else _lib.DnEpilogue.from_buffer_copy(self.epi_in)
        if F:
            e.kind, e.glu_from, e.y2 = _lib.DN_STORE_GLU, self.nm, f
            e.glu_act, e.glu_alpha, e.glu_limit = self.epi_glu.glu_act, self.epi_glu.glu_alpha, self.epi_glu.glu_limit
        self.inp.row(self.norm1.prologue(x), y, e, M=self.nm + F)
        pro = m.step_core(pk, y, tail, mid, cache)
        if F and pro.kind == _lib.DN_IN_NORM:
            pro.n1, pro.x2 = m.nin, f                       # a typed input already has f behind it
        self.out.row(pro, x, self.epi_out)

    def rows(self, pk, st, caches):
        R, Ep, m, F = st.R, st.ldx, self.mixer, self.F
        h = st.buf("h", R * Ep, pk.dtype)
        self.norm1.rows(st.x, Ep, h, Ep, pk.f32, R, Ep)
        y, tail = self._project_rows(pk, st, self.inp, h, Ep)
        ld = m.nin + F
        X = st.buf("mid", R * ld, pk.dtype)
        if F:
            self.inp.rows(h, Ep, X + m.nin * pk.esize, ld, R, self.epi_glu, M=F, first=self.nm)
        m.rows_core(pk, st, y, tail, X, ld, caches)
        self.out.rows(X, ld, st.x, Ep, R, self.epi_out)


# --------------------------------------------------------------------------- a model's packed weights

class _Bufs:
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

        A = archs.of(cfg)

        def norm(name):
            return Norm(_pad_rows(w[name].float() + A.norm_offset, Ep), E, Ep, eps)

        def scale(name):
            return _pad_rows(w[name].float(), Ep).cuda() if name in w else None
        self.first_values = None                 # (heads, size) of the values that later layers mix in
        self.layers = []
        for i, ly in enumerate(cfg["layers"]):
            kind, mlp = ly["type"], ly.get("mlp")
            if kind not in A.mixers:
                raise NotImplementedError(f"layer {i}: mixer {kind!r}; known are {', '.join(sorted(A.mixers))}")
            mixer = A.mixers[kind](self, cfg, ly["mixer"], lambda n, p=f"l{i}.mix.": w[p + n])
            ff = None
            if mlp is not None:
                kind = mlp.get("kind", "dense")
                if kind not in A.feed_forwards:
                    raise NotImplementedError(f"layer {i}: feed-forward {kind!r}; known are {', '.join(sorted(A.feed_forwards))}")
                ff = A.feed_forwards[kind](self, cfg, mlp, lambda n, p=f"l{i}.mlp.": w[p + n])
            self.layers.append(A.block(self, cfg, mixer, ff, lambda n, p=f"l{i}.": norm(p + n), lambda n, p=f"l{i}.": scale(p + n)))
        if cfg.get("loop"):
            W = w["loop.in"]
            self.loop_in = Linear(_pad_rows(torch.cat([_pad_cols(W[:, :E], Ep), _pad_cols(W[:, E:], Ep)], dim=1), Ep), self.dtype)
            self.loop_step = _pad_cols(w["loop.step"].float(), Ep).cuda().contiguous()
            self.epi_loop = [epilogue(bias=self.loop_step[t], out_f32=True) for t in range(self.loop_step.shape[0])]
        self.embed_norm = (w["embed.norm"].float() + A.norm_offset).cuda() if A.embed_norm else None
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
        typed = dict(dtype=self.dtype, device="cuda")
        b.y, b.mid, b.vfirst = [torch.zeros(max(n.get(k, 0), 8), **typed) for k in ("y", "mid", "vfirst")]
        b.o, b.tail, b.ws = [torch.zeros(max(n.get(k, 0), 8), **f32) for k in ("o", "tail", "ws")]
        b.tickets = torch.zeros(max(n.get("tickets", 0), 1), dtype=torch.int32, device="cuda")
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
    """Nugusun, and what designs made of mixer layers have in common."""
    device_token = True
    max_rows = 2048
    mixers = MIXERS
    feed_forwards = {"dense": gelu_feed_forward}
    block = SequentialBlock
    norm_offset = 0.0       # added to stored norm weights
    embed_norm = False      # the embedding row is normed ("embed.norm")

    # ------------------------------------------------------------------ configuration and weights
    def config_from_json(self, js, dtype):
        if dtype not in DTYPES:
            raise ValueError(f"dtype {dtype!r}: known are {', '.join(sorted(DTYPES))}")
        cfg = {"arch": js["architecture"], "dtype": dtype, "n_layers": len(js["layers"]), "n_embd": int(js["width"]),
               "vocab": int(js["vocab"]), "norm_eps": float(js["norm"]["eps"]), "layers": js["layers"], **self.design_config(js)}
        lp = cfg["loop"]
        if lp is not None:
            if not (0 <= lp["start"] < lp["stop"] <= cfg["n_layers"] and lp["times"] >= 1):
                raise ValueError(f"loop {lp} over {cfg['n_layers']} layers")
        return cfg

    def design_config(self, js):
        """What only this design's config has."""
        return {"loop": js.get("loop"), "embed_scale": float(js["embedding"]["scale"])}

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

    def _embed_norm(self, pk, cfg):
        return (None if pk.embed_norm is None else pk.embed_norm.data_ptr()), cfg["norm_eps"]

    def embed_step(self, w, cfg, tok):
        pk = packed(w, cfg)
        b = pk.step
        if dr._DEVICE_EMBED is not None:
            tok_ptr = dr._DEVICE_EMBED[2]
        else:
            b.tok.fill_(int(tok.reshape(-1)[0]))
            tok_ptr = b.tok.data_ptr()
        b.cur = 0
        _lib.call("lt_dn_embed", pk.embed.data_ptr(), pk.f32, cfg["n_embd"], tok_ptr, cfg["embed_scale"],
                  *self._embed_norm(pk, cfg), b.x[0].data_ptr(), b.x0.data_ptr() if cfg["loop"] else None, cfg["n_embd"], pk.Ep, cfg["vocab"], 1, dr._stream())
        return b.x[0].data_ptr()

    def layer_step(self, w, cfg, run, x, cache):
        pk = packed(w, cfg)
        L, b = pk.layers[run.layer], pk.step
        if run.opens_pass:
            b.cur ^= 1
            nxt = b.x[b.cur].data_ptr()
            pk.loop_in.row(cast_input(x, pk.Ep, b.x0.data_ptr()), nxt, pk.epi_loop[run.loop_pass])
            x = nxt
        L.step(pk, x, cache)
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
        _lib.call("lt_dn_embed", pk.embed.data_ptr(), pk.f32, cfg["n_embd"], ids.data_ptr(), cfg["embed_scale"],
                  *self._embed_norm(pk, cfg), st.x, None if st._x0 is None else st._x0.data_ptr(), cfg["n_embd"], pk.Ep, cfg["vocab"], st.R, dr._stream())
        st.ids = ids
        return st

    def layer_rows(self, st, run, caches):
        pk, R, Ep = st.pk, st.R, st.ldx
        L = pk.layers[run.layer]
        if run.opens_pass:
            xx = st.buf("xx", R * 2 * Ep, pk.dtype)
            _lib.call("lt_dn_concat_rows", st.x, Ep, Ep, st._x0.data_ptr(), Ep, Ep, xx, 2 * Ep, pk.f32, R, dr._stream())
            pk.loop_in.rows(xx, 2 * Ep, st.x, Ep, R, pk.epi_loop[run.loop_pass])
        L.rows(pk, st, caches)

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


class Pakalix(Layered):
    feed_forwards = {"dense": clamped_feed_forward}
    block = ParallelBlock
    norm_offset = 1.0
    embed_norm = True

    def design_config(self, js):
        return {"loop": None, "embed_scale": 1.0, "residual_mult": float(js["residual_mult"])}


ARCH = Layered()
PAKALIX = Pakalix()
