"""Plain CPU restatement of the decoder made of per-layer mixers (config "layers": gated linear attention,
lightning attention, windowed latent attention; loops over a range of layers; layer scale).

TEST INFRASTRUCTURE ONLY: one slow numpy function per mechanism, written from the equations, token by token where
the mechanism is a recurrence; it shares no code with the product.  Everything is computed in `F` (float64 by
default), so a difference from the product is the product's rounding.

Notation: x residual stream [T, E]; h a normed input [T, E]; tensors are a dict name -> array, linears [out, in].
"""
import numpy as np

F = np.float64


def linear(W, x):
    return x @ np.asarray(W, F).T


def rms(x, w, eps):
    x = np.asarray(x, F)
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + F(eps)) * np.asarray(w, F)


def sigmoid(z):
    z = np.asarray(z, F)
    return np.where(z >= 0, 1 / (1 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1 + np.tanh(np.sqrt(2 / np.pi) * (z + 0.044715 * z ** 3)))


def rotate_half(x, pos, base, dims):
    """x [T, ..., d]: the first `dims` of the last axis are rotated, component i with component i + dims/2, by the
    angle pos * base^(-2 i / dims)."""
    half = dims // 2
    f = F(base) ** (-2.0 * np.arange(half) / dims)
    ang = np.asarray(pos, F).reshape((-1,) + (1,) * (x.ndim - 1)) * f
    c, s = np.cos(ang), np.sin(ang)
    out = np.array(x, F)
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


def decayed_outer_recurrence(q, k, v, alpha, S):
    """S <- diag(alpha_t) S + k_t v_t^T;  o_t = S^T q_t, per head.  q, k, alpha [T, H, d], v [T, H, dv],
    S [H, d, dv] (updated in place).  Returns o [T, H, dv]."""
    o = np.zeros(v.shape, F)
    for t in range(q.shape[0]):
        S *= alpha[t][:, :, None]
        S += k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    return o


def gla(h, m, w, eps, S):
    """Gated linear attention of mixer config m; w(name) gives the mixer's tensors; S the carried state."""
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = linear(w("q"), h).reshape(T, H, d) * F(d) ** -0.5
    k = linear(w("k"), h).reshape(T, H, d)
    v = linear(w("v"), h).reshape(T, H, dv)
    z = linear(w("a2"), linear(w("a1"), h)) + np.asarray(w("a2.b"), F)
    alpha = (sigmoid(z) ** (1 / F(m["tau"]))).reshape(T, H, d)
    o = decayed_outer_recurrence(q, k, v, alpha, S)
    o = rms(o, w("norm"), eps).reshape(T, H * dv)
    return linear(w("o"), o * silu(linear(w("g"), h)))


def lightning(h, m, w, eps, S):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(linear(w("q"), h)).reshape(T, H, d)
    k = silu(linear(w("k"), h)).reshape(T, H, d)
    v = silu(linear(w("v"), h)).reshape(T, H, dv)
    alpha = np.broadcast_to(np.asarray(m["decay"], F)[None, :, None], (T, H, d))
    o = decayed_outer_recurrence(q, k, v, alpha, S).reshape(T, H * dv)
    return linear(w("o"), rms(o, w("norm"), eps) * sigmoid(linear(w("g"), h)))


def window_visible(i, n, size):
    """Indices j <= i of the last `size` positions, the query's own included."""
    return np.arange(max(0, i - size + 1), min(i + 1, n))


def latent_attention(h, m, w, eps, cache, pos0):
    """cache: dict with lists 'c' and 'kr', one entry per position so far (appended here)."""
    T, H, d, dr, dv, r = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(pos0, pos0 + T)
    q = linear(w("q"), h).reshape(T, H, d + dr)
    qn, qr = q[..., :d], rotate_half(q[..., d:], pos, m["rot"]["base"], m["rot"]["dims"])
    ckr = linear(w("dkv"), h)
    cache["c"] += list(rms(ckr[:, :r], w("dkv.norm"), eps))
    cache["kr"] += list(rotate_half(ckr[:, r:], pos, m["rot"]["base"], m["rot"]["dims"]))
    c, kr = np.array(cache["c"]), np.array(cache["kr"])
    kn = linear(w("uk"), c).reshape(-1, H, d)
    v = linear(w("uv"), c).reshape(-1, H, dv)
    out = np.zeros((T, H, dv), F)
    for t in range(T):
        j = window_visible(pos0 + t, c.shape[0], m["mask"]["size"])
        s = (np.einsum("hd,jhd->hj", qn[t], kn[j]) + np.einsum("hd,jd->hj", qr[t], kr[j])) * F(m["scale"])
        p = np.exp(s - s.max(axis=1, keepdims=True))
        p /= p.sum(axis=1, keepdims=True)
        out[t] = np.einsum("hj,jhv->hv", p, v[j])
    return linear(w("o"), out.reshape(T, H * dv))


def feed_forward(h, w):
    return linear(w("down"), gelu_tanh(linear(w("gate"), h)) * linear(w("up"), h))


def layer_runs(cfg):
    """[(layer, pass or None)] in the order they run; pass is None outside the loop."""
    n = len(cfg["layers"])
    lp = cfg.get("loop")
    if not lp:
        return [(i, None) for i in range(n)]
    return ([(i, None) for i in range(lp["start"])] +
            [(i, t) for t in range(lp["times"]) for i in range(lp["start"], lp["stop"])] +
            [(i, None) for i in range(lp["stop"], n)])


class Model:
    """One sequence: run(tokens) advances it and returns the logits of those tokens."""

    def __init__(self, cfg, tensors):
        self.cfg = cfg
        self.w = {k: np.asarray(v, F if np.asarray(v).dtype.kind == "f" else np.int32) for k, v in tensors.items()}
        self.runs = layer_runs(cfg)
        self.pos = 0
        self.state = []
        for i, _t in self.runs:
            m = cfg["layers"][i]["mixer"]
            if cfg["layers"][i]["type"] == "latent_attention":
                self.state.append({"c": [], "kr": []})
            else:
                self.state.append(np.zeros((m["heads"], m["dim"], m["vdim"]), F))
        self.taps = []

    def layer(self, i, x, st):
        ly, eps, p = self.cfg["layers"][i], self.cfg["norm"]["eps"], f"l{i}."
        mix = lambda n: self.w[p + "mix." + n]
        h = rms(x, self.w[p + "norm1"], eps)
        if ly["type"] == "gla":
            y = gla(h, ly["mixer"], mix, eps, st)
        elif ly["type"] == "lightning":
            y = lightning(h, ly["mixer"], mix, eps, st)
        else:
            y = latent_attention(h, ly["mixer"], mix, eps, st, self.pos)
        x = x + y * self.w[p + "ls1"]
        if ly["mlp"] is not None:
            x = x + feed_forward(rms(x, self.w[p + "norm2"], eps), lambda n: self.w[p + "mlp." + n]) * self.w[p + "ls2"]
        return x

    def run(self, tokens):
        cfg, w = self.cfg, self.w
        x0 = w["embed"][np.asarray(tokens)] * F(cfg["embedding"]["scale"])
        x = x0
        self.taps = []
        for st, (i, t) in zip(self.state, self.runs):
            if t is not None and i == cfg["loop"]["start"]:
                x = linear(w["loop.in"], np.concatenate([x, x0], axis=1)) + w["loop.step"][t]
            x = self.layer(i, x, st)
            self.taps.append(x)
        self.pos += len(tokens)
        return linear(w["head"], rms(x, w["final.norm"], cfg["norm"]["eps"]))
