"""Plain CPU restatement of the Pakalix decoder: parallel blocks (mixer and feed-forward read one norm), mixers Mamba-2 and
grouped-query attention (norm over the whole query / key projection, rotation, capped scores, value mixing, gate per head),
feed-forward with clamped gate and up.

TEST INFRASTRUCTURE ONLY: one slow numpy function per mechanism, written from the equations, token by token where the
mechanism is a recurrence; it shares no code with the product.  Everything is computed in float64.

Notation: x residual stream [T, E]; h a normed input [T, E]; tensors are a dict name -> array, linears [out, in].
"""
import numpy as np

from .layered import F, linear, rms, rotate_half, sigmoid, silu


def one_plus_rms(x, w, eps):
    return rms(x, 1.0 + np.asarray(w, F), eps)


def softplus(z):
    z = np.asarray(z, F)
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def causal_conv(u, taps, bias, before):
    """y_t = bias + sum_i taps[:, i] * u_(t - n + 1 + i) per channel, n = number of taps.  u [T, C], taps [C, n]; before
    [n - 1, C] are the inputs ahead of u (zeros at the start of a sequence).  Returns (y, the next `before`)."""
    taps = np.asarray(taps, F)
    n = taps.shape[1]
    ext = np.concatenate([before, u], axis=0)
    y = np.tile(np.asarray(bias, F), (u.shape[0], 1))
    for t in range(u.shape[0]):
        for i in range(n):
            y[t] += taps[:, i] * ext[t + i]
    return y, ext[ext.shape[0] - (n - 1):]


def ssd_recurrence(x, B, C, dt, A, D, S):
    """S <- exp(A_h dt_t) S + dt_t B_t x_t^T;  y_t = S^T C_t + D_h x_t, head by head.
    x [T, H, P], B and C [T, G, N], dt [T, H], A and D [H], S [H, N, P] (updated in place)."""
    T, H, _ = x.shape
    per = H // B.shape[1]
    y = np.zeros(x.shape, F)
    for t in range(T):
        for h in range(H):
            g = h // per
            S[h] = np.exp(A[h] * dt[t, h]) * S[h] + dt[t, h] * np.outer(B[t, g], x[t, h])
            y[t, h] = S[h].T @ C[t, g] + D[h] * x[t, h]
    return y


def rms_in_parts(y, w, parts, eps):
    T, n = y.shape
    p = y.reshape(T, parts, n // parts)
    p = p / np.sqrt(np.mean(p * p, axis=-1, keepdims=True) + F(eps))
    return p.reshape(T, n) * np.asarray(w, F)


def mamba2(h, m, w, eps, st):
    """st: {'S': [H, N, P], 'before': [taps - 1, channels]}"""
    T, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    y = linear(w("in"), h)
    z, xbc, dt = np.split(y, [inner, inner + inner + 2 * G * N], axis=1)
    xbc, st["before"] = causal_conv(xbc, w("conv"), w("conv.b"), st["before"])
    x, B, C = np.split(silu(xbc), [inner, inner + G * N], axis=1)
    dt = softplus(dt + np.asarray(w("dt_bias"), F))
    o = ssd_recurrence(x.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N), dt, -np.exp(np.asarray(w("A_log"), F)),
                       np.asarray(w("D"), F), st["S"]).reshape(T, inner)
    return linear(w("o"), rms_in_parts(o * silu(z), w("norm"), m["norm_groups"], eps))


def capped(s, cap):
    return cap * np.tanh(s / cap)


def softmax_over(s):
    p = np.exp(s - s.max(axis=-1, keepdims=True))
    return p / p.sum(axis=-1, keepdims=True)


def grouped_attention(h, m, w, eps, st, pos0, first_v):
    """st: {'k': [...], 'v': [...]} one entry per position so far.  first_v: {} or {'v': [T, G * dv]} (the values of the first
    mixing layer for these tokens; filled by that layer)."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = np.arange(pos0, pos0 + T)
    rot = lambda a, n: rotate_half(a.reshape(T, n, d), pos, m["rot"]["base"], m["rot"]["dims"])
    q = rot(rms(linear(w("q"), h), w("q.norm"), eps), H)
    k = rot(rms(linear(w("k"), h), w("k.norm"), eps), G)
    v = linear(w("v"), h)
    if m.get("v_mix"):
        if "v" not in first_v:
            first_v["v"] = v
        else:
            lam = float(np.asarray(w("vmix"), F).reshape(()))
            v = (1 - lam) * v + lam * first_v["v"]
    st["k"] += list(k)
    st["v"] += list(v.reshape(T, G, dv))
    K, V = np.array(st["k"]), np.array(st["v"])
    out = np.zeros((T, H, dv), F)
    for t in range(T):
        n = pos0 + t + 1
        for hh in range(H):
            g = hh // (H // G)
            s = K[:n, g] @ q[t, hh] * F(m["scale"])
            if m.get("softcap"):
                s = capped(s, F(m["softcap"]))
            out[t, hh] = softmax_over(s) @ V[:n, g]
    out *= sigmoid(linear(w("g"), h))[:, :, None]
    return linear(w("o"), out.reshape(T, H * dv))


def clamped_feed_forward(h, w, limit):
    g = np.minimum(linear(w("gate"), h), limit)
    u = np.clip(linear(w("up"), h), -limit, limit)
    return linear(w("down"), g * sigmoid(1.702 * g) * (u + 1))


class Model:
    """One sequence: run(tokens) advances it and returns the logits of those tokens."""

    def __init__(self, cfg, tensors):
        self.cfg = cfg
        self.w = {k: np.asarray(v, F) for k, v in tensors.items()}
        self.pos = 0
        self.state = []
        for i, ly in enumerate(cfg["layers"]):
            m = ly["mixer"]
            if ly["type"] == "mamba2":
                ch, taps = self.w[f"l{i}.mix.conv"].shape
                self.state.append({"S": np.zeros((m["heads"], m["state"], m["vdim"]), F), "before": np.zeros((taps - 1, ch), F)})
            else:
                self.state.append({"k": [], "v": []})
        self.taps = []

    def run(self, tokens):
        cfg, w, eps = self.cfg, self.w, self.cfg["norm"]["eps"]
        x = one_plus_rms(w["embed"][np.asarray(tokens)], w["embed.norm"], eps)
        self.taps, first_v = [], {}
        for i, (ly, st) in enumerate(zip(cfg["layers"], self.state)):
            mix = lambda n: w[f"l{i}.mix." + n]
            h = one_plus_rms(x, w[f"l{i}.norm1"], eps)
            if ly["type"] == "mamba2":
                y = mamba2(h, ly["mixer"], mix, eps, st)
            else:
                y = grouped_attention(h, ly["mixer"], mix, eps, st, self.pos, first_v)
            if ly["mlp"] is not None:
                y = y + clamped_feed_forward(h, lambda n: w[f"l{i}.mlp." + n], ly["mlp"]["limit"])
            x = x + cfg["residual_mult"] * y
            self.taps.append(x)
        self.pos += len(tokens)
        return linear(w["head"], one_plus_rms(x, w["final.norm"], eps))
