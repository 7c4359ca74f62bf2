"""Prefill and decode throughput of the mixer-layer models (`layered`) beside the Q8_0 llama block at equal size, and the
time of every kernel against its roofline.  `bench.py --layered`; every number is CUDA events on the launching stream
after warm-up, weights are random.

A size names width, feed-forward, heads and head size; the mixer model's layers are, in turn, lightning, gla, latent
attention (window as given) and gla, the llama model has the same number of attention blocks of the same sizes.  The Pakalix
model has three Mamba-2 layers (inner size twice the width, heads of 64, state 128) to one of grouped-query attention.
"""
import ctypes

import numpy as np
import torch

from . import _lib, archs, dense_ops, layered
from . import dev_residency as dr
from . import prefill as pf
from .fact_dispatch import Q8Weight
from .measure import peaks

SIZES = {
    "0.5b": dict(E=896, F=4864, H=14, nkv=2, hd=64, rank_a=16, kv_rank=256, rot=32, window=1024, layers=8, V=32768),
    "3b": dict(E=2048, F=8192, H=16, nkv=4, hd=128, rank_a=16, kv_rank=512, rot=64, window=2048, layers=8, V=32768),
    "8b": dict(E=4096, F=14336, H=32, nkv=8, hd=128, rank_a=32, kv_rank=512, rot=64, window=4096, layers=4, V=32768),
}
KINDS = ("lightning", "gla", "latent_attention", "gla")
PAKALIX_KINDS = ("mamba2", "attention", "mamba2", "mamba2")


def ssd_sizes(s):
    """heads, value size, state, groups, taps of the Mamba-2 layers of a size"""
    return 2 * s["E"] // 64, 64, 128, 1, 4


def mixer_model(s, dtype="bfloat16", seed=0):
    """(cfg, w) of the mixer model of a size, random weights (made on the GPU, kept on the host)."""
    g = torch.Generator(device="cuda").manual_seed(seed)
    E, F, H, hd, V = s["E"], s["F"], s["H"], s["hd"], s["V"]

    def lin(o, i):
        return (torch.randn(o, i, generator=g, device="cuda") / i ** 0.5).bfloat16().cpu()

    def vec(n, m=1.0):
        return (m + 0.1 * torch.randn(n, generator=g, device="cuda")).bfloat16().cpu()
    w = {"embed": lin(V, E), "final.norm": vec(E), "head": lin(V, E)}
    layers = []
    for i in range(s["layers"]):
        kind, p = KINDS[i % len(KINDS)], f"l{i}.mix."
        w[f"l{i}.norm1"], w[f"l{i}.norm2"], w[f"l{i}.ls1"], w[f"l{i}.ls2"] = vec(E), vec(E), vec(E, 0.5), vec(E, 0.5)
        if kind == "latent_attention":
            m = {"heads": H, "dim": hd, "rot_dim": s["rot"], "vdim": hd, "kv_rank": s["kv_rank"], "mask": {"size": s["window"]},
                 "rot": {"base": 10000.0, "dims": s["rot"]}, "scale": (hd + s["rot"]) ** -0.5}
            w[p + "q"], w[p + "dkv"] = lin(H * (hd + s["rot"]), E), lin(s["kv_rank"] + s["rot"], E)
            w[p + "dkv.norm"] = vec(s["kv_rank"])
            w[p + "uk"], w[p + "uv"] = lin(H * hd, s["kv_rank"]), lin(H * hd, s["kv_rank"])
        else:
            m = {"heads": H, "dim": hd, "vdim": hd}
            for n in "qkvg":
                w[p + n] = lin(H * hd, E)
            if kind == "gla":
                m["tau"] = 16.0
                w[p + "a1"], w[p + "a2"], w[p + "a2.b"], w[p + "norm"] = lin(s["rank_a"], E), lin(H * hd, s["rank_a"]), vec(H * hd), vec(hd)
            else:
                m["decay"] = [float(1 - 2.0 ** -(1 + 8 * h / H)) for h in range(H)]
                w[p + "norm"] = vec(H * hd)
        w[p + "o"] = lin(E, H * hd)
        for n, o, k in (("gate", F, E), ("up", F, E), ("down", E, F)):
            w[f"l{i}.mlp.{n}"] = lin(o, k)
        layers.append({"type": kind, "mixer": m, "mlp": {"kind": "dense", "ff": F}})
    js = {"architecture": "Nugusun", "embedding": {"scale": 1.0}, "layers": layers, "norm": {"eps": 1e-6}, "vocab": V, "width": E}
    cfg = layered.ARCH.config_from_json(js, dtype)
    return cfg, layered.DenseWeights(w)


def pakalix_model(s, dtype="bfloat16", seed=0):
    """(cfg, w) of the Pakalix model of a size, random weights."""
    g = torch.Generator(device="cuda").manual_seed(seed)
    E, F, H, hd, V, G = s["E"], s["F"], s["H"], s["hd"], s["V"], s["nkv"]
    SH, P, N, SG, taps = ssd_sizes(s)

    def lin(o, i):
        return (torch.randn(o, i, generator=g, device="cuda") / i ** 0.5).bfloat16().cpu()

    def vec(n, m=0.0):
        return (m + 0.1 * torch.randn(n, generator=g, device="cuda")).bfloat16().cpu()
    w = {"embed": lin(V, E), "embed.norm": vec(E), "final.norm": vec(E), "head": lin(V, E)}
    layers = []
    for i in range(s["layers"]):
        kind, p = PAKALIX_KINDS[i % len(PAKALIX_KINDS)], f"l{i}.mix."
        w[f"l{i}.norm1"] = vec(E)
        if kind == "attention":
            m = {"heads": H, "kv_heads": G, "dim": hd, "vdim": hd, "rot": {"base": 10000.0, "dims": hd}, "scale": hd ** -0.5, "softcap": 30.0,
                 "v_mix": True}
            w[p + "q"], w[p + "k"], w[p + "v"], w[p + "g"], w[p + "o"] = lin(H * hd, E), lin(G * hd, E), lin(G * hd, E), lin(H, E), lin(E, H * hd)
            w[p + "q.norm"], w[p + "k.norm"], w[p + "vmix"] = vec(H * hd, 1.0), vec(G * hd, 1.0), torch.tensor(0.4).bfloat16()
        else:
            m = {"heads": SH, "groups": SG, "vdim": P, "state": N, "conv": taps, "norm_groups": 1}
            inner, ch = SH * P, SH * P + 2 * SG * N
            w[p + "in"], w[p + "conv"], w[p + "conv.b"], w[p + "norm"], w[p + "o"] = lin(inner + ch + SH, E), lin(ch, taps), vec(ch), vec(inner, 1.0), lin(E, inner)
            w[p + "dt_bias"], w[p + "A_log"], w[p + "D"] = vec(SH, -2.0), vec(SH, 0.5), vec(SH, 1.0)
        for n, o, k in (("gate", F, E), ("up", F, E), ("down", E, F)):
            w[f"l{i}.mlp.{n}"] = lin(o, k)
        layers.append({"type": kind, "mixer": m, "mlp": {"kind": "dense", "ff": F, "limit": 7.0}})
    js = {"architecture": "Pakalix", "layers": layers, "norm": {"eps": 1e-6}, "residual_mult": 0.25, "vocab": V, "width": E}
    cfg = layered.PAKALIX.config_from_json(js, dtype)
    return cfg, layered.DenseWeights(w)


def llama_model(s, seed=0):
    """(cfg, w) of the llama block of a size with random Q8_0 blocks."""
    rng = np.random.default_rng(seed)
    pool = rng.integers(-127, 128, size=1 << 24, dtype=np.int8)

    def q8(N, K):
        return Q8Weight(np.resize(pool, N * K), np.full(N * (K // 32), K ** -0.5 / 73.0, np.float16), N, K)

    def vec(n):
        return torch.from_numpy((1 + 0.1 * rng.standard_normal(n)).astype(np.float32))
    E, F, V, nq, nk = s["E"], s["F"], s["V"], s["H"] * s["hd"], s["nkv"] * s["hd"]
    w = {"token_embd.weight": q8(V, E), "output_norm.weight": vec(E)}
    for i in range(s["layers"]):
        p = f"blk.{i}"
        w[p + ".attn_norm.weight"], w[p + ".ffn_norm.weight"] = vec(E), vec(E)
        for n, o, k in (("attn_q", nq, E), ("attn_k", nk, E), ("attn_v", nk, E), ("attn_output", E, nq), ("ffn_gate", F, E),
                        ("ffn_up", F, E), ("ffn_down", E, F)):
            w[f"{p}.{n}.weight"] = q8(o, k)
    cfg = dict(n_layers=s["layers"], n_head=s["H"], n_head_kv=s["nkv"], n_embd=E, rope_theta=1e6, norm_eps=1e-6, arch="llama")
    return cfg, w


def run_model(cfg, w, tokens, steps, reps=5, warmup=3):
    """Throughput of one sequence: a prompt of `tokens`, then `steps` tokens with the loop on the device."""
    A = archs.of(cfg)
    dr._KV_MAX_SEQ = max(256, tokens + steps * 2 + 64)
    V = 32768
    toks = torch.from_numpy(np.random.default_rng(1).integers(0, V, tokens))
    ms = []
    for r in range(warmup + reps):
        kv = [None] * A.n_slots(cfg)
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        for c0 in range(0, tokens, A.max_rows):
            pf.prefill_resident(w, cfg, toks[c0:c0 + A.max_rows], kv, want_logits=c0 + A.max_rows >= tokens)
        e1.record()
        torch.cuda.synchronize()
        ms.append(e0.elapsed_time(e1))
    pre = float(np.median(ms[warmup:]))
    kv = [None] * A.n_slots(cfg)
    gr = dr.GraphRunner(w, cfg, kv)
    gr.seed(toks, torch.arange(tokens))
    gr.capture_device_loop(1, capacity=4 * steps + 64)
    gr.replay_device(max(3, steps // 4))
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    with torch.cuda.stream(gr.stream):
        e0.record()
    gr.replay_device(steps)
    with torch.cuda.stream(gr.stream):
        e1.record()
    torch.cuda.synchronize()
    dec = e0.elapsed_time(e1) / steps
    return {"prefill_tok_s": tokens / pre * 1e3, "prefill_ms": pre, "decode_tok_s": 1e3 / dec, "decode_us": dec * 1e3,
            "launches_per_token": gr.launches_per_step}


# --------------------------------------------------------------------------- kernels one by one

def _chain_us(fns, reps=6):
    """Device time per launch of a captured chain of launches (rotating buffers: nothing is found in L2)."""
    side = torch.cuda.Stream()
    for f in fns[:3]:
        f()
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g, stream=side):
        for f in fns:
            f()
    with torch.cuda.stream(side):
        for _ in range(3):
            g.replay()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        for _ in range(reps):
            g.replay()
        e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) * 1e3 / reps / len(fns)


def _copies(nbytes):
    return int(max(3, min(64, (400 << 20) // max(nbytes, 1))))


def kernel_times(s, T, only=None):
    """[{kernel, us, roofline_us, frac, bound}] of the new kernels and of the like kernels of the Q8_0 block."""
    hbm, tf, _src = peaks()
    E, F, H, hd, W, r, rot = s["E"], s["F"], s["H"], s["hd"], s["window"], s["kv_rank"], s["rot"]
    dev = dict(device="cuda")
    out = []

    def add(name, us, nbytes, flops, like=None):
        tb, tc = nbytes / hbm * 1e-3, flops / tf * 1e-6
        roof = max(tb, tc)
        out.append({"kernel": name, "us": round(us, 2), "roofline_us": round(roof, 2), "frac": round(roof / us, 4),
                    "bound": "hbm" if tb >= tc else "tensor", "like": like})

    def st():
        return dr._stream()

    def want(name):
        return only is None or any(o in name for o in only)
    bf = lambda *sh: torch.randn(*sh, device="cuda").bfloat16()
    i8 = lambda n: torch.randint(-127, 128, (n,), dtype=torch.int8, **dev)
    f16 = lambda n: torch.full((n,), 0x2000, dtype=torch.int16, **dev)

    # ---- linears over a prompt
    for name, M, K, kind in (("qkvg", 4 * H * hd, E, 0), ("o", E, H * hd, 1), ("gate|up", F, E, 2), ("down", E, F, 1)):
        if not want("linear"):
            break
        rows = 2 * M if kind == 2 else M
        n = _copies(rows * K * 2 + T * K * 2)
        Ws = [bf(rows, K) for _ in range(n)]
        Xs = [bf(T, K) for _ in range(n)]
        Y = torch.zeros(T, M, dtype=torch.float32 if kind == 1 else torch.bfloat16, **dev)
        e = dense_ops.epilogue(kind, segs=[(M, "silu", 1.0)] if kind == 0 else ())
        us = _chain_us([lambda W=W_, X=X_: _lib.call("lt_dn_linear", W.data_ptr(), K, X.data_ptr(), K, Y.data_ptr(), M, 0, M, K, T,
                                                     ctypes.byref(e), 0, st()) for W_, X_ in zip(Ws, Xs)])
        add(f"linear {name} {rows}x{K}, {T} rows", us, rows * K * 2 + T * K * 2 + T * M * (8 if kind == 1 else 2), 2.0 * rows * K * T, "q8 gemm")
        del Ws, Xs
        qn = rows if name != "qkvg" else (H + 2 * s["nkv"]) * hd
        n = 3
        q, d, xq, xd = [i8(qn * K) for _ in range(n)], f16(qn * K // 32), i8(T * K), f16(T * K // 32)
        Yq = torch.zeros(T, qn, **dev)
        us = _chain_us([lambda q=q_: _lib.call("lt_q8_gemm_tc", q.data_ptr(), d.data_ptr(), xq.data_ptr(), xd.data_ptr(), None, 0, Yq.data_ptr(),
                                               qn, K, T, 0, st()) for q_ in q], reps=3)
        # roofline of the Q8_0 form: int8 tensor rate is twice the bf16 one
        add(f"q8 gemm {name} {qn}x{K}, {T} rows", us, qn * K * 34 // 32 + T * K * 34 // 32 + T * qn * 4, 1.0 * qn * K * T)
        del q, Yq
    # ---- linears of one token
    for name, M, K, kind in (("qkvg", 4 * H * hd, E, 0), ("o", E, H * hd, 1), ("gate|up", F, E, 2), ("down", E, F, 1), ("head", s["V"], E, 0)):
        if not want("gemv"):
            break
        rows = 2 * M if kind == 2 else M
        n = _copies(rows * K * 2)
        Ws = [bf(rows, K) for _ in range(n)]
        x, w = torch.randn(K, **dev), torch.ones(K)
        nm = dense_ops.Norm(w, K, K, 1e-6)
        xt = bf(K)
        pro = dense_ops.typed_input(xt.data_ptr()) if name == "down" else nm.prologue(x.data_ptr())
        Y = torch.zeros(M, **dev)
        e = dense_ops.epilogue(kind, out_f32=True)
        us = _chain_us([lambda W=W_: _lib.call("lt_dn_gemv", W.data_ptr(), K, Y.data_ptr(), 0, M, K, ctypes.byref(pro), ctypes.byref(e), st())
                        for W_ in Ws])
        add(f"gemv {name} {rows}x{K}", us, rows * K * 2, 0, "q8 gemv")
        del Ws
        qn = rows if name != "qkvg" else (H + 2 * s["nkv"]) * hd
        n = _copies(qn * K)
        q, d = [i8(qn * K) for _ in range(n)], [f16(qn * K // 32) for _ in range(n)]
        wn, Yq, xq, xd = torch.ones(K, **dev), torch.zeros(qn, **dev), i8(K), f16(K // 32)
        if name in ("o", "down"):
            one = lambda q, d: _lib.call("lt_q8_gemv", q.data_ptr(), d.data_ptr(), xq.data_ptr(), xd.data_ptr(), None, Yq.data_ptr(), qn, K, 1, st())
        else:
            one = lambda q, d: _lib.call("lt_rmsnorm_q8_gemv", q.data_ptr(), d.data_ptr(), x.data_ptr(), wn.data_ptr(), 1e-6, None, Yq.data_ptr(),
                                         qn, K, st())
        us = _chain_us([lambda q=q_, d=d_: one(q, d) for q_, d_ in zip(q, d)])
        add(f"q8 gemv {name} {qn}x{K}", us, qn * K * 34 // 32, 0)
        del q, d
    # ---- recurrence
    nk, ld = H * hd, 4 * H * hd
    if want("recurrence"):
        n = _copies(T * ld * 2)
        ys = [(torch.randn(T, ld, device="cuda") * 0.3).bfloat16() for _ in range(n)]
        o = torch.empty(T, nk, **dev)
        S = torch.zeros(H, hd, hd, **dev)
        la = -torch.rand(T, nk, **dev) * 0.1
        lam = torch.full((H,), 0.95, **dev)
        ws = torch.empty(_lib.dense().lt_dn_recurrence_chunked_ws(T, H, hd, hd), **dev)
        for kind in ("gla", "lightning"):
            dec = _lib.DnDecay()
            if kind == "gla":
                dec.la, dec.ldla = la.data_ptr(), nk
            else:
                dec.decay = lam.data_ptr()
            us = _chain_us([lambda y=y_: _lib.call("lt_dn_recurrence_chunked", y.data_ptr(), y.data_ptr() + nk * 2, y.data_ptr() + 4 * nk, ld,
                                                   S.data_ptr(), o.data_ptr(), nk, T, H, hd, hd, ctypes.byref(dec), ws.data_ptr(), st()) for y_ in ys])
            nb = T * nk * (3 * 2 + 4 + (4 if kind == "gla" else 0))
            add(f"recurrence {kind}, {H} heads of {hd}, {T} rows", us, nb, 2.0 * T * H * (2 * hd * hd + 64 * hd), "q8 attention prompt")
        Ss = [torch.zeros(H, hd, hd, **dev) for _ in range(_copies(H * hd * hd * 4))]
        a2, b, a1 = bf(nk, s["rank_a"]), torch.zeros(nk, **dev), bf(s["rank_a"])
        y = ys[0]
        for kind in ("gla", "lightning"):
            dec = _lib.DnDecay()
            if kind == "gla":
                dec.a1, dec.a2, dec.lda2, dec.rank, dec.bias, dec.inv_tau = a1.data_ptr(), a2.data_ptr(), s["rank_a"], s["rank_a"], b.data_ptr(), 0.06
            else:
                dec.decay = lam.data_ptr()
            us = _chain_us([lambda S=S_: _lib.call("lt_dn_recurrence", y.data_ptr(), y.data_ptr() + nk * 2, y.data_ptr() + 4 * nk, ld, S.data_ptr(),
                                                   o.data_ptr(), nk, 0, 1, H, hd, hd, ctypes.byref(dec), st()) for S_ in Ss])
            add(f"recurrence {kind}, one token", us, 2 * H * hd * hd * 4, 0, "q8 attention token")
        del ys, Ss
    # ---- attention
    if want("latent"):
        hs, wr = hd + rot, r + rot
        cap = W - 1 + T
        freq, cn = torch.rand(rot // 2, **dev), torch.ones(r, **dev)
        L = _lib.DnLatent(H, hd, rot, hd, rot, r, r, W, cap, hs ** -0.5, 1e-6, freq.data_ptr(), cn.data_ptr())
        wy = H * hs + wr
        np_ = 0
        y = bf(T, wy)
        kv, kr = bf(T, 2 * nk), bf(T, wr)
        att = torch.empty(T, nk, dtype=torch.bfloat16, **dev)
        ring = bf(cap, wr)
        keys = torch.empty(T, wr, dtype=torch.bfloat16, **dev)
        pairs = sum(min(t + 1, W) for t in range(T))
        us = _chain_us([lambda: _lib.call("lt_dn_window_attn", y.data_ptr(), wy, kv.data_ptr(), 2 * nk, kr.data_ptr() + r * 2, wr,
                                          kv.data_ptr() + nk * 2, 2 * nk, att.data_ptr(), nk, 0, T, np_, ctypes.byref(L), st())] * 4)
        add(f"latent window attention, {H} heads, {T} rows, window {W}", us, T * (H * hs + 3 * nk) * 2, 2.0 * pairs * H * (hs + hd), "q8 attention prompt")
        us = _chain_us([lambda: _lib.call("lt_dn_latent_rows", y.data_ptr(), wy, ring.data_ptr(), keys.data_ptr(), 0, 0, 0, T, ctypes.byref(L), st())] * 4)
        add(f"latent rows, {T} rows", us, T * (2 * H * rot + 3 * wr) * 2, 0, None)
        groups = (H + 7) // 8
        splits = max(1, min((W + 31) // 32, 148 // groups))
        ukT, uv = [bf(H * r, hd) for _ in range(8)], [bf(H * hd, r) for _ in range(8)]
        rings = [bf(cap, wr) for _ in range(8)]
        ws = torch.empty(_lib.dense().lt_dn_latent_step_ws(H, r, rot, splits), **dev)
        ln = torch.full((1,), T, dtype=torch.int32, **dev)
        us = _chain_us([lambda i=i: _lib.call("lt_dn_latent_step", y.data_ptr(), rings[i % 8].data_ptr(), ln.data_ptr(), ukT[i % 8].data_ptr(),
                                              uv[i % 8].data_ptr(), att.data_ptr(), 0, ctypes.byref(L), splits, ws.data_ptr(), st()) for i in range(16)])
        add(f"latent step (3 launches), window {W}", us, min(T, W) * wr * 2 + 2 * H * hd * r * 2, 0, "q8 attention token")
    if want("latent") or want("recurrence"):
        nq, kvw = H * hd, s["nkv"] * hd
        qkv = torch.randn(T, nq + 2 * kvw, **dev)
        kc, vc = torch.randn(T + 8, kvw, **dev), torch.randn(T + 8, kvw, **dev)
        yq = torch.empty(T, nq, **dev)
        ln = torch.full((1,), T, dtype=torch.int32, **dev)      # the rows are already appended
        us = _chain_us([lambda: _lib.call("lt_attn_prefill", qkv.data_ptr(), nq + 2 * kvw, kc.data_ptr(), vc.data_ptr(), ln.data_ptr(), yq.data_ptr(),
                                          nq, hd, H, s["nkv"], float(hd ** -0.5), T, T, st())] * 2, reps=2)
        add(f"q8 attention prompt, {T} rows", us, T * (2 * nq + 2 * kvw) * 4, 2.0 * (T * T // 2) * H * 2 * hd)
        us = _chain_us([lambda: _lib.call("lt_attn_decode_masked", qkv.data_ptr(), kc.data_ptr(), vc.data_ptr(), ln.data_ptr(), yq.data_ptr(), hd, H,
                                          s["nkv"], float(hd ** -0.5), T + 8, st())] * 8)
        add(f"q8 attention token, {T} positions", us, T * 2 * kvw * 4, 0)
    if want("pakalix"):
        pakalix_kernels(s, T, add, st)
    # ---- row operators
    if want("norm"):
        n = _copies(T * E * 4)
        xs, w = [torch.randn(T, E, **dev) for _ in range(n)], dense_ops.Norm(torch.ones(E), E, E, 1e-6)
        h = torch.empty(T, E, dtype=torch.bfloat16, **dev)
        us = _chain_us([lambda x=x_: w.rows(x.data_ptr(), E, h.data_ptr(), E, 0, T, E) for x_ in xs])
        add(f"norm rows {T}x{E}", us, T * E * 6, 0, "q8 rmsnorm")
        wn, hf = torch.ones(E, **dev), torch.empty(T, E, **dev)
        us = _chain_us([lambda x=x_: _lib.call("lt_rmsnorm", x.data_ptr(), wn.data_ptr(), hf.data_ptr(), T, E, 1e-6, st()) for x_ in xs])
        add(f"q8 rmsnorm {T}x{E}", us, T * E * 8, 0)
    torch.cuda.synchronize()
    return out


def pakalix_kernels(s, T, add, st):
    """The kernels of the Pakalix layers; `like` names the kernel of the other mixer model to compare with."""
    E, F, H, hd, G = s["E"], s["F"], s["H"], s["hd"], s["nkv"]
    SH, P, N, SG, taps = ssd_sizes(s)
    dev = dict(device="cuda")
    bf = lambda *sh: torch.randn(*sh, device="cuda").bfloat16()
    inner, ch = SH * P, SH * P + 2 * SG * N
    f32e = torch.zeros(T, max(SH, H), **dev)
    # ---- linears: (name, rows, K, kind); gate and up rows follow those of the input projection
    ins = (("in, state space", inner + ch, SH, inner), ("in, attention", (H + 2 * G) * hd, H, H * hd))
    for name, M, tail, nin in ins:
        W = [bf(M + tail + 2 * F, E) for _ in range(_copies((M + tail + 2 * F) * E * 2))]
        X = [bf(T, E) for _ in range(3)]
        Y, Z = torch.zeros(T, M, dtype=torch.bfloat16, **dev), torch.zeros(T, nin + F, dtype=torch.bfloat16, **dev)
        e = dense_ops.with_tail(dense_ops.epilogue(segs=[(M, None, 1.0), (M + tail, "sigmoid", 1.0)], tail_from=M), f32e.data_ptr(), tail)
        n = max(len(W), 3)
        us = _chain_us([lambda i=i: _lib.call("lt_dn_linear", W[i % len(W)].data_ptr(), E, X[i % 3].data_ptr(), E, Y.data_ptr(), M, 0, M + tail, E, T,
                                              ctypes.byref(e), 0, st()) for i in range(n)])
        add(f"linear {name} {M + tail}x{E}, {T} rows", us, (M + tail) * E * 2 + T * E * 2 + T * M * 2, 2.0 * (M + tail) * E * T, "linear qkvg")
        if name == "in, state space":
            g = dense_ops.epilogue(_lib.DN_GLU, glu=(_lib.DN_GLU_CLAMPED, 1.702, 7.0))
            us = _chain_us([lambda i=i: _lib.call("lt_dn_linear", W[i % len(W)].data_ptr() + (M + tail) * E * 2, E, X[i % 3].data_ptr(), E,
                                                  Z.data_ptr() + nin * 2, nin + F, 0, F, E, T, ctypes.byref(g), 0, st()) for i in range(n)])
            add(f"linear gate|up clamped {2 * F}x{E}, {T} rows", us, 2 * F * E * 2 + T * E * 2 + T * F * 2, 4.0 * F * E * T, "linear gate|up")
        x, y, z = torch.randn(E, **dev), torch.zeros(M, dtype=torch.bfloat16, **dev), torch.zeros(F, dtype=torch.bfloat16, **dev)
        pro = dense_ops.Norm(torch.ones(E), E, E, 1e-6).prologue(x.data_ptr())
        c = _lib.DnEpilogue.from_buffer_copy(e)
        c.kind, c.glu_from, c.y2, c.glu_act, c.glu_alpha, c.glu_limit = _lib.DN_STORE_GLU, M + tail, z.data_ptr(), 1, 1.702, 7.0
        us = _chain_us([lambda i=i: _lib.call("lt_dn_gemv", W[i].data_ptr(), E, y.data_ptr(), 0, M + tail + F, E, ctypes.byref(pro), ctypes.byref(c), st())
                        for i in range(len(W))])
        add(f"gemv {name} and gate|up {M + tail + 2 * F}x{E}", us, (M + tail + 2 * F) * E * 2, 0, "gemv gate|up")
        del W
        K = nin + F
        W = [bf(E, K) for _ in range(_copies(E * K * 2))]
        X = [bf(T, K) for _ in range(3)]
        R, ls = torch.zeros(T, E, **dev), torch.full((E,), 0.25, **dev)
        e = dense_ops.epilogue(_lib.DN_RESID, ls=ls)
        n = max(len(W), 3)
        us = _chain_us([lambda i=i: _lib.call("lt_dn_linear", W[i % len(W)].data_ptr(), K, X[i % 3].data_ptr(), K, R.data_ptr(), E, 0, E, K, T,
                                              ctypes.byref(e), 0, st()) for i in range(n)])
        add(f"linear o and down, {name[4:]} {E}x{K}, {T} rows", us, E * K * 2 + T * K * 2 + T * E * 8, 2.0 * E * K * T, "linear down")
        o, f = torch.randn(nin, **dev), bf(K)
        if name == "in, state space":
            pro = dense_ops.Norm(torch.ones(nin), nin, nin, 1e-6, gate_first=True).prologue(o.data_ptr(), f.data_ptr())
            pro.n1, pro.x2 = nin, f.data_ptr()
        else:
            pro = dense_ops.typed_input(f.data_ptr())
        us = _chain_us([lambda i=i: _lib.call("lt_dn_gemv", W[i].data_ptr(), K, R.data_ptr(), 0, E, K, ctypes.byref(pro), ctypes.byref(e), st())
                        for i in range(len(W))])
        add(f"gemv o and down, {name[4:]} {E}x{K}", us, E * K * 2, 0, "gemv down")
        del W, X
    # ---- state space
    ld = inner + ch
    ys = [(torch.randn(T, ld, device="cuda") * 0.5).bfloat16() for _ in range(_copies(T * ld * 2))]
    conv, cb, one, A = torch.randn(taps, ch, **dev), torch.zeros(ch, **dev), torch.ones(SH, **dev), -torch.ones(SH, **dev)
    desc = _lib.DnSsd(SH, SG, N, P, taps, conv.data_ptr(), cb.data_ptr(), one.data_ptr(), A.data_ptr(), one.data_ptr())
    ring, u = torch.zeros(taps, ch, dtype=torch.bfloat16, **dev), torch.zeros(T, ch, dtype=torch.bfloat16, **dev)
    dt, hla, hdt = torch.randn(T, SH, **dev), torch.zeros(T, SH, **dev), torch.zeros(T, SH, **dev)
    us = _chain_us([lambda y=y_: _lib.call("lt_dn_ssd_rows", y.data_ptr() + inner * 2, ld, dt.data_ptr(), SH, ring.data_ptr(), u.data_ptr(), ch,
                                           hla.data_ptr(), hdt.data_ptr(), 0, T, 0, ctypes.byref(desc), st()) for y_ in ys])
    add(f"state-space convolution (2 launches), {ch} channels, {T} rows", us, T * ch * 4 + T * SH * 12, 0, "latent rows")
    us_ = [(torch.randn(T, ch, device="cuda") * 0.5).bfloat16() for _ in range(_copies(T * ch * 2))]
    S, o = torch.zeros(SH, P, N, **dev), torch.empty(T, inner, **dev)
    hdt.fill_(0.05); hla.fill_(-0.05)
    ws = torch.empty(_lib.dense().lt_dn_recurrence_chunked_ws(T, SH, N, P), **dev)
    dec = _lib.DnDecay()
    dec.hla, dec.hdt, dec.D, dec.ldh, dec.per = hla.data_ptr(), hdt.data_ptr(), one.data_ptr(), SH, SH // SG
    us = _chain_us([lambda x=x_: _lib.call("lt_dn_recurrence_chunked", x.data_ptr() + (inner + SG * N) * 2, x.data_ptr() + inner * 2, x.data_ptr(), ch,
                                           S.data_ptr(), o.data_ptr(), inner, T, SH, N, P, ctypes.byref(dec), ws.data_ptr(), st()) for x_ in us_])
    add(f"recurrence state space, {SH} heads of {N}x{P}, {T} rows", us, T * (ch * 2 + inner * 4), 2.0 * T * SH * (2 * N * P + 64 * P) + 2.0 * T * SG * 64 * N,
        "recurrence lightning")
    Ss = [torch.zeros(SH, P, N, **dev) for _ in range(_copies(SH * P * N * 4))]
    ln, tk = torch.full((1,), 100, dtype=torch.int32, **dev), torch.zeros(1, dtype=torch.int32, **dev)
    us = _chain_us([lambda S=S_: _lib.call("lt_dn_ssd_step", ys[0].data_ptr() + inner * 2, dt.data_ptr(), ring.data_ptr(), S.data_ptr(), o.data_ptr(), 0,
                                           ln.data_ptr(), tk.data_ptr(), ctypes.byref(desc), st()) for S_ in Ss])
    add("state-space step, one token", us, 2 * SH * N * P * 4 + ch * taps * 6, 0, "recurrence lightning, one token")
    os_ = [torch.randn(T, inner, **dev) for _ in range(_copies(T * inner * 4))]
    nm, X = dense_ops.Norm(torch.ones(inner), inner, inner, 1e-6, gate_first=True), torch.zeros(T, inner + F, dtype=torch.bfloat16, **dev)
    us = _chain_us([lambda i=i: nm.rows(os_[i].data_ptr(), inner, X.data_ptr(), inner + F, 0, T, inner, gate=ys[i % len(ys)].data_ptr(), ldg=ld)
                    for i in range(len(os_))])
    add(f"gated norm rows {T}x{inner}", us, T * inner * 8, 0, "norm rows")
    del ys, us_, Ss, os_
    # ---- attention
    cap, w = T + 64, (H + 2 * G) * hd
    half = hd // 2
    freq, qn, kn = torch.rand(half, 2, **dev), torch.ones(H * hd, **dev), torch.ones(G * hd, **dev)
    freq[:, 1] = 0
    a = _lib.DnGqa(H, G, hd, hd, hd, H * hd, G * hd, cap, hd ** -0.5, 30.0, 1e-6, 0.4, freq.data_ptr(), qn.data_ptr(), kn.data_ptr())
    ys = [bf(T, w) for _ in range(_copies(T * w * 2))]
    kc, vc, vf = bf(cap, G * hd), bf(cap, G * hd), bf(T, G * hd)
    gate, out = torch.rand(T, H, **dev), torch.zeros(T, H * hd, dtype=torch.bfloat16, **dev)
    us = _chain_us([lambda y=y_: _lib.call("lt_dn_gqa_rows", y.data_ptr(), w, kc.data_ptr(), vc.data_ptr(), vf.data_ptr(), 0, 0, T, 0, ctypes.byref(a), st())
                    for y_ in ys])
    add(f"grouped attention rows, {T} rows", us, T * (2 * H + 5 * G) * hd * 2, 0, "latent rows")
    for cap_on in (True, False):
        a.softcap = 30.0 if cap_on else 0.0
        us = _chain_us([lambda y=y_: _lib.call("lt_dn_gqa_attn", y.data_ptr(), w, kc.data_ptr(), vc.data_ptr(), gate.data_ptr(), H, out.data_ptr(), H * hd, 0,
                                               T, 0, ctypes.byref(a), st()) for y_ in ys[:4]])
        add(f"grouped attention, {H} heads on {G}, {T} rows" + ("" if cap_on else ", no cap"), us, T * (2 * H + 2 * G) * hd * 2,
            2.0 * (T * (T + 1) // 2) * H * 2 * hd, "latent window attention")
    a.softcap = 30.0
    kcs, vcs = [bf(cap, G * hd) for _ in range(24)], [bf(cap, G * hd) for _ in range(24)]
    tk = torch.zeros(_lib.dense().lt_dn_gqa_step_tickets(H, G), dtype=torch.int32, **dev)
    splits = max(1, min(74, 296 // (tk.numel() - 1)))
    ws = torch.empty(_lib.dense().lt_dn_gqa_step_ws(H, hd, splits), **dev)
    lens = [torch.full((1,), T, dtype=torch.int32, **dev) for _ in range(24)]

    def one_step(i):
        _lib.call("lt_dn_gqa_step", ys[0].data_ptr(), kcs[i % 24].data_ptr(), vcs[i % 24].data_ptr(), vf.data_ptr(), 0, gate.data_ptr(), out.data_ptr(), 0,
                  lens[i % 24].data_ptr(), ctypes.byref(a), splits, ws.data_ptr(), tk.data_ptr(), st())
    us = _chain_us([lambda i=i: one_step(i) for i in range(24)])
    add(f"grouped attention step, {T} positions", us, T * 2 * G * hd * 2, 0, "latent step")


def run(sizes=("0.5b", "3b", "8b"), tokens=2048, steps=64, kernels=True, models=True, only=None):
    res = []
    hbm, tf, src = peaks()
    for name in sizes:
        s = SIZES[name]
        r = {"size": name, **{k: s[k] for k in ("E", "F", "H", "hd", "layers", "window", "kv_rank")}, "prompt": tokens}
        if models:
            for label, make in (("pakalix_bf16", pakalix_model), ("mixers_bf16", mixer_model), ("llama_q8", llama_model)):
                dr.reset_engine_state(); dr.apply_production_profile()
                cfg, w = make(s)
                fused = dr._FUSED_STEP
                if s["E"] > 2048:       # a gate|up block of the llama model's fused step exceeds an SM's shared memory there
                    dr._FUSED_STEP = False
                try:
                    r[label] = run_model(cfg, w, tokens, steps)
                finally:
                    dr._FUSED_STEP = fused
                if label != "llama_q8":
                    wb = sum(L.numel() * 2 for k, L in w.items() if k != "embed")
                else:
                    wb = sum(q.N * q.K * 34 // 32 for q in w.values() if isinstance(q, Q8Weight))
                r[label]["weight_bytes"] = wb
                r[label]["decode_frac_of_weight_stream"] = wb / hbm * 1e-3 / r[label]["decode_us"]
                del w
                torch.cuda.empty_cache()
        dr.reset_engine_state()
        torch.cuda.empty_cache()
        if kernels:
            r["kernels"] = kernel_times(s, tokens, only)
        r["device_status"] = sorted(_lib.device_status())
        res.append(r)
    return {"peaks": {"hbm_gbs": hbm, "bf16_tflops": tf, "source": src}, "sizes": res}
