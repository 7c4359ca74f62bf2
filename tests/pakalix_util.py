"""Small random Pakalix models for the tests: configurations, weights, oracle runs."""
import copy

import torch

from tests.layered_util import as_numpy


def attention(heads=6, kv_heads=2, dim=24, vdim=40, rot=16, base=5000.0, scale=None, softcap=15.0, v_mix=True):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot},
            "scale": dim ** -0.5 if scale is None else scale, "softcap": softcap, "v_mix": v_mix}


def mamba2(heads=6, groups=2, vdim=24, state=40, conv=4, norm_groups=3):
    return {"heads": heads, "groups": groups, "vdim": vdim, "state": state, "conv": conv, "norm_groups": norm_groups}


def layer(kind, mixer, ff=88, limit=0.9):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def config(layers=None, width=80, vocab=203, eps=1e-5, residual_mult=0.6):
    if layers is None:
        layers = [layer("mamba2", mamba2()), layer("attention", attention()), layer("mamba2", mamba2(heads=4, groups=1, norm_groups=1), None),
                  layer("attention", attention(heads=4, softcap=6.0), 40, 2.5), layer("attention", attention(v_mix=False, kv_heads=3))]
    return {"architecture": "Pakalix", "layers": copy.deepcopy(layers), "norm": {"eps": eps}, "residual_mult": residual_mult,
            "vocab": vocab, "width": width}


def random_tensors(cfg, seed=0, gain=1.0):
    """bf16 tensors; gains so that every branch matters to the logits and clamps and caps bite."""
    g = torch.Generator().manual_seed(seed)

    def lin(o, i, s=1.0):
        return (torch.randn(o, i, generator=g) * (s * gain / i ** 0.5)).bfloat16()

    def vec(n, mean=1.0, s=0.2):
        return (mean + s * torch.randn(n, generator=g)).bfloat16()
    E = cfg["width"]
    t = {"embed": torch.randn(cfg["vocab"], E, generator=g).bfloat16(), "embed.norm": vec(E, 0.0), "final.norm": vec(E, 0.0),
         "head": lin(cfg["vocab"], E)}
    for i, ly in enumerate(cfg["layers"]):
        m, p, H = ly["mixer"], f"l{i}.mix.", ly["mixer"]["heads"]
        t[f"l{i}.norm1"] = vec(E, 0.0)
        if ly["type"] == "mamba2":
            inner, gn = H * m["vdim"], m["groups"] * m["state"]
            t[p + "in"] = torch.cat([lin(2 * inner, E), lin(2 * gn, E, 1.5), lin(H, E)])
            t[p + "conv"], t[p + "conv.b"] = lin(inner + 2 * gn, m["conv"], 1.5), vec(inner + 2 * gn, 0.0, 0.3)
            t[p + "dt_bias"], t[p + "A_log"], t[p + "D"] = vec(H, -1.0, 1.0), vec(H, -1.0, 1.5), vec(H, 0.7, 0.5)
            t[p + "norm"] = vec(inner)
            t[p + "o"] = lin(E, inner)
        else:
            G = m["kv_heads"]
            t[p + "q"], t[p + "k"], t[p + "v"] = lin(H * m["dim"], E), lin(G * m["dim"], E), lin(G * m["vdim"], E)
            t[p + "q.norm"], t[p + "k.norm"] = vec(H * m["dim"], 1.5, 0.4), vec(G * m["dim"], 1.5, 0.4)
            t[p + "g"] = lin(H, E, 1.5)
            t[p + "o"] = lin(E, H * m["vdim"], 1.5)
            if m.get("v_mix"):
                t[p + "vmix"] = torch.tensor(0.2 + 0.1 * i).bfloat16()
        if ly["mlp"] is not None:
            F, p = ly["mlp"]["ff"], f"l{i}.mlp."
            t[p + "gate"], t[p + "up"], t[p + "down"] = lin(F, E), lin(F, E), lin(E, F)
    return t


def oracle_logits(cfg, tensors, tokens):
    from oracle import pakalix as O
    return O.Model(cfg, as_numpy(tensors)).run(tokens)
