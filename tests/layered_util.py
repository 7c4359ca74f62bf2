"""Small random models made of mixer layers, for the tests: configurations, weights, oracle runs."""
import copy
import json
import os

import numpy as np
import torch

from llamatov_b200.safetensors_io import write_safetensors


def lightning(heads=3, dim=16, vdim=24, decay=None):
    if decay is None:
        decay = [float(1.0 - 0.5 ** (1 + 2 * i)) for i in range(heads)]
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}


def gla(heads=2, dim=24, vdim=40, tau=8.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def latent(heads=3, dim=24, rot_dim=16, vdim=40, kv_rank=32, window=19, base=10000.0, scale=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": window},
            "rot": {"base": base, "dims": rot_dim}, "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}


def layer(kind, mixer, ff=88):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers=None, loop="default", width=80, vocab=203, eps=1e-5, scale=7.5):
    if layers is None:
        layers = [layer("gla", gla()), layer("latent_attention", latent()), layer("lightning", lightning(), None),
                  layer("latent_attention", latent(heads=2, window=7))]
    c = {"architecture": "Nugusun", "embedding": {"scale": scale}, "layers": copy.deepcopy(layers), "norm": {"eps": eps},
         "vocab": vocab, "width": width}
    if loop == "default":
        c["loop"] = {"start": 1, "stop": 3, "times": 2}
    elif loop is not None:
        c["loop"] = dict(loop)
    return c


def random_tensors(cfg, seed=0, rank_a=12, gain=1.0):
    """bf16 tensors; linears of unit gain so that every branch matters to the logits."""
    g = torch.Generator().manual_seed(seed)

    def lin(o, i, s=1.0):
        return (torch.randn(o, i, generator=g) * (s * gain / i ** 0.5)).bfloat16()

    def vec(n, mean=1.0, s=0.2):
        return (mean + s * torch.randn(n, generator=g)).bfloat16()
    E = cfg["width"]
    t = {"embed": (torch.randn(cfg["vocab"], E, generator=g) / E ** 0.5).bfloat16(), "final.norm": vec(E), "head": lin(cfg["vocab"], E)}
    if cfg.get("loop"):
        t["loop.in"] = lin(E, 2 * E, 1.4)
        t["loop.step"] = vec(cfg["loop"]["times"] * E, 0.0, 0.3).reshape(-1, E)
    for i, ly in enumerate(cfg["layers"]):
        m, p = ly["mixer"], f"l{i}.mix."
        t[f"l{i}.norm1"], t[f"l{i}.ls1"] = vec(E), vec(E, 0.8)
        H = m["heads"]
        if ly["type"] == "latent_attention":
            t[p + "q"] = lin(H * (m["dim"] + m["rot_dim"]), E, 1.5)
            t[p + "dkv"] = lin(m["kv_rank"] + m["rot_dim"], E, 1.5)
            t[p + "dkv.norm"] = vec(m["kv_rank"])
            t[p + "uk"] = lin(H * m["dim"], m["kv_rank"], 1.5)
            t[p + "uv"] = lin(H * m["vdim"], m["kv_rank"])
        else:
            for n, d in (("q", m["dim"]), ("k", m["dim"]), ("v", m["vdim"]), ("g", m["vdim"])):
                t[p + n] = lin(H * d, E)
            if ly["type"] == "gla":
                t[p + "norm"] = vec(m["vdim"])
                t[p + "a1"] = lin(rank_a, E)
                t[p + "a2"] = lin(H * m["dim"], rank_a)
                t[p + "a2.b"] = vec(H * m["dim"], 1.0, 1.0)
            else:
                t[p + "norm"] = vec(H * m["vdim"])
        t[p + "o"] = lin(E, H * m["vdim"])
        if ly["mlp"] is not None:
            F, p = ly["mlp"]["ff"], f"l{i}.mlp."
            t[f"l{i}.norm2"], t[f"l{i}.ls2"] = vec(E), vec(E, 0.8)
            t[p + "gate"], t[p + "up"], t[p + "down"] = lin(F, E), lin(F, E), lin(E, F)
    return t


def as_numpy(tensors):
    return {k: v.float().numpy() for k, v in tensors.items()}


def write_model(path, cfg, tensors):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(path, "model.safetensors"), tensors)
    return str(path)


def product(cfg, tensors, dtype):
    """(cfg, w) as the loader returns them, without a file."""
    from llamatov_b200 import archs
    A = archs.by_name(cfg["architecture"])
    c = A.config_from_json(json.loads(json.dumps(cfg)), dtype)
    return c, A.weights_from_safetensors({k: v.clone() for k, v in tensors.items()}, c)


def oracle_logits(cfg, tensors, tokens):
    from oracle import layered as L
    return L.Model(cfg, as_numpy(tensors)).run(tokens)


def rel_rms(got, want):
    """Largest row error: root mean square of the difference over that of the wanted rows, means taken off."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d -= d.mean(axis=-1, keepdims=True)
    w = want - want.mean(axis=-1, keepdims=True)
    return float((np.sqrt((d * d).mean(axis=-1)) / np.sqrt((w * w).mean())).max())
