"""Small random Vegilix checkpoints for the tests: configuration builders and seeded weights (values representable in
bfloat16, so that both storage types and the float64 oracle read the same numbers).  The safetensors writer is the one of
tests/pikavik_util.py."""
from __future__ import annotations

import torch

from tests.pikavik_util import rel_err, write_checkpoint  # noqa: F401  (re-exported)

SCALING = {"factor": 3.0, "low": 0.8, "high": 2.5, "original": 60}   # wavelengths on both sides and in between for the bases used here


def moe(experts=6, top=2, ff=20, shared_ff=12):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top},
            "shared": {"ff": shared_ff} if shared_ff else None}


def attention(heads=6, kv_heads=2, dim=10, vdim=14, window=24, keep=3, scale=0.4, dims=6, base=300.0, scaling="default", diff=0.4, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    if dims:
        m["rot"] = {"base": base, "dims": dims}
        if scaling:
            m["rot"]["scaling"] = SCALING if scaling == "default" else scaling
    return {"type": "attention", "mixer": m, "mlp": mlp}


def retention(heads=3, dim=12, vdim=7, dims=8, base=500.0, decay=None, mlp=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or [1.0 - 2.0 ** -(2 + 2 * (i % 4)) for i in range(heads)]}
    if dims:
        m["rot"] = {"base": base, "dims": dims}
    return {"type": "retention", "mixer": m, "mlp": mlp}


def config(layers, width=40, vocab=50, eps=1e-5, loop=None, mult=0.6):
    cfg = {"architecture": "Vegilix", "layers": layers, "norm": {"eps": eps}, "residual_mult": mult, "vocab": vocab, "width": width}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def random_tensors(cfg: dict, seed: int = 0) -> dict[str, torch.Tensor]:
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def lin(o, i, gain=1.0):
        return torch.randn(o, i, generator=g) * gain / i ** 0.5

    def vec(n, mean=0.0, std=0.2):
        return mean + std * torch.randn(n, generator=g)

    t = {"embed": torch.randn(cfg["vocab"], W, generator=g), "head": lin(cfg["vocab"], W), "final.norm": vec(W)}
    for i, lc in enumerate(cfg["layers"]):
        p, mx, m = f"l{i}.", f"l{i}.mix.", lc["mixer"]
        H, D, V = m["heads"], m["dim"], m["vdim"]
        t[p + "norm1"], t[p + "norm1b"] = vec(W), vec(W)
        if lc["type"] == "attention":
            G = m["kv_heads"]
            t[mx + "q"], t[mx + "k"], t[mx + "v"] = lin(2 * H * D, W), lin(2 * G * D, W), lin(G * V, W)
            t[mx + "q.norm"], t[mx + "k.norm"] = vec(D, 1.0, 0.3), vec(D, 1.0, 0.3)
            for s in ("lq1", "lk1", "lq2", "lk2"):
                t[mx + s] = vec(D, 0.1, 0.3)
        else:
            t[mx + "q"], t[mx + "k"], t[mx + "v"], t[mx + "g"] = lin(H * D, W), lin(H * D, W), lin(H * V, W), lin(H * V, W, 2.0)
        t[mx + "o"] = lin(W, H * V)
        mlp = lc.get("mlp")
        if not mlp:
            continue
        q, ff = p + "mlp.", mlp["expert"]["ff"]
        t[p + "norm2"], t[p + "norm2b"] = vec(W), vec(W)
        t[q + "router"] = lin(mlp["router"]["experts"], W, 3.0)
        for e in range(mlp["router"]["experts"]):
            t[f"{q}e{e}.gate"], t[f"{q}e{e}.up"], t[f"{q}e{e}.down"] = lin(ff, W, 1.5), lin(ff, W, 1.5), lin(W, ff)
        if mlp.get("shared"):
            sff = mlp["shared"]["ff"]
            t[q + "shared.gate"], t[q + "shared.up"], t[q + "shared.down"] = lin(sff, W, 1.5), lin(sff, W, 1.5), lin(W, sff)
    return {k: v.to(torch.bfloat16).to(torch.float32) for k, v in t.items()}


def one_hot_tensors(cfg: dict, seed: int = 0) -> dict[str, torch.Tensor]:
    """As random_tensors, but token t's embedding is the unit vector t (times the root of the width, so the first norm leaves it as it
    is) and the first norm's weight is zero: column t of a first-layer projection, times sqrt(width), is what token t projects to."""
    assert cfg["vocab"] <= cfg["width"]
    t = random_tensors(cfg, seed)
    W = cfg["width"]
    t["embed"] = torch.eye(cfg["vocab"], W)
    t["l0.norm1"] = torch.zeros(W)
    return t


def set_token(tensors: dict, name: str, token: int, rows: torch.Tensor) -> None:
    """What token `token` projects to through the first layer's matrix `name` (one_hot_tensors)."""
    w = tensors[name]
    w[:, token] = (rows / w.shape[1] ** 0.5).to(torch.bfloat16).to(torch.float32)
