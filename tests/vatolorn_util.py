"""Small random Vatolorn checkpoints for the tests: configuration builders and seeded weights (values representable in
bfloat16, so that both storage types and the float64 oracle read the same numbers).  The safetensors writer is the one of
tests/pikavik_util.py."""
from __future__ import annotations

import torch

from tests.pikavik_util import rel_err, write_checkpoint  # noqa: F401  (re-exported)


def dense(ff=28):
    return {"kind": "dense", "ff": ff}


def attention(heads=6, kv_heads=2, dim=10, vdim=6, conv=4, chunk=24, scale=0.4, dims=6, base=300.0, scaling="default"):
    a = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "mask": {"size": chunk}, "scale": scale}
    if dims:
        a["rot"] = {"base": base, "dims": dims}
        if scaling == "default":
            a["rot"]["scaling"] = {"factor": 3.0, "original": 80, "fast": 6.0, "slow": 0.5}
        elif scaling:
            a["rot"]["scaling"] = scaling
    return a


def delta(heads=6, kv_heads=3, dim=12, vdim=7, conv=3, decay_rank=5, gate_rank=9):
    # (the two ranks are private to the builders: a checkpoint shows them only in its tensors' shapes)
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "_decay_rank": decay_rank, "_gate_rank": gate_rank}


def parallel(left=None, right=None, mlp=None):
    return {"type": "parallel", "mixer": {"left": left or attention(), "right": right or delta()}, "mlp": mlp}


def config(layers, width=40, vocab=50, eps=1e-5, streams=2, logit_scale=0.7):
    return {"architecture": "Vatolorn", "layers": layers, "logit_scale": logit_scale, "norm": {"eps": eps}, "streams": streams,
            "vocab": vocab, "width": width}


def write(path, cfg, tensors):
    """write_checkpoint without the builders' private keys."""
    def public(x):
        if isinstance(x, dict):
            return {k: public(v) for k, v in x.items() if not k.startswith("_")}
        return [public(v) for v in x] if isinstance(x, list) else x
    return write_checkpoint(path, public(cfg), tensors)


def random_tensors(cfg: dict, seed: int = 0) -> dict[str, torch.Tensor]:
    g = torch.Generator().manual_seed(seed)
    W, S = cfg["width"], cfg["streams"]

    def lin(o, i, gain=1.0):
        return torch.randn(o, i, generator=g) * gain / i ** 0.5

    def vec(n, mean=0.0, std=0.1):
        return mean + std * torch.randn(n, generator=g)

    def uni(n, lo, hi):
        return lo + (hi - lo) * torch.rand(n, generator=g)

    t = {"embed": torch.randn(cfg["vocab"], W, generator=g), "head": lin(cfg["vocab"], W, 2.0), "final.norm": vec(W, 1.0, 0.2)}
    for i, lc in enumerate(cfg["layers"]):
        p, mx, m = f"l{i}.", f"l{i}.mix.", lc["mixer"]
        for k in ("1", "2") if lc.get("mlp") else ("1",):
            t[p + "norm" + k] = vec(W, 1.0, 0.2)
            t[f"{p}hc{k}.in"], t[f"{p}hc{k}.out"] = vec(S, 1.0 / S, 0.3), vec(S, 0.8, 0.3)
            t[f"{p}hc{k}.mix"] = 0.9 * torch.eye(S) + 0.15 * torch.randn(S, S, generator=g)   # not symmetric: [from, to]
        a, d = m["left"], m["right"]
        q, H, G, D, V = mx + "left.", a["heads"], a["kv_heads"], a["dim"], a["vdim"]
        for s, rows in (("q", H * D), ("k", G * D), ("v", G * V)):
            t[q + s], t[q + s + ".b"] = lin(rows, W), vec(rows, 0.0, 0.3)
            if a.get("conv"):
                t[q + s + ".conv"] = 0.6 * torch.randn(rows, a["conv"], generator=g)
        t[q + "q.norm"], t[q + "k.norm"] = vec(H * D, 1.0, 0.3), vec(G * D, 1.0, 0.3)
        t[q + "o"], t[q + "out"] = lin(W, H * V), vec(W, 1.0, 0.3)
        q, H, G, D, V, taps = mx + "right.", d["heads"], d["kv_heads"], d["dim"], d["vdim"], d["conv"]
        for s, rows in (("q", G * D), ("k", G * D), ("v", H * V)):
            t[q + s], t[q + s + ".conv"] = lin(rows, W, 2.0), 0.6 * torch.randn(rows, taps, generator=g)
        t[q + "b"], t[q + "A_log"], t[q + "dt_bias"] = lin(H, W, 2.0), uni(H, -2.5, 0.3), uni(H * D, -2.5, 1.0)
        t[q + "a1"], t[q + "a2"] = lin(d["_decay_rank"], W), lin(H * D, d["_decay_rank"], 2.0)
        t[q + "g1"], t[q + "g2"] = lin(d["_gate_rank"], W), lin(H * V, d["_gate_rank"], 2.0)
        t[q + "norm"], t[q + "o"], t[q + "out"] = vec(V, 1.0, 0.2), lin(W, H * V), vec(W, 1.0, 0.3)
        if lc.get("mlp"):
            ff = lc["mlp"]["ff"]
            t[p + "mlp.gate"], t[p + "mlp.up"], t[p + "mlp.down"] = lin(ff, W, 2.0), lin(ff, W, 2.0), lin(W, ff)
    return {k: v.to(torch.bfloat16).to(torch.float32) for k, v in t.items()}
