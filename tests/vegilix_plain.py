"""Plain, slow restatement of the Vegilix design in float64 on the CPU — the oracle of tests/test_vegilix_*.py.
One function per mechanism, written from the design's equations; it shares no code with ssd_b200 (it reads the raw
checkpoint tensors by name, not the packed layout, and keeps its own state dictionaries).

A mixer takes the rows of ONE sequence (`h` [n, width], first position `p0`) and a state dict that carries what the sequence
left behind (cached keys and values, the retention's matrices), so a prompt can be fed whole, in portions or token by token.
Every RUN of a layer has a state of its own: a layer that the loop repeats appears once per pass."""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm_offset(x, w, eps):
    """The weight is stored around zero."""
    return unit_rms(x, eps) * (1.0 + w)


def silu(z):
    return z * torch.sigmoid(z)


# ------------------------------------------------------------------------------------------------ program of layers
def layer_runs(cfg):
    """Indices of the layers in the order they run: start .. stop - 1 is repeated `times` times."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    body = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + body * loop["times"] + list(range(loop["stop"], n))


# ------------------------------------------------------------------------------------------------ rotary positions
def rotary_frequencies(rot):
    """base^(-2i / dims); with 'scaling', a frequency is slowed by `factor` when its wavelength exceeds original / low, kept when it
    is below original / high, and blended in between."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        sc = rot.get("scaling")
        if sc:
            wave = 2.0 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif not wave < sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate_half(v, p0, rot):
    """v [n, heads, dim]: entry i turns with entry i + dims / 2 by position * f_i; entries from dims on pass."""
    out = v.clone()
    if not rot or rot.get("dims", 0) < 2:
        return out
    half = rot["dims"] // 2
    pos = torch.arange(p0, p0 + v.shape[0], dtype=F64)
    for i, f in enumerate(rotary_frequencies(rot)):
        c, s = torch.cos(pos * f)[:, None], torch.sin(pos * f)[:, None]
        a, b = v[..., i], v[..., i + half]
        out[..., i], out[..., i + half] = a * c - b * s, b * c + a * s
    return out


# ------------------------------------------------------------------------------------------------ differential attention
def visible(i, j, mask):
    """Query positions i, key positions j (tensors that broadcast): a causal window of `size` positions beside the sequence's first
    `keep_first` keys."""
    if not mask or not mask.get("size"):
        return j <= i
    return (j <= i) & ((i - j < mask["size"]) | (j < mask.get("keep_first", 0)))


def masked_softmax_attention(q, k, v, p0, scale, mask):
    """One map of one head: q [n, D] at positions p0 .., k [ctx, D], v [ctx, Dv] from position 0."""
    seen = visible(torch.arange(p0, p0 + q.shape[0])[:, None], torch.arange(k.shape[0])[None, :], mask)
    s = torch.where(seen, (q @ k.T) * scale, torch.tensor(-math.inf, dtype=F64))
    return torch.softmax(s, -1) @ v


def difference_weight(lq1, lk1, lq2, lk2, diff):
    return torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff


def difference_heads(a1, a2, lam, diff, eps):
    """Two maps' outputs [.., Dv] -> one head."""
    return unit_rms(a1 - lam * a2, eps) * (1.0 - diff)


def attention_mixer(h, W, p, m, eps, state, p0):
    n, H, G, D, V = h.shape[0], m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m.get("vdim", m["dim"])
    q = unit_rms((h @ W[p + ".q"].T).view(n, H * 2, D), eps) * W[p + ".q.norm"]
    k = unit_rms((h @ W[p + ".k"].T).view(n, G * 2, D), eps) * W[p + ".k.norm"]
    q = rotate_half(q, p0, m.get("rot")).view(n, H, 2, D)
    k = rotate_half(k, p0, m.get("rot")).view(n, G, 2, D)
    v = (h @ W[p + ".v"].T).view(n, G, V)
    state["k"] = torch.cat([state["k"], k]) if "k" in state else k
    state["v"] = torch.cat([state["v"], v]) if "v" in state else v
    lam = difference_weight(W[p + ".lq1"], W[p + ".lk1"], W[p + ".lq2"], W[p + ".lk2"], m["diff"])
    heads = []
    for hd in range(H):
        g = hd // (H // G)
        a = [masked_softmax_attention(q[:, hd, i], state["k"][:, g, i], state["v"][:, g], p0, m["scale"], m.get("mask")) for i in (0, 1)]
        heads.append(difference_heads(a[0], a[1], lam, m["diff"], eps))
    return torch.cat(heads, -1) @ W[p + ".o"].T


# ------------------------------------------------------------------------------------------------ retention
def retention_step(S, q, k, v, decay):
    """One head, one token: S [D, Dv] -> (new S, o [Dv])."""
    S = decay * S + torch.outer(k, v)
    return S, S.T @ q


def retention_mixer(h, W, p, m, eps, state, p0):
    n, H, D, V = h.shape[0], m["heads"], m["dim"], m.get("vdim", m["dim"])
    q = rotate_half((h @ W[p + ".q"].T).view(n, H, D), p0, m.get("rot"))
    k = rotate_half((h @ W[p + ".k"].T).view(n, H, D), p0, m.get("rot")) * D ** -0.5
    v = (h @ W[p + ".v"].T).view(n, H, V)
    S = state.get("S", torch.zeros(H, D, V, dtype=F64)).clone()
    o = torch.zeros(n, H, V, dtype=F64)
    for t in range(n):
        for hd in range(H):
            S[hd], o[t, hd] = retention_step(S[hd], q[t, hd], k[t, hd], v[t, hd], m["decay"][hd])
    state["S"] = S
    y = unit_rms(o, eps).reshape(n, H * V) * silu(h @ W[p + ".g"].T)
    return y @ W[p + ".o"].T


# ------------------------------------------------------------------------------------------------ mixture of experts
def silu_expert(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def route_top(z, top):
    """The `top` largest logits (ties to the lower index) and the softmax over just those."""
    order = sorted(range(z.shape[0]), key=lambda e: (-float(z[e]), e))[:top]
    return order, torch.softmax(z[order], -1)


def moe_ff(h, W, p, m):
    z = h @ W[p + ".router"].T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen, wts = route_top(z[t], m["router"]["top"])
        for e, wt in zip(chosen, wts):
            q = f"{p}.e{e}."
            out[t] += wt * silu_expert(h[t:t + 1], W[q + "gate"], W[q + "up"], W[q + "down"])[0]
    if m.get("shared"):
        out = out + silu_expert(h, W[p + ".shared.gate"], W[p + ".shared.up"], W[p + ".shared.down"])
    return out


# ------------------------------------------------------------------------------------------------ model
class PlainModel:
    def __init__(self, cfg: dict, tensors: dict):
        self.cfg = cfg
        self.W = {k: v.to(F64) for k, v in tensors.items()}
        self.runs = layer_runs(cfg)

    def new_state(self):
        return [dict() for _ in self.runs]

    def run(self, tokens, state=None, p0=0, layers_out=None):
        """Logits [n, vocab] of `tokens` continuing a sequence at position p0 with `state` (None: a new sequence)."""
        cfg, W = self.cfg, self.W
        eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
        state = state if state is not None else self.new_state()
        x = W["embed"][torch.tensor(list(tokens))]
        for r, i in enumerate(self.runs):
            p, lc = f"l{i}", cfg["layers"][i]
            mixer = {"attention": attention_mixer, "retention": retention_mixer}[lc["type"]]
            y = mixer(rms_norm_offset(x, W[p + ".norm1"], eps), W, p + ".mix", lc["mixer"], eps, state[r], p0)
            x = x + m * rms_norm_offset(y, W[p + ".norm1b"], eps)
            if lc.get("mlp"):
                y = moe_ff(rms_norm_offset(x, W[p + ".norm2"], eps), W, p + ".mlp", lc["mlp"])
                x = x + m * rms_norm_offset(y, W[p + ".norm2b"], eps)
            if layers_out is not None:
                layers_out.append(x.clone())
        return rms_norm_offset(x, W["final.norm"], eps) @ W["head"].T

    def greedy(self, prompt, n_new):
        state = self.new_state()
        logits = self.run(prompt, state, 0)
        out, pos = [], len(prompt)
        for _ in range(n_new):
            tok = int(torch.argmax(logits[-1]))
            out.append(tok)
            logits = self.run([tok], state, pos)
            pos += 1
        return out
