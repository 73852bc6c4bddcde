"""Plain, slow restatement of the Vatolorn design in float64 on the CPU — the oracle of tests/test_vatolorn_*.py.
One function per mechanism, written from the design's equations; it shares no code with ssd_b200 (it reads the raw
checkpoint tensors by name, not the packed layout, and keeps its own state dictionaries).

Notation: X [streams, n, width] residual streams, t a position, H heads, G key/value (or query/key) heads.  A mixer takes
the rows of ONE sequence (`h` [n, width], first position `p0`) and a state dict that carries what the sequence left behind
(cached keys and values, the last taps - 1 inputs of every short convolution, the delta rule's matrices), so a prompt can be
fed whole, in portions or token by token."""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


# ------------------------------------------------------------------------------------------------ residual streams
def read_streams(X, w_in):
    """What a sublayer reads: the streams' weighted sum."""
    return sum(w_in[s] * X[s] for s in range(X.shape[0]))


def write_streams(X, y, mix, w_out):
    """Every new stream is a mixture of the old ones (mix[from, to]) plus its share of the sublayer's result."""
    S = X.shape[0]
    return torch.stack([sum(mix[s, t] * X[s] for s in range(S)) + w_out[t] * y for t in range(S)])


# ------------------------------------------------------------------------------------------------ short convolution
def short_conv(u, w, state, key):
    """Causal convolution over time, per channel.  u [n, C]; w [C, taps], the last column multiplies the current row; zeros
    before the sequence's start.  state[key] keeps the last taps - 1 rows of u."""
    C, taps = w.shape
    hist = state.get(key, torch.zeros(taps - 1, C, dtype=F64))
    full = torch.cat([hist, u], 0)
    state[key] = full[full.shape[0] - (taps - 1):].clone()
    return sum(w[:, j] * full[j:j + u.shape[0]] for j in range(taps))


# ------------------------------------------------------------------------------------------------ attention
def rotary_table(rot):
    """(frequencies [dims / 2], factor on cos and sin), with the YaRN correction if rot has 'scaling'."""
    dims, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def dim_of(turns):
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(dim_of(sc["fast"])), 0)
    hi = min(math.ceil(dim_of(sc["slow"])), dims - 1)
    ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(dims // 2)]
    return [fi / sc["factor"] * r + fi * (1.0 - r) for fi, r in zip(f, ramp)], 0.1 * math.log(sc["factor"]) + 1.0


def rotate_interleaved(v, p0, rot):
    """v [n, heads, dim]: entries 2i and 2i + 1 of the first rot.dims entries turn together by position * f_i."""
    freqs, mult = rotary_table(rot)
    pos = torch.arange(p0, p0 + v.shape[0], dtype=F64)
    out = v.clone()
    for i, f in enumerate(freqs):
        c, s = (torch.cos(pos * f) * mult)[:, None], (torch.sin(pos * f) * mult)[:, None]
        a, b = v[..., 2 * i], v[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = a * c - b * s, b * c + a * s
    return out


def first_visible(pos, chunk):
    """The first key a query at `pos` sees: chunks of `chunk` positions are counted from the sequence's start (0: no chunks)."""
    return pos // chunk * chunk if chunk else 0


def chunked_softmax_attention(q, K, V, p0, scale, chunk):
    """One head: q [n, D] at positions p0 .., K [ctx, D], V [ctx, Dv] from position 0."""
    out = []
    for t in range(q.shape[0]):
        pos = p0 + t
        lo = first_visible(pos, chunk)
        s = (K[lo:pos + 1] @ q[t]) * scale
        out.append(torch.softmax(s, 0) @ V[lo:pos + 1])
    return torch.stack(out)


def attention_mixer(h, W, p, mx, eps, state, p0):
    n, H, G, D, Dv = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    z = {}
    for c in "qkv":
        u = h @ W[f"{p}.{c}"].T
        if f"{p}.{c}.b" in W:
            u = u + W[f"{p}.{c}.b"]
        if f"{p}.{c}.conv" in W:
            u = short_conv(u, W[f"{p}.{c}.conv"], state, "conv_" + c)
        z[c] = u
    q = rms_norm(z["q"], W[p + ".q.norm"], eps).view(n, H, D)     # over the whole projection, before the heads are split
    k = rms_norm(z["k"], W[p + ".k.norm"], eps).view(n, G, D)
    v = z["v"].view(n, G, Dv)
    rot = mx.get("rot")
    if rot and rot.get("dims", 0) >= 2:
        q, k = rotate_interleaved(q, p0, rot), rotate_interleaved(k, p0, rot)
    state["K"] = torch.cat([state["K"], k]) if "K" in state else k
    state["V"] = torch.cat([state["V"], v]) if "V" in state else v
    chunk = (mx.get("mask") or {}).get("size", 0)
    o = [chunked_softmax_attention(q[:, hd], state["K"][:, hd // (H // G)], state["V"][:, hd // (H // G)], p0, mx["scale"], chunk)
         for hd in range(H)]
    return torch.cat(o, -1) @ W[p + ".o"].T


# ------------------------------------------------------------------------------------------------ gated delta rule
def delta_step(S, q, k, v, beta, g):
    """One token of all heads.  S [H, D, V] (rows: key channels), q, k, g [H, D], v [H, V], beta [H] -> (new S, read-out)."""
    S = g[:, :, None] * S
    u = beta[:, None] * (v - torch.einsum("hdv,hd->hv", S, k))
    S = S + k[:, :, None] * u[:, None, :]
    return S, torch.einsum("hdv,hd->hv", S, q)


def channel_decay(h, W, p, H, D):
    """g [n, H, D] = exp(-exp(A_log) * softplus(low-rank projection + bias)): one decay per head and key channel."""
    z = (h @ W[p + ".a1"].T) @ W[p + ".a2"].T + W[p + ".dt_bias"]
    return torch.exp(-torch.exp(W[p + ".A_log"])[None, :, None] * softplus(z).view(-1, H, D))


def gated_delta_mixer(h, W, p, mx, eps, state):
    n, H, G, D, Dv = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    z = {c: silu(short_conv(h @ W[f"{p}.{c}"].T, W[f"{p}.{c}.conv"], state, "conv_" + c)) for c in "qkv"}

    def unit(x):
        return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)

    q = unit(z["q"].view(n, G, D)) * D ** -0.5
    k = unit(z["k"].view(n, G, D))
    q, k = q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1)   # head h reads query/key head h / (H / G)
    v = z["v"].view(n, H, Dv)
    beta = torch.sigmoid(h @ W[p + ".b"].T)
    g = channel_decay(h, W, p, H, D)
    S = state.get("S", torch.zeros(H, D, Dv, dtype=F64))
    o = []
    for t in range(n):
        S, ot = delta_step(S, q[t], k[t], v[t], beta[t], g[t])
        o.append(ot)
    state["S"] = S
    gate = torch.sigmoid((h @ W[p + ".g1"].T) @ W[p + ".g2"].T).view(n, H, Dv)
    return (rms_norm(torch.stack(o), W[p + ".norm"], eps) * gate).reshape(n, H * Dv) @ W[p + ".o"].T


def parallel_mixer(h, W, p, mx, eps, state, p0):
    left = attention_mixer(h, W, p + ".left", mx["left"], eps, state.setdefault("left", {}), p0)
    right = gated_delta_mixer(h, W, p + ".right", mx["right"], eps, state.setdefault("right", {}))
    return 0.5 * (rms_norm(left, W[p + ".left.out"], eps) + rms_norm(right, W[p + ".right.out"], eps))


# ------------------------------------------------------------------------------------------------ feed-forward, model
def dense_ff(h, W, p):
    return (silu(h @ W[p + ".gate"].T) * (h @ W[p + ".up"].T)) @ W[p + ".down"].T


def forward(cfg, W, tokens, state, p0):
    """Runs `tokens` (positions p0 ..) of one sequence.  W: name -> float64 tensor.  state: dict carried between calls
    (empty for a new sequence).  Returns (logits [n, vocab], sum of the streams after every layer [layers, n, width])."""
    eps = cfg["norm"]["eps"]
    e = W["embed"][torch.tensor(tokens)]
    X = torch.stack([e] * cfg["streams"])
    taps = []
    for i, lc in enumerate(cfg["layers"]):
        p = f"l{i}"
        if lc["type"] != "parallel":
            raise ValueError(lc["type"])
        h = rms_norm(read_streams(X, W[p + ".hc1.in"]), W[p + ".norm1"], eps)
        y = parallel_mixer(h, W, p + ".mix", lc["mixer"], eps, state.setdefault(i, {}), p0)
        X = write_streams(X, y, W[p + ".hc1.mix"], W[p + ".hc1.out"])
        if lc.get("mlp"):
            if lc["mlp"]["kind"] != "dense":
                raise ValueError(lc["mlp"]["kind"])
            y = dense_ff(rms_norm(read_streams(X, W[p + ".hc2.in"]), W[p + ".norm2"], eps), W, p + ".mlp")
            X = write_streams(X, y, W[p + ".hc2.mix"], W[p + ".hc2.out"])
        taps.append(X.sum(0))
    logits = rms_norm(X.sum(0), W["final.norm"], eps) @ W["head"].T * cfg["logit_scale"]
    return logits, torch.stack(taps)


class PlainModel:
    """The oracle over raw tensors: whole prompts, portions (through a carried state) and greedy continuation."""

    def __init__(self, cfg, tensors):
        self.cfg, self.W = cfg, {k: v.to(F64) for k, v in tensors.items()}

    def run(self, tokens, layers_out=None, state=None, p0=0):
        logits, taps = forward(self.cfg, self.W, list(tokens), {} if state is None else state, p0)
        if layers_out is not None:
            layers_out.extend(taps)
        return logits

    def greedy(self, prompt, n):
        state, out, pos = {}, [], len(prompt)
        logits = self.run(prompt, state=state)
        for _ in range(n):
            out.append(int(torch.argmax(logits[-1])))
            logits = self.run([out[-1]], state=state, p0=pos)
            pos += 1
        return out
