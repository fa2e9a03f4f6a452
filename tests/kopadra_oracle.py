"""Plain, slow Kopadra in float64, one function per mechanism, from the equations only: the yardstick of the Kopadra tests.

Nothing of the package is used here.  Weights are a dict of checkpoint names; a sequence is processed whole, the
recurrence one token after the other.
"""
from __future__ import annotations

import math

import torch

DOUBLE = torch.float64


# ------------------------------------------------------------------------------------------------ mechanisms
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def frequencies(rot):
    """(angle per position of every rotated pair, factor of cos and sin)."""
    dims, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return plain, 1.0

    def turns(t):                                              # the pair that makes t turns over the original context
        return dims * math.log(sc["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo, hi = max(math.floor(turns(sc["fast"])), 0), min(math.ceil(turns(sc["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * r + f * (1 - r))
    return out, 0.1 * math.log(sc["factor"]) + 1


def rotate(x, rot):
    """x [n, heads, dim]: dimension i turns with i + dims / 2 by position times frequency i; dimensions behind them stay."""
    freqs, size = frequencies(rot)
    half = rot["dims"] // 2
    y = x.clone()
    for p in range(x.shape[0]):
        for i, f in enumerate(freqs):
            c, s = math.cos(p * f) * size, math.sin(p * f) * size
            u, v = x[p, :, i], x[p, :, i + half]
            y[p, :, i], y[p, :, i + half] = u * c - v * s, v * c + u * s
    return y


def attend(q, k, v, scale, hide=()):
    """q [n, H, d], k [n, G, d], v [n, G, dv] -> [n, H * dv], causal.  ``hide``: key positions left out, to show that they
    matter."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    at = torch.arange(n)
    seen = at[None] <= at[:, None]
    for j in hide:
        seen[j + 1:, j] = False
    out = []
    for h in range(H):
        s = (q[:, h] @ k[:, h // (H // G)].T * scale).masked_fill(~seen, -math.inf)
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out.append(e / e.sum(-1, keepdim=True) @ v[:, h // (H // G)])
    return torch.cat(out, dim=-1)


def attention(h, w, p, m, eps, held, hide=()):
    """``held``: keys and values of earlier layers by number; this layer's are returned (None where it reads another's)."""
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def project(name):
        return h @ w[p + name].T + w[p + name + ".b"]
    q = rotate((unit_rms(project("q"), eps) * w[p + "q.norm"]).view(n, H, d), m["rot"])
    if m.get("kv_from") is not None:
        kv, (k, v) = None, held[m["kv_from"]]
    else:
        k = rotate((unit_rms(project("k"), eps) * w[p + "k.norm"]).view(n, G, d), m["rot"])
        kv = k, v = k, project("v").view(n, G, dv)
    o = attend(q, k, v, m["scale"], hide) * sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T, kv


def matrix_memory(q, k, v, i, f, state=None):
    """q (scaled), k [n, H, d], v [n, H, dv], log input and log forget gates [n, H] -> (o [n, H, dv], (S, n, m)).

    The state is (S [H, d, dv], n [H, d], m [H]): S and n are kept divided by exp(m)."""
    n, H, d = q.shape
    S, N, m = (torch.zeros(H, d, v.shape[-1], dtype=q.dtype), torch.zeros(H, d, dtype=q.dtype),
               torch.zeros(H, dtype=q.dtype)) if state is None else [t.clone() for t in state]
    o = torch.zeros_like(v)
    for t in range(n):
        for h in range(H):
            top = max(float(f[t, h] + m[h]), float(i[t, h]))
            keep, new = torch.exp(f[t, h] + m[h] - top), torch.exp(i[t, h] - top)
            S[h] = keep * S[h] + new * torch.outer(k[t, h], v[t, h])
            N[h] = keep * N[h] + new * k[t, h]
            m[h] = top
            o[t, h] = S[h].T @ q[t, h] / (max(abs(float(N[h] @ q[t, h])), math.exp(-top)) + 1e-6)
    return o, (S, N, m)


def memory_gates(h, w, p, cap):
    """(log input gate, log forget gate) [n, heads]."""
    def capped(name):
        return cap * torch.tanh((h @ w[p + name].T + w[p + name + ".b"]) / cap)
    return capped("i"), -torch.log1p(torch.exp(-capped("f")))


def mlstm(h, w, p, m, eps):
    n, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w[p + "q"].T).view(n, H, d) * d ** -0.5, (h @ w[p + "k"].T).view(n, H, d), (h @ w[p + "v"].T).view(n, H, dv)
    o, _ = matrix_memory(q, k, v, *memory_gates(h, w, p, m["gate_cap"]))
    return (unit_rms(o, eps).reshape(n, H * dv) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def gated(h, w, p, act):
    return (act(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def choose(scores, correction, top, count, keep):
    """Expert numbers [n, top] by score plus correction, from the best ``keep`` of ``count`` groups only."""
    out = []
    for row in scores + correction:
        size = len(row) // count
        best = sorted(range(count), key=lambda g: -float(row[g * size:(g + 1) * size].max()))[:keep]
        ok = [e for e in range(len(row)) if e // size in best]
        out.append(sorted(ok, key=lambda e: -float(row[e]))[:top])
    return torch.tensor(out)


def experts(h, w, p, mlp):
    r = mlp["router"]
    z = h @ w[p + "router"].T
    s = torch.exp(z - z.max(-1, keepdim=True).values)
    s = s / s.sum(-1, keepdim=True)
    g = r.get("groups") or dict(count=1, keep=1)
    ids = choose(s, w[p + "correction"], r["top"], g["count"], g["keep"])
    out = gated(h, w, p + "shared.", silu) if mlp.get("shared") else torch.zeros_like(h)
    for t in range(h.shape[0]):
        total = s[t, ids[t]].sum() + 1e-20
        for e in ids[t].tolist():
            y = gated(h[t], w, f"{p}e{e}.", silu) if e < r["experts"] else h[t]
            out[t] += s[t, e] / total * r["scale"] * y
    return out


# ------------------------------------------------------------------------------------------------ the model
def forward(cfg, weights, tokens, hide=(), layers=None):
    """Logits [n, vocab] of a whole sequence; ``layers`` (a list) receives the stream after every layer."""
    w = {k: v.to(DOUBLE) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    held = {}
    x = w["embed"][torch.tensor(tokens)]
    for i, spec in enumerate(cfg["layers"]):
        m, p = spec["mixer"], f"l{i}.mix."
        h = layer_norm(x, w[f"l{i}.norm1"], eps)
        if spec["type"] == "mlstm":
            y = mlstm(h, w, p, m, eps)
        else:
            y, held[i] = attention(h, w, p, m, eps, held, hide)
        x = x + y
        if spec.get("mlp"):
            h, p = layer_norm(x, w[f"l{i}.norm2"], eps), f"l{i}.mlp."
            x = x + (gated(h, w, p, gelu_tanh) if spec["mlp"]["kind"] == "dense" else experts(h, w, p, spec["mlp"]))
        if layers is not None:
            layers.append(x)
    z = layer_norm(x, w["final.norm"], eps) @ w["embed"].T
    return cfg["logit_softcap"] * torch.tanh(z / cfg["logit_softcap"])


def greedy(cfg, weights, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, weights, toks)[-1].argmax()))
    return toks[len(prompt):]
