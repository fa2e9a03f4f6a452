"""Plain, slow Gizilorn in float64, one function per mechanism, from the equations only: the yardstick of the Gizilorn tests.

Nothing of the package is used here.  Weights are a dict of checkpoint names; a sequence is processed whole.
"""
from __future__ import annotations

import copy
import math

import torch

DOUBLE = torch.float64


# ------------------------------------------------------------------------------------------------ mechanisms
def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def xielu(z, p, q):
    a, b = math.log1p(math.exp(p)), 0.5 + math.log1p(math.exp(q))
    return torch.where(z > 0, a * z * z, b * (torch.expm1(torch.clamp(z, max=0.0)) - torch.clamp(z, max=0.0))) + z / 2


def turn(x, base, dims, halves, back=False, first=0):
    """x [n, heads, width]; the pairs of the first ``dims`` dimensions turn by position * base^(-2 i / dims) (``back``: the other way
    round); pair i is (i, i + dims / 2) with ``halves``, else (2 i, 2 i + 1).  ``first``: position of the first row."""
    y = x.clone()
    for r in range(x.shape[0]):
        for i in range(dims // 2):
            a = (first + r) * base ** (-2.0 * i / dims)
            c, s = math.cos(a), -math.sin(a) if back else math.sin(a)
            m, n = (i, i + dims // 2) if halves else (2 * i, 2 * i + 1)
            u, v = x[r, :, m], x[r, :, n]
            y[r, :, m], y[r, :, n] = u * c - v * s, v * c + u * s
    return y


def seen(n, window, hide=()):
    """[n, n]: key j is seen from i; ``hide``: positions that later ones do not see, to show that they matter."""
    at = torch.arange(n)
    ok = (at[None] <= at[:, None]) & (at[:, None] - at[None] < window)
    for j in hide:
        ok[j + 1:, j] = False
    return ok


def sink_weights(scores, ok):
    """exp(s) / (1 + sum exp(s)) over the visible keys."""
    s = scores.masked_fill(~ok, -math.inf)
    top = torch.clamp(s.max(-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def softmax_weights(scores, ok):
    s = scores.masked_fill(~ok, -math.inf)
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def talking_attention(q, k, v, scale, cap, window, talk, hide=()):
    """q [n, H, d], k [n, G, d], v [n, G, dv] -> [n, H, dv]: capped scores, weights with a sink of score zero, mixed across heads."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    ok = seen(n, window, hide)
    own = []
    for h in range(H):
        s = q[:, h] @ k[:, h // (H // G)].T * scale
        own.append(sink_weights(cap * torch.tanh(s / cap), ok))
    out = []
    for h in range(H):
        mixed = sum(talk[h, g] * own[g] for g in range(H))
        out.append(mixed @ v[:, h // (H // G)])
    return torch.stack(out, 1)


def attention(h, w, p, m, hide=()):
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    base, dims = m["rot"]["base"], m["rot"]["dims"]

    def project(name, heads):
        return (h @ w[p + name].T + w[p + name + ".b"]).view(n, heads, -1)
    q, k = [turn(project(*a), base, dims, True) for a in (("q", H), ("k", G))]
    v = turn(project("v", G), base, dv, True)
    o = talking_attention(q, k, v, m["scale"], m["softcap"], m["mask"]["size"], w[p + "talk"], hide)
    return turn(o, base, dv, True, back=True).reshape(n, H * dv) @ w[p + "o"].T


def latent_attention(h, w, p, m, eps, held, hide=()):
    """``held``: (latents, rotated key parts) of earlier layers by number; this layer's are returned (None where it reads another's)."""
    n, H, d, r, dv = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    base = m["rot"]["base"]
    q = (h @ w[p + "q"].T).view(n, H, d + r)
    q_flat, q_turned = q[..., :d], turn(q[..., d:], base, r, False)
    own = None
    if m.get("kv_from") is not None:
        c, kr = held[m["kv_from"]]
    else:
        low = h @ w[p + "dkv"].T
        c = rms_norm(low[:, :m["kv_rank"]], w[p + "dkv.norm"], eps)
        kr = turn(low[:, None, m["kv_rank"]:], base, r, False)[:, 0]
        own = c, kr
    k, v = (c @ w[p + "uk"].T).view(n, H, d), (c @ w[p + "uv"].T).view(n, H, dv)
    ok, out = seen(n, m["mask"]["size"], hide), []
    for a in range(H):
        s = (q_flat[:, a] @ k[:, a].T + q_turned[:, a] @ kr.T) * m["scale"]
        out.append(softmax_weights(s, ok) @ v[:, a])
    o = torch.cat(out, -1) * sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T, own


def feed_forward(h, w, p):
    return xielu(h @ w[p + "up"].T + w[p + "up.b"], *w[p + "act"].tolist()) @ w[p + "down"].T + w[p + "down.b"]


def hyper(xs, w, p, sublayer):
    """xs [streams, n, width] -> the streams after a sublayer."""
    u = sum(w[p + "in"][s] * xs[s] for s in range(len(xs)))
    y = sublayer(u)
    return torch.stack([sum(w[p + "mix"][s, t] * xs[s] for s in range(len(xs))) + w[p + "out"][t] * y for t in range(len(xs))])


# ------------------------------------------------------------------------------------------------ the model
def forward(cfg, weights, tokens, hide=(), layers=None):
    """Logits [n, vocab] of a whole sequence; ``layers`` (a list) receives the sum of the streams after every layer."""
    w = {k: v.to(DOUBLE) for k, v in weights.items()}
    eps, held = cfg["norm"]["eps"], {}
    e = rms_norm(w["embed"][torch.tensor(tokens)], w["embed.norm"], eps)
    xs = torch.stack([e] * cfg["streams"])
    for i, spec in enumerate(cfg["layers"]):
        m, p = spec["mixer"], f"l{i}."

        def mixer(u):
            h = rms_norm(u, w[p + "norm1"], eps)
            if spec["type"] == "attention":
                return attention(h, w, p + "mix.", m, hide)
            y, held[i] = latent_attention(h, w, p + "mix.", m, eps, held, hide)
            return y
        xs = hyper(xs, w, p + "hc1.", mixer)
        if spec.get("mlp"):
            xs = hyper(xs, w, p + "hc2.", lambda u: feed_forward(rms_norm(u, w[p + "norm2"], eps), w, p + "mlp."))
        if layers is not None:
            layers.append(xs.sum(0))
    return rms_norm(xs.sum(0), w["final.norm"], eps) @ w["head"].T


def greedy(cfg, weights, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, weights, toks)[-1].argmax()))
    return toks[len(prompt):]
