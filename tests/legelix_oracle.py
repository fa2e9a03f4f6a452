"""Plain, slow Legelix in float64, one function per mechanism, from the equations only: the yardstick of the Legelix tests.

Nothing of the package is used here.  Weights are a dict of checkpoint names; a sequence is processed whole, the
recurrences one token after the other.
"""
from __future__ import annotations

import json
import math
import os

import torch

DOUBLE = torch.float64


# ------------------------------------------------------------------------------------------------ mechanisms
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def silu(z):
    return z / (1 + torch.exp(-z))


def frequencies(rot):
    """Angle per position of every rotated pair, stretched for wavelengths beyond the original context."""
    out = []
    sc = rot.get("scaling")
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        if sc:
            wave = 2 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wave >= sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate(x, freqs):
    """x [n, heads, dim]: neighbours (2i, 2i + 1) turn by position times frequency i; dimensions behind them stay."""
    y = x.clone()
    for p in range(x.shape[0]):
        for i, f in enumerate(freqs):
            c, s = math.cos(p * f), math.sin(p * f)
            u, v = x[p, :, 2 * i], x[p, :, 2 * i + 1]
            y[p, :, 2 * i], y[p, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


def attend(q, k, v, scale, size, sink, hide=()):
    """q [n, H, d], k [n, G, d], v [n, G, dv] -> [n, H * dv].  Position i sees 0..i of its own chunk of ``size``; every head
    has a sink in its denominator (``None``: none).  ``hide``: key positions left out, to show that they matter."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    at = torch.arange(n)
    seen = (at[None] <= at[:, None]) & (at[None] // size == at[:, None] // size)
    for j in hide:
        seen[j + 1:, j] = False
    out = []
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T * scale).masked_fill(~seen, -math.inf)
        top = s.max(-1, keepdim=True).values
        if sink is not None:
            top = top.clamp(min=float(sink[h]))
        e = torch.exp(s - top)
        den = e.sum(-1, keepdim=True) + (0 if sink is None else torch.exp(sink[h] - top))
        out.append(e / den @ v[:, g])
    return torch.cat(out, dim=-1)


def attention(h, w, p, m, eps, hide=()):
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(n, H, d)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).view(n, G, d)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(n, G, dv)
    f = frequencies(m["rot"])
    q = rotate(unit_rms(q, eps) * w[p + "q.norm"], f)
    k = rotate(unit_rms(k, eps) * w[p + "k.norm"], f)
    return attend(q, k, v, m["scale"], m["mask"]["size"], w[p + "sink"], hide) @ w[p + "o"].T + w[p + "o.b"]


def short_conv(x, w, b, before=None):
    """x [n, C], w [C, taps]; ``before`` [taps - 1, C]: the inputs ahead of x (zeros at a sequence's start)."""
    taps = w.shape[1]
    ext = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype) if before is None else before, x])
    return torch.stack([(ext[t:t + taps] * w.T).sum(0) + b for t in range(x.shape[0])])


def ssd(x, B, C, dt, A_log, D, state=None):
    """x [n, H, P], B and C [n, G, N], dt [n, H] (positive) -> (y [n, H, P], state [H, N, P])."""
    n, H, P = x.shape
    G, N = B.shape[1:]
    S = torch.zeros(H, N, P, dtype=x.dtype) if state is None else state.clone()
    y = torch.zeros_like(x)
    for t in range(n):
        for h in range(H):
            g = h // (H // G)
            S[h] = torch.exp(-torch.exp(A_log[h]) * dt[t, h]) * S[h] + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = S[h].T @ C[t, g] + D[h] * x[t, h]
    return y, S


def mamba2(h, w, p, m, eps):
    n, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, xbc, dt = (h @ w[p + "in"].T).split([inner, inner + 2 * G * N, H], dim=-1)
    x, B, C = silu(short_conv(xbc, w[p + "conv"], w[p + "conv.b"])).split([inner, G * N, G * N], dim=-1)
    dt = torch.nn.functional.softplus(dt + w[p + "dt_bias"], threshold=1e9)
    y, _ = ssd(x.view(n, H, P), B.view(n, G, N), C.view(n, G, N), dt, w[p + "A_log"], w[p + "D"])
    y = y.reshape(n, inner) * silu(z)
    y = unit_rms(y.view(n, m["norm_groups"], -1), eps).view(n, inner) * w[p + "norm"]
    return y @ w[p + "o"].T


def gated_scan(q, k, v, alpha, state=None):
    """q, k, alpha [n, H, d], v [n, H, dv] -> (o [n, H, dv], state [H, d, dv])."""
    n, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    o = torch.zeros_like(v)
    for t in range(n):
        for h in range(H):
            S[h] = alpha[t, h][:, None] * S[h] + torch.outer(k[t, h], v[t, h])
            o[t, h] = S[h].T @ q[t, h]
    return o, S


def gla(h, w, p, m, eps):
    n, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(n, H, d) * d ** -0.5
    k, v = (h @ w[p + "k"].T).view(n, H, d), (h @ w[p + "v"].T).view(n, H, dv)
    z = ((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]).view(n, H, d)
    o, _ = gated_scan(q, k, v, torch.sigmoid(z) ** (1.0 / m["tau"]))
    o = (unit_rms(o, eps) * w[p + "norm"]).reshape(n, H * dv) * silu(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def feed_forward(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


# ------------------------------------------------------------------------------------------------ the model
def forward(cfg, weights, tokens, hide=(), layers=None):
    """Logits [n, vocab] of a whole sequence; ``layers`` (a list) receives the stream after every layer."""
    w = {k: v.to(DOUBLE) for k, v in weights.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]

    def norm(x, name):
        return layer_norm(x, w[name], w[name + ".b"], eps)
    x = w["embed"][torch.tensor(tokens)]
    for i, spec in enumerate(cfg["layers"]):
        m, p = spec["mixer"], f"l{i}.mix."
        h = norm(x, f"l{i}.norm1")
        if spec["type"] == "gla":
            y = gla(h, w, p, m, eps)
        else:
            y = (m["left_scale"] * attention(h, w, p + "left.", m["left"], eps, hide)
                 + m["right_scale"] * mamba2(h, w, p + "right.", m["right"], eps))
        x = x + mult * norm(y, f"l{i}.norm1b")
        if spec.get("mlp"):
            x = x + mult * norm(feed_forward(norm(x, f"l{i}.norm2"), w, f"l{i}.mlp."), f"l{i}.norm2b")
        if layers is not None:
            layers.append(x)
    return norm(x, "final.norm") @ w["head"].T


def greedy(cfg, weights, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, weights, toks)[-1].argmax()))
    return toks[len(prompt):]


# ------------------------------------------------------------------------------------------------ small models
def left(heads, kv_heads, dim, vdim, chunk, rot=None, scale=None, base=3000.0, scaling=(4.0, 1.0, 4.0, 256)):
    """``scaling``: (factor, low, high, original) or None."""
    r = dict(base=base, dims=rot if rot is not None else dim)
    if scaling:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, mask=dict(size=chunk), rot=r, scale=scale if scale is not None else dim ** -0.5)


def right(heads, vdim, state, groups=1, conv=4, norm_groups=1):
    return dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups)


def parallel(a, s, ff, left_scale=1.0, right_scale=1.0):
    return dict(type="parallel", mixer=dict(left=a, right=s, left_scale=left_scale, right_scale=right_scale),
                mlp=None if ff is None else dict(kind="dense", ff=ff))


def gated(heads, dim, vdim, tau, ff):
    return dict(type="gla", mixer=dict(heads=heads, dim=dim, vdim=vdim, tau=tau), mlp=None if ff is None else dict(kind="dense", ff=ff))


def config(width, vocab, layers, eps=1e-5, residual_mult=0.8):
    return dict(architecture="Legelix", vocab=vocab, width=width, norm=dict(eps=eps), residual_mult=residual_mult, layers=layers)


def small():
    """Layers that differ in every size, two without a feed-forward."""
    return config(96, 208, [
        parallel(left(6, 2, 24, 24, 50, rot=16), right(4, 24, 16, groups=2, conv=3, norm_groups=2), 72, 1.2, 0.7),
        gated(3, 20, 28, 8.0, 56),
        parallel(left(4, 4, 16, 40, 24, scale=0.4, base=500.0, scaling=(8.0, 1.0, 2.0, 64)), right(3, 16, 40), None, 0.6, 1.1),
        gated(2, 32, 16, 4.0, None)])


def uneven():
    """Sizes that no vectorised path takes: nothing is a multiple of four; taps, groups and heads of one."""
    return config(50, 101, [
        gated(1, 7, 9, 3.0, 30),
        parallel(left(3, 1, 10, 6, 33, rot=6, scaling=None), right(1, 13, 5, conv=1), 22, 0.9, 1.0),
        parallel(left(5, 5, 6, 14, 1), right(6, 5, 9, groups=3, conv=2, norm_groups=5), 18)], residual_mult=1.0, eps=1e-3)


def wide():
    """Head sizes of the tensor-core attention kernels, states of real sizes, a chunk that ends inside pages and tiles."""
    return config(128, 160, [
        parallel(left(8, 2, 128, 128, 96, rot=64), right(4, 64, 128, groups=2, norm_groups=4), 192, 0.8, 0.9),
        gated(2, 128, 128, 16.0, 128),
        parallel(left(2, 1, 128, 128, 200), right(2, 128, 64), 136, 1.1, 0.5)])


def only_gated():
    """No attention, hence no pages at all."""
    return config(64, 96, [gated(2, 16, 24, 6.0, 40), gated(4, 24, 8, 16.0, 24)])


MODELS = dict(small=small, uneven=uneven, wide=wide, only_gated=only_gated)


def make_weights(cfg, seed=0, rank=6, sink=0.5, lasting=False):
    """``lasting``: decays close to one, so that a state remembers the first tokens for hundreds of steps."""
    g = torch.Generator().manual_seed(seed)

    def mat(*shape, size=1.0):
        return (torch.randn(*shape, generator=g) * size / math.sqrt(shape[-1])).to(torch.bfloat16).float()

    def vec(*shape, size=0.2, centre=0.0):
        return (centre + torch.randn(*shape, generator=g) * size).to(torch.bfloat16).float()
    H = cfg["width"]
    w = {"embed": vec(cfg["vocab"], H, size=1.0), "head": mat(cfg["vocab"], H)}

    def norm(name):
        w[name], w[name + ".b"] = vec(H, centre=1.0), vec(H)
    norm("final.norm")
    for i, spec in enumerate(cfg["layers"]):
        m, p = spec["mixer"], f"l{i}.mix."
        norm(f"l{i}.norm1")
        norm(f"l{i}.norm1b")
        if spec["type"] == "gla":
            qk, v = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            w[p + "q"], w[p + "k"], w[p + "v"], w[p + "g"] = mat(qk, H), mat(qk, H), mat(v, H), mat(v, H)
            w[p + "a1"], w[p + "a2"] = mat(rank, H), mat(qk, rank, size=0.5 if lasting else 1.5)
            w[p + "a2.b"], w[p + "norm"], w[p + "o"] = vec(qk, size=0.5, centre=5.0 if lasting else 0.5), vec(m["vdim"], centre=1.0), mat(H, v)
        else:
            a, s = m["left"], m["right"]
            for n, k in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                w[f"{p}left.{n}"], w[f"{p}left.{n}.b"] = mat(k, H), vec(k)
            w[p + "left.q.norm"], w[p + "left.k.norm"] = vec(a["dim"], centre=1.5), vec(a["dim"], centre=1.5)
            w[p + "left.sink"] = vec(a["heads"], size=1.0, centre=sink)
            w[p + "left.o"], w[p + "left.o.b"] = mat(H, a["heads"] * a["vdim"]), vec(H)
            inner = s["heads"] * s["vdim"]
            ch = inner + 2 * s["groups"] * s["state"]
            w[p + "right.in"], w[p + "right.conv"], w[p + "right.conv.b"] = mat(inner + ch + s["heads"], H), vec(ch, s["conv"], size=0.5), vec(ch)
            w[p + "right.dt_bias"] = vec(s["heads"], size=0.5, centre=-3.0 if lasting else -0.5)
            w[p + "right.A_log"] = vec(s["heads"], size=0.3, centre=-2.0 if lasting else 0.0)
            w[p + "right.D"], w[p + "right.norm"], w[p + "right.o"] = vec(s["heads"], centre=1.0), vec(inner, centre=1.0), mat(H, inner)
        if spec.get("mlp"):
            norm(f"l{i}.norm2")
            norm(f"l{i}.norm2b")
            ff = spec["mlp"]["ff"]
            w[f"l{i}.mlp.gate"], w[f"l{i}.mlp.up"], w[f"l{i}.mlp.down"] = mat(ff, H), mat(ff, H), mat(H, ff)
    return w


def plant_key(cfg, w, key_token, query_token, gain=3.0):
    """Make every head of layer 0 look at ``key_token`` from ``query_token``, however far apart: one dimension behind the rotated
    ones is given to that pair alone."""
    m, p = cfg["layers"][0]["mixer"]["left"], "l0.mix.left."
    d, e = m["dim"], m["rot"]["dims"]
    assert e < d
    h = layer_norm(w["embed"].double(), w["l0.norm1"].double(), w["l0.norm1.b"].double(), cfg["norm"]["eps"])
    for n, heads, tok in (("q", m["heads"], query_token), ("k", m["kv_heads"], key_token)):
        a = w[p + n].view(heads, d, -1)
        a *= 0.3
        a[:, e] = (4.0 * h[tok] / (h[tok] @ h[tok])).to(torch.bfloat16).float()
        b = w[p + n + ".b"].view(heads, d)
        b *= 0.3
        b[:, e] = 0.0
        w[p + n + ".norm"][e] = gain
    w["l0.mix.left.sink"] *= 0.0
    for k in w:                                                # what a checkpoint can hold
        w[k] = w[k].to(torch.bfloat16).float()
