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


# ------------------------------------------------------------------------------------------------ small models
def attn(heads, kv_heads, dim, vdim, rot, scale=None, base=3000.0, scaling=(4.0, 256, 8.0, 1.0), kv_from=None):
    """``scaling``: (factor, original, fast, slow) or None."""
    r = dict(base=base, dims=rot)
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot=r, scale=scale if scale is not None else dim ** -0.5)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="attention", mixer=m)


def memory(heads, dim, vdim, cap=8.0):
    return dict(type="mlstm", mixer=dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap))


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(ff, experts, identity, top, groups=None, shared=None, scale=1.0):
    """``groups``: (count, keep) over experts and identity experts together."""
    r = dict(experts=experts, identity=identity, top=top, scale=scale)
    if groups:
        r["groups"] = dict(zip(("count", "keep"), groups))
    return dict(dict(kind="moe", expert=dict(ff=ff), router=r), **(dict(shared=dict(ff=shared)) if shared else {}))


def config(width, vocab, layers, eps=1e-5, softcap=20.0):
    """``layers``: (mixer, feed-forward or None) pairs."""
    return dict(architecture="Kopadra", vocab=vocab, width=width, norm=dict(eps=eps), logit_softcap=softcap,
                layers=[dict(m, mlp=f) for m, f in layers])


def small():
    """Layers that differ in every size; one without a feed-forward, two that read an earlier layer's keys."""
    return config(96, 208, [
        (attn(6, 2, 24, 40, 16), moe(40, 7, 2, 3, (3, 2), 56, 1.7)),
        (memory(3, 20, 28), dense(72)),
        (attn(4, 4, 32, 16, 8, scale=0.3, base=500.0, scaling=(8.0, 64, 4.0, 0.5)), None),
        (attn(6, 2, 24, 40, 10, scale=0.15, base=90.0, scaling=None, kv_from=0), dense(48)),
        (memory(2, 32, 12, cap=3.0), moe(24, 6, 0, 2)),
        (attn(4, 4, 32, 16, 32, kv_from=2), moe(16, 4, 4, 5, (4, 3), None, 0.6))])


def uneven():
    """Sizes that no vectorised path takes: nothing is a multiple of four; heads, groups and choices of one."""
    return config(50, 101, [
        (memory(1, 7, 9, cap=5.0), moe(11, 3, 2, 1, (5, 2), 13, 2.5)),
        (attn(3, 1, 10, 6, 6, scaling=None), dense(22)),
        (memory(5, 13, 6), None),
        (attn(3, 1, 10, 6, 10, scaling=(2.0, 40, 2.0, 1.0), kv_from=1), moe(9, 1, 1, 1)),
        (attn(2, 2, 6, 14, 2, scale=0.7), dense(18))], eps=1e-3, softcap=7.0)


def wide():
    """Head sizes of the tensor-core attention kernels, states of real sizes."""
    return config(128, 160, [
        (attn(8, 2, 128, 128, 64), moe(64, 9, 3, 4, (3, 1), 72, 2.2)),
        (memory(4, 64, 96, cap=15.0), dense(136)),
        (attn(8, 2, 128, 128, 128, scale=0.06, kv_from=0), moe(96, 6, 6, 6, (2, 2), 64)),
        (memory(2, 128, 128), dense(64))])


def middling():
    """Head sizes of the 16-bit CUDA-core attention kernel."""
    return config(64, 96, [(attn(4, 2, 64, 64, 32), dense(40)), (memory(2, 16, 24), moe(32, 4, 2, 2, (2, 1), 40)),
                           (attn(4, 2, 64, 64, 64, scale=0.2, kv_from=0), None)])


def only_memory():
    """No attention, hence no pages at all."""
    return config(64, 96, [(memory(2, 16, 24), dense(40)), (memory(4, 24, 8, cap=2.0), moe(24, 4, 2, 2, (3, 2), 24))])


def only_attention():
    """No recurrent layer, hence no state slots; finished prompts stay in the prefix cache, for the layers that share keys too."""
    return config(64, 96, [(attn(4, 1, 16, 16, 8), dense(40)), (attn(4, 1, 16, 16, 16, scale=0.4, kv_from=0), moe(24, 5, 1, 3, (3, 2))),
                           (attn(4, 1, 16, 16, 4, kv_from=0), None)])


MODELS = dict(small=small, uneven=uneven, wide=wide, middling=middling, only_memory=only_memory, only_attention=only_attention)


def make_weights(cfg, seed=0, steady=False, lasting=False, input_bias=0.0):
    """Embeddings have a part in common, and a memory's keys resemble its queries, so that S^T q does not lie near zero, where the norm
    behind it would blow up any rounding.  ``steady``: choice scores far apart, so that 16-bit rounding cannot change which experts are chosen.  ``lasting``: forget gates
    close to one, so that a state remembers the first tokens for hundreds of steps.  ``input_bias``: centre of the input gates."""
    g = torch.Generator().manual_seed(seed)

    def mat(*shape, size=1.0):
        return (torch.randn(*shape, generator=g) * size / math.sqrt(shape[-1])).to(torch.bfloat16).float()

    def vec(*shape, size=0.2, centre=0.0):
        return (centre + torch.randn(*shape, generator=g) * size).to(torch.bfloat16).float()
    H = cfg["width"]
    w = {"embed": vec(cfg["vocab"], H, size=1.0), "final.norm": vec(H, centre=1.0)}
    w["embed"][:, :H // 2] += vec(H // 2, size=2.0)
    w["embed"] = w["embed"].to(torch.bfloat16).float()
    w["final.norm"][:H // 2] *= 0.03125                        # the part in common shall not fill the logits

    def ffn(p, ff):
        w[p + "gate"], w[p + "up"], w[p + "down"] = mat(ff, H, size=1.3), mat(ff, H), mat(H, ff)
    for i, spec in enumerate(cfg["layers"]):
        m, p = spec["mixer"], f"l{i}.mix."
        w[f"l{i}.norm1"] = vec(H, centre=1.0)
        if spec["type"] == "mlstm":
            n, qk, v = m["heads"], m["heads"] * m["dim"], m["heads"] * m["vdim"]
            w[p + "q"], w[p + "k"], w[p + "v"], w[p + "g"], w[p + "o"] = mat(qk, H), mat(qk, H), mat(v, H), mat(v, H), mat(H, v, size=1.5)
            w[p + "k"] = (0.8 * w[p + "q"] + 0.6 * w[p + "k"]).to(torch.bfloat16).float()
            w[p + "norm"] = vec(v, centre=1.0)
            w[p + "i"], w[p + "i.b"] = mat(n, H, size=0.3 if lasting else 2.0), vec(n, size=1.0, centre=input_bias)
            w[p + "f"], w[p + "f.b"] = mat(n, H, size=0.3 if lasting else 2.0), vec(n, size=0.5, centre=6.0 if lasting else 1.5)
        else:
            parts = [("q", m["heads"] * m["dim"])]
            if m.get("kv_from") is None:
                parts += [("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])]
            for n, k in parts:
                w[p + n], w[p + n + ".b"] = mat(k, H), vec(k, size=0.5)
                if n != "v":
                    w[p + n + ".norm"] = vec(k, size=0.4, centre=1.4)
            v = m["heads"] * m["vdim"]
            w[p + "g"], w[p + "o"] = mat(v, H, size=1.5), mat(H, v, size=2.0)
        if spec.get("mlp"):
            mlp, p = spec["mlp"], f"l{i}.mlp."
            w[f"l{i}.norm2"] = vec(H, centre=1.0)
            if mlp["kind"] == "dense":
                ffn(p, mlp["ff"])
                continue
            E = mlp["router"]["experts"] + mlp["router"]["identity"]
            w[p + "router"], w[p + "correction"] = mat(E, H, size=1.5), vec(E, size=0.15, centre=-0.3)
            if steady:                                         # scores are below one: steps of more than that decide
                w[p + "correction"] = (1.25 * torch.randperm(E, generator=g) - 1.25 * E).to(torch.bfloat16).float()
            for e in range(mlp["router"]["experts"]):
                ffn(f"{p}e{e}.", mlp["expert"]["ff"])
            if mlp.get("shared"):
                ffn(p + "shared.", mlp["shared"]["ff"])
    return w


def plant_key(cfg, w, key_token, query_token, reader=0, gain=3.0):
    """Make every head of layer ``reader`` look at ``key_token`` from ``query_token``, however far apart: one dimension behind the
    rotated ones is given to that pair alone.  The keys are layer 0's; with ``reader`` 1 layer 0 adds nothing to the stream."""
    assert reader == 0 or (cfg["layers"][0]["mlp"] is None and cfg["layers"][1]["mixer"]["kv_from"] == 0)
    m = cfg["layers"][0]["mixer"]
    d, e = m["dim"], max(cfg["layers"][j]["mixer"]["rot"]["dims"] for j in (0, reader))
    assert e < d

    def finder(layer, tok):
        """A row that gives 4 for this token's input and little for the others'."""
        h = layer_norm(w["embed"].double(), w[f"l{layer}.norm1"].double(), cfg["norm"]["eps"])
        own = h[tok] - h.mean(0)
        return (4.0 * own / (own @ h[tok])).float()
    if reader:
        w["l0.mix.o"] *= 0.0
    for layer, n, heads, tok in ((reader, "q", m["heads"], query_token), (0, "k", m["kv_heads"], key_token)):
        p = f"l{layer}.mix.{n}"
        a, b = w[p].view(heads, d, -1), w[p + ".b"].view(heads, d)
        a *= 0.3
        a[:, e] = finder(layer, tok)
        b *= 0.3
        b[:, e] = 0.0
        w[p + ".norm"].view(heads, d)[:, e] = gain
    for k in w:                                                # what a checkpoint can hold
        w[k] = w[k].to(torch.bfloat16).float()
