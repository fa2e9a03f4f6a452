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
    at = torch.arange(first, first + x.shape[0], dtype=x.dtype)[:, None]
    for i in range(dims // 2):
        a = at * base ** (-2.0 * i / dims)
        c, s = torch.cos(a), -torch.sin(a) if back else torch.sin(a)
        m, n = (i, i + dims // 2) if halves else (2 * i, 2 * i + 1)
        y[..., m], y[..., n] = x[..., m] * c - x[..., n] * s, x[..., n] * c + x[..., m] * s
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


# ------------------------------------------------------------------------------------------------ small models
def attn(heads, kv_heads, dim, vdim, rot, window, softcap=4.0, scale=None, base=3000.0):
    return dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot=dict(base=base, dims=rot),
                                             mask=dict(size=window), softcap=softcap, scale=scale if scale is not None else dim ** -0.5))


def latent(heads, dim, rot_dim, vdim, kv_rank, window, scale=None, base=900.0, kv_from=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, rot=dict(base=base, dims=rot_dim), mask=dict(size=window),
             scale=scale if scale is not None else (dim + rot_dim) ** -0.5)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="latent_attention", mixer=m)


def config(width, vocab, layers, streams, eps=1e-5):
    """``layers``: (mixer, width of the feed-forward or None) pairs."""
    return dict(architecture="Gizilorn", vocab=vocab, width=width, norm=dict(eps=eps), streams=streams,
                layers=[dict(copy.deepcopy(m), mlp=f and dict(kind="dense", ff=f)) for m, f in layers])


def small():
    """Layers that differ in every size; one without a feed-forward, two that read an earlier layer's latents."""
    return config(96, 208, [
        (attn(6, 2, 24, 40, 16, 70), 72),
        (latent(4, 20, 12, 28, 48, 50), 56),
        (attn(4, 4, 32, 16, 8, 33, softcap=9.0, scale=0.3, base=500.0), None),
        (latent(6, 8, 12, 44, 48, 90, scale=0.2, kv_from=1), 40),
        (latent(2, 32, 20, 16, 40, 64, base=70.0), None),
        (attn(2, 1, 16, 24, 16, 129, softcap=2.0), 96),
        (latent(4, 24, 20, 20, 40, 17, base=70.0, kv_from=4), 64)], 3)


def uneven():
    """Sizes that no vectorised path takes: nothing is a multiple of four; heads and groups of one, more streams than are unrolled."""
    return config(50, 101, [
        (attn(3, 1, 10, 6, 6, 21, softcap=7.0), 22),
        (latent(1, 7, 2, 5, 9, 40), 11),
        (attn(2, 2, 6, 14, 2, 100, softcap=1.5, scale=0.7), None),
        (latent(3, 5, 2, 7, 9, 66, scale=0.5, kv_from=1), 13)], 5, eps=1e-3)


def wide():
    """Head sizes of the tensor-core kernels; two heads per KV head, and four."""
    return config(128, 160, [
        (attn(8, 2, 128, 128, 64, 100, softcap=20.0), 136),
        (latent(4, 64, 32, 64, 128, 80), 128),
        (attn(4, 2, 128, 128, 128, 190, softcap=3.0, scale=0.06), 64),
        (latent(8, 128, 32, 96, 128, 130, kv_from=1, scale=0.09), 200)], 2)


def broad():
    """Many heads: all of the decode kernel's columns, and more heads than it takes; latents of the full width."""
    return config(128, 96, [
        (attn(32, 8, 128, 128, 128, 150, softcap=50.0), 64),
        (latent(20, 128, 64, 128, 512, 90), 64),
        (attn(48, 3, 128, 128, 32, 70, softcap=30.0), None)], 4)


def plain():
    """One stream, one head of everything, a window of one token and one longer than any sequence."""
    return config(64, 90, [(attn(1, 1, 16, 16, 16, 1), 40), (latent(1, 16, 8, 16, 24, 5000), None), (attn(1, 1, 8, 32, 4, 4000), 24),
                           (latent(2, 8, 8, 8, 24, 1, kv_from=1), 32)], 1)


def only_latent():
    return config(64, 96, [(latent(2, 16, 8, 24, 32, 40), 40), (latent(4, 24, 8, 8, 32, 70, scale=0.4, kv_from=0), 32)], 2)


def only_attention():
    return config(64, 96, [(attn(4, 1, 16, 16, 8, 60), 40), (attn(4, 2, 24, 16, 16, 90, scale=0.4), None)], 3)


MODELS = dict(small=small, uneven=uneven, wide=wide, broad=broad, plain=plain, only_latent=only_latent, only_attention=only_attention)


def make_weights(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)

    def mat(*shape, size=1.0):
        return (torch.randn(*shape, generator=g) * size / math.sqrt(shape[-1])).to(torch.bfloat16).float()

    def vec(*shape, size=0.2, centre=0.0):
        return (centre + torch.randn(*shape, generator=g) * size).to(torch.bfloat16).float()
    W, S = cfg["width"], cfg["streams"]
    w = {"embed": vec(cfg["vocab"], W, size=1.0), "embed.norm": vec(W, centre=1.0), "final.norm": vec(W, centre=1.0),
         "head": mat(cfg["vocab"], W)}

    def connection(p):
        w[p + "in"], w[p + "out"] = vec(S, size=0.3, centre=0.8), vec(S, size=0.4, centre=1.0)
        w[p + "mix"] = (0.8 * torch.eye(S) + torch.randn(S, S, generator=g) * 0.2).to(torch.bfloat16).float()
    for i, spec in enumerate(cfg["layers"]):
        m, p = spec["mixer"], f"l{i}.mix."
        w[f"l{i}.norm1"] = vec(W, centre=1.0)
        connection(f"l{i}.hc1.")
        H, dv = m["heads"], m["vdim"]
        if spec["type"] == "attention":
            for n, k in (("q", H * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * dv)):
                w[p + n], w[p + n + ".b"] = mat(k, W, size=1.5 if n != "v" else 1.0), vec(k, size=0.5)
            w[p + "talk"] = (0.6 * torch.eye(H) + torch.randn(H, H, generator=g) * 0.5 / math.sqrt(H)).to(torch.bfloat16).float()
        else:
            R, r = m["kv_rank"], m["rot_dim"]
            w[p + "q"], w[p + "g"] = mat(H * (m["dim"] + r), W, size=1.5), mat(H * dv, W, size=1.5)
            if m.get("kv_from") is None:
                w[p + "dkv"], w[p + "dkv.norm"] = mat(R + r, W, size=1.5), vec(R, centre=1.0)
            w[p + "uk"], w[p + "uv"] = mat(H * m["dim"], R), mat(H * dv, R)
        w[p + "o"] = mat(W, H * dv, size=1.5)
        if spec.get("mlp"):
            p = f"l{i}.mlp."
            w[f"l{i}.norm2"] = vec(W, centre=1.0)
            connection(f"l{i}.hc2.")
            ff = spec["mlp"]["ff"]
            w[p + "up"], w[p + "up.b"], w[p + "down"], w[p + "down.b"] = mat(ff, W), vec(ff, size=0.5), mat(W, ff, size=0.7), vec(W, size=0.3)
            w[p + "act"] = vec(2, size=0.7)
    return w


def plant_key(cfg, w, X, Q, layer=0, gain=9.0):
    """Token Q's query in ``layer`` scores high with token X's key there, at any distance: dimension 0 of the input marks X, dimension 1
    marks Q, and an unrotated key dimension carries the product."""
    W, m, p = cfg["width"], cfg["layers"][layer]["mixer"], f"l{layer}.mix."
    w["embed"][:, :2] = 0.0
    for n in w:
        if n.endswith((".o", ".down", ".down.b")):
            w[n][:2] = 0.0                                     # nothing else writes to the marks
    w["embed"][X, 0] = w["embed"][Q, 1] = math.sqrt(W)
    H = m["heads"]
    if cfg["layers"][layer]["type"] == "attention":
        d, at = m["dim"], m["dim"] - 1                         # the last dimension does not turn (rot dims < dim)
        assert m["rot"]["dims"] < d
        for h in range(H):
            w[p + "q"][h * d + at] = 0.0
            w[p + "q"][h * d + at, 1] = gain
            w[p + "q.b"][h * d + at] = 0.0
        for c in range(m["kv_heads"]):
            w[p + "k"][c * d + at] = 0.0
            w[p + "k"][c * d + at, 0] = 2.0
            w[p + "k.b"][c * d + at] = 0.0
    else:
        d, r = m["dim"], m["rot_dim"]
        own = f"l{m.get('kv_from', layer)}.mix."
        w[own + "dkv"][0] = 0.0
        w[own + "dkv"][0, 0] = 4.0
        w[own + "dkv.norm"][0] = 1.0
        for h in range(H):
            w[p + "q"][h * (d + r)] = 0.0
            w[p + "q"][h * (d + r), 1] = gain
            w[p + "uk"][h * d] = 0.0
            w[p + "uk"][h * d, 0] = 1.0
