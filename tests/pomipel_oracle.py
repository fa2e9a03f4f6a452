"""Plain, slow Pomipel in float64, one function per mechanism, from the equations only: the yardstick of the Pomipel tests.

Nothing of the package is used here.  Weights are a dict of checkpoint names; sequences are processed whole, one
head, one expert and (in the router) one token at a time.
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


def centred_norm(x, w, eps):
    """RMS norm whose gain is one plus the stored weight."""
    return unit_rms(x, eps) * (1.0 + w)


def embed(tokens, table, positions, scale, start=0):
    return torch.stack([table[t] * scale + positions[start + i] for i, t in enumerate(tokens)])


def query_latent(h, w_dq, g, eps):
    return unit_rms(h @ w_dq.T, eps) * g


def kv_latent(h, w_dkv, g, eps):
    return unit_rms(h @ w_dkv.T, eps) * g


def attend(c_q, c, w_uq, w_uk, w_uv, heads, dim, vdim, scale, hide=()):
    """[n, heads * vdim]; query i sees latents 0..i (``hide``: key positions left out, to show that they matter)."""
    n = c.shape[0]
    q, k, v = (c_q @ w_uq.T).view(n, heads, dim), (c @ w_uk.T).view(n, heads, dim), (c @ w_uv.T).view(n, heads, vdim)
    seen = torch.ones(n, n, dtype=torch.bool).tril()
    for j in hide:
        seen[j + 1:, j] = False
    out = []
    for h in range(heads):
        s = (q[:, h] @ k[:, h].T * scale).masked_fill(~seen, -math.inf)
        out.append(torch.softmax(s, dim=-1) @ v[:, h])
    return torch.cat(out, dim=-1)


def route(h, w_router, correction, top, count, keep):
    """One token: [(expert, weight)] in order of choice."""
    s = torch.sigmoid(w_router @ h)
    choice = (s + correction).tolist()
    size = len(choice) // count
    rank = []
    for g in range(count):
        best = sorted(choice[g * size:(g + 1) * size], reverse=True)[:2]
        rank.append((sum(best), -g))
    open_groups = {-g for _, g in sorted(rank, reverse=True)[:keep]}
    cand = [(choice[e], -e) for e in range(len(choice)) if e // size in open_groups]
    return [(-e, float(s[-e])) for _, e in sorted(cand, reverse=True)[:top]]


def expert(h, up, down):
    return torch.clamp(h @ up.T, min=0.0) ** 2 @ down.T


def feed_forward(h, w, p, spec):
    r = spec["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    mine = [[] for _ in range(r["experts"])]                   # expert: [(token, weight)]
    for t in range(h.shape[0]):
        for e, weight in route(h[t], w[p + "router"], w[p + "correction"], r["top"], groups["count"], groups["keep"]):
            mine[e].append((t, weight))
    out = torch.zeros_like(h)
    for e, pairs in enumerate(mine):
        if pairs:
            at = [t for t, _ in pairs]
            weight = torch.tensor([x for _, x in pairs], dtype=h.dtype)
            out[at] += weight[:, None] * expert(h[at], w[f"{p}e{e}.up"], w[f"{p}e{e}.down"])
    return out


# ------------------------------------------------------------------------------------------------ the model
def forward(cfg, weights, tokens, hide=(), layers=None):
    """Logits [n, vocab] of a whole sequence; ``layers`` (a list) receives the stream after every layer."""
    w = {k: v.to(DOUBLE) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = embed(tokens, w["embed"], w["pos"], cfg["embedding"]["scale"])
    latents = {}
    for i, spec in enumerate(cfg["layers"]):
        m, p = spec["mixer"], f"l{i}.mix."
        if m.get("kv_from") is None:
            latents[i] = kv_latent(x, w[p + "dkv"], w[p + "dkv.norm"], eps)
        c = latents[m["kv_from"] if m.get("kv_from") is not None else i]
        c_q = query_latent(x, w[p + "dq"], w[p + "dq.norm"], eps)
        o = attend(c_q, c, w[p + "uq"], w[p + "uk"], w[p + "uv"], m["heads"], m["dim"], m["vdim"], m["scale"], hide)
        x = x + centred_norm(o @ w[p + "o"].T, w[f"l{i}.norm1"], eps)
        if spec.get("mlp"):
            x = x + centred_norm(feed_forward(x, w, f"l{i}.mlp.", spec["mlp"]), w[f"l{i}.norm2"], eps)
        if layers is not None:
            layers.append(x)
    return centred_norm(x, w["final.norm"], eps) @ w["head"].T * cfg["logit_scale"]


def greedy(cfg, weights, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, weights, toks)[-1].argmax()))
    return toks[len(prompt):]


# ------------------------------------------------------------------------------------------------ small models
def mixer(heads, dim, vdim, q_rank, kv_rank, scale=None, kv_from=None):
    m = dict(heads=heads, dim=dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale if scale is not None else dim ** -0.5)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def moe(ff, experts, top, count, keep):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top, groups=dict(count=count, keep=keep)))


def config(width, vocab, layers, max_positions=512, eps=1e-6, embed_scale=3.0, logit_scale=1.0):
    return dict(architecture="Pomipel", vocab=vocab, width=width, max_positions=max_positions, embedding=dict(scale=embed_scale),
                norm=dict(eps=eps), logit_scale=logit_scale,
                layers=[dict(type="latent_attention", mixer=m, mlp=f) for m, f in layers])


def small(**kw):
    """Layers that differ in every size, one without a feed-forward, two that read an earlier layer's latents."""
    return config(**dict(dict(width=96, vocab=208, layers=[
        (mixer(3, 32, 24, 40, 48), moe(40, 8, 2, 4, 2)),
        (mixer(2, 16, 40, 24, 32, scale=0.4), None),
        (mixer(5, 24, 16, 56, 48, kv_from=0), moe(72, 12, 5, 3, 2)),
        (mixer(1, 64, 8, 16, 32, kv_from=1), moe(24, 4, 1, 1, 1))], logit_scale=0.7, eps=1e-5), **kw))


def uneven():
    """Sizes that no tensor-core path takes: nothing is a multiple of eight."""
    return config(50, 101, [(mixer(3, 10, 6, 14, 18), moe(20, 6, 3, 2, 1)), (mixer(2, 12, 14, 9, 18, kv_from=0), moe(11, 5, 2, 5, 3))],
                  logit_scale=1.3, embed_scale=1.0)


def wide():
    """Head and latent widths that need two 64-wide blocks, more heads than one tile of the decode kernel holds."""
    return config(128, 160, [(mixer(17, 80, 72, 96, 136), moe(64, 8, 2, 2, 1)), (mixer(4, 128, 128, 64, 264), moe(136, 16, 6, 4, 3))])


def make_weights(cfg, seed=0, dtype=torch.float32, pos_size=0.3, steady=False):
    """``steady``: choice scores far apart, so that 16-bit rounding cannot change which experts are chosen."""
    g = torch.Generator().manual_seed(seed)

    def mat(*shape, size=1.0):
        return (torch.randn(*shape, generator=g) * size / math.sqrt(shape[-1])).to(torch.bfloat16).to(dtype)

    def vec(n, size, centre=0.0):
        return (centre + torch.randn(n, generator=g) * size).to(torch.bfloat16).to(dtype)
    H = cfg["width"]
    w = {"embed": vec((cfg["vocab"], H), 0.4), "pos": vec((cfg["max_positions"], H), pos_size), "final.norm": vec(H, 0.2),
         "head": mat(cfg["vocab"], H)}
    for i, spec in enumerate(cfg["layers"]):
        m, p = spec["mixer"], f"l{i}.mix."
        w[f"l{i}.norm1"] = vec(H, 0.2)
        w[p + "dq"], w[p + "dq.norm"] = mat(m["q_rank"], H), vec(m["q_rank"], 0.2, 1.0)
        w[p + "uq"] = mat(m["heads"] * m["dim"], m["q_rank"], size=2.0)          # scores with a spread of a few units
        if m.get("kv_from") is None:
            w[p + "dkv"], w[p + "dkv.norm"] = mat(m["kv_rank"], H), vec(m["kv_rank"], 0.2, 1.0)
        w[p + "uk"], w[p + "uv"] = mat(m["heads"] * m["dim"], m["kv_rank"]), mat(m["heads"] * m["vdim"], m["kv_rank"])
        w[p + "o"] = mat(H, m["heads"] * m["vdim"])
        if spec.get("mlp"):
            w[f"l{i}.norm2"] = vec(H, 0.2)
            r, ff, p = spec["mlp"]["router"], spec["mlp"]["expert"]["ff"], f"l{i}.mlp."
            w[p + "router"], w[p + "correction"] = mat(r["experts"], H), vec(r["experts"], 0.6)
            if steady:
                w[p + "router"] = w[p + "router"] * 0.125
                order = torch.randperm(r["experts"], generator=g).to(dtype)
                # growing steps: sums of two (the rank of a group) do not tie either
                w[p + "correction"] = (0.5 * order + 0.0625 * order * order - 0.25 * r["experts"] - 1.0 / 16).to(torch.bfloat16).to(dtype)
            for e in range(r["experts"]):
                w[f"{p}e{e}.up"], w[f"{p}e{e}.down"] = mat(ff, H), mat(H, ff)
    return w


def plant_key(cfg, w, key_token, query_token, gain=14.0):
    """Make every head of layer 0 look at ``key_token`` from ``query_token`` with a score ``gain`` above the noise: W_uq
    gets a rank-one part that turns the query's latent into the key of that token."""
    m, eps = cfg["layers"][0]["mixer"], cfg["norm"]["eps"]
    d = {k: v.to(DOUBLE) for k, v in w.items() if k in ("embed",) or k.startswith("l0.mix.")}
    x = d["embed"] * cfg["embedding"]["scale"]
    c = kv_latent(x[key_token], d["l0.mix.dkv"], d["l0.mix.dkv.norm"], eps)
    c_q = query_latent(x[query_token], d["l0.mix.dq"], d["l0.mix.dq.norm"], eps)
    k = (d["l0.mix.uk"] @ c).view(m["heads"], m["dim"])
    k = k / (k * k).sum(-1, keepdim=True) * gain / m["scale"]
    uq = 0.2 * d["l0.mix.uq"] + torch.outer(k.reshape(-1), c_q / (c_q @ c_q))
    w["l0.mix.uq"] = uq.to(torch.bfloat16).to(w["l0.mix.uq"].dtype)
    # ... and let the rest of the layer be read from what attention brings
    w["l0.norm1"] = torch.full_like(w["l0.norm1"], 1.0)


def save_model(cfg, w, path):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in w.items()}, os.path.join(path, "model.safetensors"))
    return str(path)


def tokens(cfg, n, seed=0, avoid=()):
    g = torch.Generator().manual_seed(1000 + seed)
    ok = torch.tensor([t for t in range(cfg["vocab"]) if t not in avoid])
    return ok[torch.randint(0, len(ok), (n,), generator=g)].tolist()


def row_error(got, want):
    """Largest error of a row of logits, mean taken off, over the spread of the expected logits."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    spread = (want.double() - want.double().mean(-1, keepdim=True)).pow(2).mean().sqrt()
    return float((d.pow(2).mean(-1).sqrt() / spread).max()) if len(d) else 0.0
