"""Kopadra on the device: every kernel it adds or extends against the plain float64 implementation."""
from types import SimpleNamespace

import pytest
import torch

from tests import kopadra_oracle as ko

pytestmark = pytest.mark.gpu
BF, F32, F64 = torch.bfloat16, torch.float32, torch.float64


def _rand(*shape, seed=0, size=1.0):
    g = torch.Generator().manual_seed(seed)
    return torch.randn(*shape, generator=g) * size


def _close(got, want, tol):
    got, want = got.double().cpu(), want.double().cpu()
    assert torch.isfinite(got).all()
    err = float((got - want).abs().max() / want.abs().max().clamp_min(1e-9))
    assert err < tol, err


def _cu():
    from vllm_b200.ops import cuda_ops
    return cuda_ops()


def _md(q_lens, ctx, table, vt=False):
    qsl = torch.tensor([0] + torch.tensor(q_lens).cumsum(0).tolist(), dtype=torch.int32, device="cuda")
    sl = torch.tensor([c + q for c, q in zip(ctx, q_lens)], dtype=torch.int32, device="cuda")
    return SimpleNamespace(num_reqs=len(q_lens), query_start_loc=qsl, seq_lens=sl, block_table=table, max_query_len=max(q_lens),
                           max_seq_len=max(c + q for c, q in zip(ctx, q_lens)), decode_only=max(q_lens) == 1, flat=False, kv_vt=vt,
                           num_splits=0)


def _slots(rows):
    return torch.tensor(rows, dtype=torch.int32, device="cuda").view(-1, 1).repeat(1, 2).contiguous()


# ------------------------------------------------------------------------------------------------ stream, gates, cap
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,H", [(1, 50), (7, 96), (4, 2048), (2, 9000), (130, 1000)])
@pytest.mark.parametrize("nxt", [True, False])
def test_add_norm(T, H, dtype, nxt):
    from vllm_b200 import ops
    x, y, w = _rand(T, H, seed=1, size=4.0) + 1.5, (_rand(T, H, seed=2) + 0.7).to(dtype), (_rand(H, seed=3, size=0.3) + 1).to(dtype)
    want = x.double() + y.double()
    xs = x.cuda()
    out = ops.add_norm(xs, y.cuda(), (w.cuda(), None) if nxt else None, 1e-3)
    _close(xs, want, 1e-7)                                   # the stream itself is never rounded to 16 bits
    assert out.dtype == dtype
    _close(out, ko.layer_norm(want, w.double(), 1e-3) if nxt else want, 6e-3 if dtype == BF else 3e-6)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,H,ff,E,ident,k,shared", [(5, 96, 40, 6, 3, 4, True), (70, 128, 64, 8, 0, 2, False), (300, 64, 24, 3, 5, 8, True),
                                                     (3, 50, 11, 4, 1, 2, False), (600, 256, 96, 16, 8, 6, True), (33, 40, 8, 2, 2, 1, True)])
def test_experts_with_identities(T, H, ff, E, ident, k, shared, dtype):
    from vllm_b200.layers.common import LayerNorm
    from vllm_b200.layers.moe import FusedMoE
    moe = FusedMoE(E, k, H, ff, dtype, act="silu", identity_experts=ident).cuda()
    w = {}
    for e in range(E):
        for n, shape, shard in (("gate", (ff, H), "w1"), ("up", (ff, H), "w3"), ("down", (H, ff), "w2")):
            w[f"e{e}.{n}"] = (_rand(*shape, seed=10 * e + len(n)) * shape[1] ** -0.5).to(dtype)
            moe.weight_loader(moe.w2_weight if n == "down" else moe.w13_weight, w[f"e{e}.{n}"], shard, e)
    g = torch.Generator().manual_seed(3)
    ids = torch.stack([torch.randperm(E + ident, generator=g)[:k] for _ in range(T)])
    pw = torch.rand(T, k, generator=g)
    h, x, y = _rand(T, H, seed=1).to(dtype), _rand(T, H, seed=2), _rand(T, H, seed=4).to(dtype)
    norm = LayerNorm(H, 1e-4, False, dtype)
    norm.weight.data.copy_((_rand(H, seed=5, size=0.2) + 1).to(dtype))
    norm = norm.cuda()
    want = x.double() + (y.double() if shared else 0)
    wd = {n: t.double() for n, t in w.items()}
    routed = torch.zeros(T, H, dtype=F64)
    for e in range(E + ident):
        out = ko.gated(h.double(), wd, f"e{e}.", ko.silu) if e < E else h.double()
        routed += out * (pw.double() * (ids == e)).sum(-1, keepdim=True)
    xs = x.cuda()
    out = moe.forward_add_norm(h.cuda(), (pw.cuda(), ids.int().cuda()), xs, y.cuda() if shared else None, norm)
    _close(xs, want + routed, 8e-3 if dtype == BF else 3e-6)
    _close(out, ko.layer_norm(want + routed, norm.weight.double().cpu(), 1e-4), 1.5e-2 if dtype == BF else 1e-5)
    _close(moe(h.cuda(), routing=(pw.cuda(), ids.int().cuda())), routed, 1.5e-2 if dtype == BF else 3e-6)


@pytest.mark.parametrize("T", [7, 400])                      # fused logits, and logits of one product
@pytest.mark.parametrize("E,k,count,keep", [(14, 5, 2, 1), (12, 3, 4, 2), (9, 5, 3, 2), (6, 1, 6, 1), (8, 8, 1, 1), (1, 1, 1, 1), (96, 8, 8, 3)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_router(E, k, count, keep, T, dtype):
    from vllm_b200 import ops
    x, w, corr = _rand(T, 72, seed=1).to(dtype), _rand(E, 72, seed=2, size=0.2).to(dtype), _rand(E, seed=3, size=0.3) - 0.5
    wt, ids = ops.router_topk(x.cuda(), w.cuda(), k, count, keep, True, "softmax", corr.cuda(), 1.9, group_score="max")
    s = torch.softmax(x.double() @ w.double().T, -1)
    want = ko.choose(s, corr.double(), k, count, keep)
    same = (ids.cpu().long() == want).all(-1)
    assert same.float().mean() > 0.98                          # all but ties
    sw = s.gather(1, want)
    _close(wt.cpu()[same], (sw / sw.sum(-1, keepdim=True) * 1.9)[same], 2e-5)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,n", [(1, 7), (5, 64), (130, 1000), (3, 4096)])
def test_sigmoid_mul_and_soft_cap(T, n, dtype):
    from vllm_b200 import ops
    a, g = _rand(T, n + 16, seed=1).to(dtype), _rand(T, n + 8, seed=2, size=4.0).to(dtype)
    x, gate = a.cuda()[:, 8:8 + n], g.cuda()[:, :n]
    got = ops.sigmoid_mul_(x, gate)
    assert got.data_ptr() == x.data_ptr()
    _close(got, a[:, 8:8 + n].double() * ko.sigmoid(g[:, :n].double()), 6e-3 if dtype == BF else 2e-6)
    l = _rand(T, n + 24, seed=3, size=30.0).to(dtype)
    buf = l.cuda()
    ops.soft_cap(buf[:, :n], 11.0)
    _close(buf[:, :n], 11.0 * torch.tanh(l[:, :n].double() / 11.0), 6e-3 if dtype == BF else 2e-6)
    assert torch.equal(buf[:, n:].cpu(), l[:, n:])


# ------------------------------------------------------------------------------------------------ attention prologue
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("H,G,d,dv,rot,vt", [(6, 2, 24, 40, 16, False), (3, 1, 10, 6, 6, False), (8, 2, 128, 128, 64, True), (4, 4, 32, 16, 32, False),
                                             (64, 8, 128, 128, 128, True), (1, 1, 2, 4, 2, False), (4, 2, 64, 64, 0, False)])
@pytest.mark.parametrize("alone", [False, True])
def test_whole_norms_rotation_and_cache(H, G, d, dv, rot, vt, alone, dtype):
    if vt and dtype == F32:
        pytest.skip("16-bit cache layout")
    T, BS, eps = 9, 64, 1e-3
    r = dict(base=300.0, dims=rot, scaling=dict(factor=4.0, original=100, fast=8.0, slow=1.0)) if rot else None
    pos = torch.tensor([0, 1, 2, 3, 70, 71, 5, 130, 131])
    slots = torch.tensor([64, 65, 66, 67, 64 * 3 + 6, 64 * 3 + 7, -1, 64 * 4 + 2, 64 * 4 + 3])
    x = _rand(T, H * d + G * d + G * dv + 8, seed=1, size=2.0).to(dtype)
    qw, kw = (_rand(H * d, seed=2, size=0.3) + 1).to(dtype), (_rand(G * d, seed=3, size=0.3) + 1).to(dtype)
    q, k, v, _ = x.double().split([H * d, G * d, G * dv, 8], -1)

    def turned(t, w, heads):
        t = (ko.unit_rms(t, eps) * w.double()).view(T, heads, d)
        if rot == 0:
            return t
        long = torch.zeros(132, heads, d, dtype=F64)
        long[pos] = t
        return ko.rotate(long, r)[pos]
    cs = torch.zeros(200, 0)
    if rot:
        f, size = ko.frequencies(r)
        a = torch.arange(200, dtype=F64)[:, None] * torch.tensor(f, dtype=F64)
        cs = (torch.cat([a.cos(), a.sin()], -1) * size).float()
    dc = max(d, dv)
    cache = torch.full((6, 2, G, BS, dc), 7.0, dtype=dtype, device="cuda")
    xs = x.cuda()
    qs, ks, vs, _ = xs.split([H * d, G * d, G * dv, 8], -1)
    kw_ = dict(v=vs, kv_cache=cache, slot_mapping=slots.cuda()) if not alone else {}
    _cu().fused_qk_norm_rope(pos.cuda(), qs, None if alone else ks, qw.cuda(), None if alone else kw.cuda(), cs.cuda(), d, eps, True,
                             vt=vt, v_head_dim=dv, whole=True, **kw_)
    tol = 8e-3 if dtype == BF else 3e-6
    _close(qs.reshape(T, H, d), turned(q, qw, H), tol)
    if alone:
        assert (cache == 7.0).all() and torch.equal(ks.cpu(), x[:, H * d:H * d + G * d])
        return
    wk = turned(k, kw, G)
    _close(ks.reshape(T, G, d), wk, tol)
    touched = torch.zeros(6 * BS, dtype=torch.bool)
    vp = cache[:, 1].reshape(6, G, dc, BS).transpose(2, 3) if vt else cache[:, 1]
    for t in range(T):
        if slots[t] < 0:
            continue
        b, o = divmod(int(slots[t]), BS)
        touched[slots[t]] = True
        _close(cache[b, 0, :, o, :d], wk[t], tol)
        assert torch.equal(vp[b, :, o, :dv].cpu().reshape(-1), x[t, (H + G) * d:(H + G) * d + G * dv])
    rest = cache[:, 0].transpose(1, 2).reshape(6 * BS, -1)[~touched.cuda()]
    assert (rest == 7.0).all()


@pytest.mark.parametrize("G", [1, 4, 8])
def test_prompt_attention_with_jumping_scores(G):
    """Row maxima that grow by different amounts at different tiles, neighbouring rows included."""
    D, Hkv, n = 128, 2, 700
    q, k, v = [_rand(n, h, D, seed=s).to(BF) for s, h in ((1, Hkv * G), (2, Hkv), (3, Hkv))]
    u = torch.nn.functional.normalize(_rand(D, seed=4), dim=0)
    q = (q.float() + 12.0 * u * (torch.arange(n) % 3 == 0)[:, None, None]).to(BF)
    for j, size in ((140, 4.0), (290, 9.0), (500, 17.0), (641, 30.0)):
        k[j] = (k[j].float() + size * u).to(BF)
    pages = -(-n // 64)
    cache = torch.zeros(pages + 1, 2, Hkv, 64, D, dtype=BF)
    for b in range(pages):
        part = slice(64 * b, min(64 * b + 64, n))
        m = part.stop - part.start
        cache[b + 1, 0, :, :m] = k[part].transpose(0, 1)
        cache[b + 1, 1].view(Hkv, D, 64)[:, :, :m] = v[part].permute(1, 2, 0)
    want = ko.attend(q.double(), k.double(), v.double(), 0.09)
    md = _md([n], [0], torch.arange(1, pages + 1, dtype=torch.int32, device="cuda").view(1, -1), vt=True)
    _close(_cu().paged_attention(q.cuda(), cache.cuda(), md, 0.09).reshape(n, -1), want, 8e-3)
    md = _md([n - 333], [333], md.block_table, vt=True)
    _close(_cu().paged_attention(q[333:].cuda(), cache.cuda(), md, 0.09).reshape(n - 333, -1), want[333:], 8e-3)


# ------------------------------------------------------------------------------------------------ matrix memory
# (tokens of each request in successive steps; 0: left out)
STEPS = [([5, 1, 40], [1, 0, 1], [1, 1, 1], [3, 17, 2]), ([300, 0, 1], [33, 2, 257]), ([1, 1, 1], [1, 1, 1])]


@pytest.mark.parametrize("H,d,dv", [(3, 16, 16), (2, 20, 36), (4, 64, 96), (2, 6, 5), (2, 128, 128), (1, 200, 96), (1, 1, 1), (2, 32, 257), (1, 300, 64)])
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("bias,spread", [(0.0, 1.0), (-8.0, 1.0), (6.0, 4.0)])
def test_matrix_memory_over_steps(H, d, dv, dtype, bias, spread):
    from vllm_b200 import ops
    rows, W, cap, eps = [3, 1, 4], 44, 9.0, 1e-4
    cols = -(-dv // 4) * 4 + 4
    m_off = H * ops.scan_state_elems(d, cols)
    w = _rand(2 * H, W, seed=1, size=spread * W ** -0.5).to(dtype)
    b = _rand(2 * H, seed=2, size=0.5) + torch.tensor([bias] * H + [2.0] * H)
    nw = (_rand(H * dv, seed=3, size=0.3) + 1).to(dtype)
    sizes = [H * d, H * d, H * dv, H * dv]
    for steps in STEPS:
        pool = torch.full((6, m_off + -(-H // 4) * 4), float("nan"), device="cuda")
        n = [sum(s[i] for s in steps) for i in range(3)]
        x = [_rand(n[i], sum(sizes) + 8, seed=10 + i).to(dtype) for i in range(3)]
        h = [_rand(n[i], W + 4, seed=20 + i).to(dtype) for i in range(3)]
        got, at = [[], [], []], [0, 0, 0]
        for s in steps:
            live = [i for i in range(3) if s[i]]
            md = _md([s[i] for i in live], [at[i] for i in live], _slots([rows[i] for i in live]))
            xs = torch.cat([x[i][at[i]:at[i] + s[i]] for i in live]).cuda()
            hs = torch.cat([h[i][at[i]:at[i] + s[i]] for i in live]).cuda()[:, :W].contiguous()
            q, k, v, g, _ = xs.split(sizes + [8], -1)
            gates = _cu().memory_gates(hs, w.cuda(), b.cuda(), cap, pool, m_off, md)
            o = _cu().memory_scan(q, k, v, gates, d ** -0.5, pool, md, H, d, dv)
            o = _cu().gated_norm(o, g, nw.cuda(), H, eps, False, gate="sigmoid", gates=gates)
            for i, part in zip(live, o.split([s[i] for i in live])):
                got[i].append(part)
                at[i] += s[i]
        for i in range(3):
            q, k, v, g, _ = x[i].double().split(sizes + [8], -1)
            z = cap * torch.tanh((h[i][:, :W].double() @ w.double().T + b.double()) / cap)
            want, _ = ko.matrix_memory(q.reshape(n[i], H, d) * d ** -0.5, k.reshape(n[i], H, d), v.reshape(n[i], H, dv), z[:, :H],
                                       -torch.log1p(torch.exp(-z[:, H:])))
            want = ko.unit_rms(want, eps).reshape(n[i], H * dv) * nw.double() * ko.sigmoid(g)
            _close(torch.cat(got[i]), want, 1e-2 if dtype == BF else 1e-4)
        assert pool[[0, 2, 5]].isnan().all()


@pytest.mark.parametrize("R", [12, 32, 60, 128, 200])
def test_scan_forms_agree(R):
    """Lanes hold few or many rows depending on how much runs at once: sequences alone, all together and token by token."""
    from vllm_b200 import ops
    C, B, n, W = 40, 48, 21, 24
    for H in (1, 24):
        x, h = _rand(B * n, 2 * H * R + H * C, seed=1).to(BF).cuda(), _rand(B * n, W, seed=2).to(BF).cuda()
        w, b = (_rand(2 * H, W, seed=3) * 0.2).to(BF).cuda(), _rand(2 * H, seed=4).cuda() + 1
        m_off = H * ops.scan_state_elems(R, C + 4)

        def run(pool, rows, q_len, at, pick):
            md = _md([q_len] * len(rows), [at] * len(rows), _slots([r + 1 for r in rows]))
            q, k, v = x[pick].split([H * R, H * R, H * C], -1)
            gates = _cu().memory_gates(h[pick], w, b, 6.0, pool, m_off, md)
            return _cu().memory_scan(q, k, v, gates, 0.3, pool, md, H, R, C)[..., :C + 1].reshape(len(rows) * q_len, -1)

        def pool():
            return torch.full((B + 1, m_off + -(-H // 4) * 4), float("nan"), device="cuda")
        everything = torch.arange(B * n).view(B, n)
        whole = pool()
        many = run(whole, range(B), n, 0, everything.flatten()).view(B, n, -1)
        p1 = pool()
        for r in (0, 17, 47):
            _close(run(p1, [r], n, 0, everything[r]), many[r], 2e-5)
        p2 = pool()
        steps = torch.stack([run(p2, range(B), 1, t, everything[:, t]) for t in range(n)], 1)
        _close(steps, many, 2e-5)
        _close(p2[1:, m_off:m_off + H], whole[1:, m_off:m_off + H], 1e-5)
