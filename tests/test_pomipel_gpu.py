"""Pomipel on the device: every kernel against the plain float64 implementation, then whole models through the engine."""
import math

import pytest
import torch

from tests import pomipel_oracle as po

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


@pytest.fixture(autouse=True)
def _no_kernel_gave_up():
    yield
    from vllm_b200.ops import cuda_ops
    cuda_ops().check_kernel_error(torch.device("cuda", torch.cuda.current_device()))


# ------------------------------------------------------------------------------------------------ stream kernels
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,H", [(1, 50), (5, 96), (33, 1024), (3, 5000)])
def test_embed_stream(T, H, dtype):
    from vllm_b200 import ops
    V, P = 77, 40
    table, pos = _rand(V, H, seed=1).to(dtype), _rand(P, H, seed=2).to(dtype)
    ids, where = torch.randint(0, V, (T,)), torch.randint(0, P, (T,))
    x, h = ops.embed_stream(ids.int().cuda(), where.cuda(), table.cuda(), pos.cuda(), 2.75)
    want = table.double()[ids] * 2.75 + pos.double()[where]
    assert x.dtype == F32 and h.dtype == dtype
    _close(x, want, 1e-6)
    _close(h, want, 5e-3 if dtype == BF else 1e-6)
    x, _ = ops.embed_stream(ids.int().cuda(), where.cuda(), table.cuda(), None, 2.75)
    _close(x, table.double()[ids] * 2.75, 1e-6)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,H", [(1, 50), (7, 96), (4, 2048), (2, 9000), (130, 1000)])
@pytest.mark.parametrize("with_next", [False, True])
def test_post_norm_add(T, H, dtype, with_next):
    from vllm_b200 import ops
    x, y = _rand(T, H, seed=3, size=4.0), _rand(T, H, seed=4).to(dtype)
    w, wn = _rand(H, seed=5, size=0.3).to(dtype), _rand(H, seed=6, size=0.3).to(dtype)
    want = x.double() + po.centred_norm(y.double(), w.double(), 1e-5)
    xs = x.cuda()
    out = ops.post_norm_add(xs, y.cuda(), w.cuda(), 1e-5, True, wn.cuda() if with_next else None, True)
    _close(xs, want, 2e-6)                                   # the stream itself is never rounded to 16 bits
    assert out.dtype == dtype
    _close(out, po.centred_norm(want, wn.double(), 1e-5) if with_next else want, 6e-3 if dtype == BF else 3e-6)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,q_rank,kv_rank", [(1, 14, 18), (5, 40, 48), (67, 384, 512), (3, 1536, 0), (2, 24, 136)])
def test_latent_norm_cache(T, q_rank, kv_rank, dtype):
    from vllm_b200 import ops
    lat = _rand(T, q_rank + kv_rank, seed=7).to(dtype)
    gq, gk = (1 + _rand(q_rank, seed=8, size=0.2)).to(dtype), (1 + _rand(max(kv_rank, 1), seed=9, size=0.2)).to(dtype)
    cache = torch.full((9, 16, max(kv_rank, 1)), 7.0, dtype=dtype)
    slots = torch.randperm(9 * 16)[:T]
    if T > 2:
        slots[1] = -1                                          # a padding row leaves the cache alone
    dev = cache.cuda()
    cq, _ = ops.latent_norm_cache(lat.cuda(), q_rank, gq.cuda(), kv_rank, gk.cuda() if kv_rank else None, 1e-5,
                                  dev if kv_rank else None, slots.cuda() if kv_rank else None)
    tol = 6e-3 if dtype == BF else 3e-6
    _close(cq, po.unit_rms(lat[:, :q_rank].double(), 1e-5) * gq.double(), tol)
    if kv_rank:
        want = cache.double().view(-1, kv_rank)
        ckv = po.unit_rms(lat[:, q_rank:].double(), 1e-5) * gk.double()
        for t in range(T):
            if slots[t] >= 0:
                want[slots[t]] = ckv[t]
        _close(dev.view(-1, kv_rank), want, tol)


# ------------------------------------------------------------------------------------------------ router and experts
@pytest.mark.parametrize("T", [1, 3, 64, 300])                # 300: logits from the large-batch product
@pytest.mark.parametrize("H,E,top,count,keep", [(50, 6, 3, 2, 1), (96, 8, 2, 4, 2), (64, 12, 5, 3, 2), (128, 64, 6, 8, 3),
                                                 (40, 5, 2, 5, 4), (256, 160, 8, 1, 1), (72, 40, 36, 4, 4)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_router(T, H, E, top, count, keep, dtype):
    from vllm_b200 import ops
    x, w = _rand(T, H, seed=10), (_rand(E, H, seed=11) / math.sqrt(H)).to(dtype)
    if T > 256 and dtype == BF:
        x = x.to(BF).float()                                   # the product reads the 16-bit copy
    corr = _rand(E, seed=12, size=0.8) - 0.6                   # most choice scores are negative
    wt, ids = ops.router_topk(x.cuda(), w.cuda(), top, count, keep, False, "sigmoid", corr.cuda(), 1.0, x.to(dtype).cuda())
    for t in range(T):
        want = po.route(x[t].double(), w.double(), corr.double(), top, count, keep)
        choice = torch.sigmoid(w.double() @ x[t].double()) + corr.double()
        got = dict(zip(ids[t].tolist(), wt[t].tolist()))
        assert len(got) == top
        if set(got) != {e for e, _ in want}:                   # only a tie within rounding may differ
            a = sorted(float(choice[e]) for e in got)
            b = sorted(float(choice[e]) for e, _ in want)
            assert max(abs(p - q) for p, q in zip(a, b)) < 1e-5
            continue
        for e, s in want:
            assert abs(got[e] - s) < 1e-5                      # the score without the correction


@pytest.mark.parametrize("scoring,bias,renorm", [("softmax", False, True), ("softmax", True, False), ("sigmoid", True, True)])
def test_grouped_topk_options_match_reference(scoring, bias, renorm):
    from vllm_b200.ops import cuda_ops, ref
    lg, b = _rand(37, 48, seed=13), _rand(48, seed=14, size=0.1) if bias else None
    w0, i0 = ref.grouped_topk(lg, 5, 6, 3, renorm, scoring, b, 2.5)
    w1, i1 = cuda_ops().grouped_topk(lg.cuda(), 5, 6, 3, renorm, scoring, None if b is None else b.cuda(), 2.5)
    assert torch.equal(i0.sort(-1).values, i1.cpu().sort(-1).values)
    _close(w1.cpu().sort(-1).values, w0.sort(-1).values, 1e-5)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,H,ff,E,top", [(1, 64, 24, 4, 1), (5, 96, 40, 8, 2), (3, 50, 11, 5, 3), (64, 128, 136, 16, 6),
                                          (700, 96, 72, 12, 5), (2100, 64, 64, 3, 2)])
def test_experts_and_their_norm(T, H, ff, E, top, dtype):
    from vllm_b200 import ops
    x = _rand(T, H, seed=15).to(dtype)
    up = (_rand(E, ff, H, seed=16) / math.sqrt(H)).to(dtype)
    down = (_rand(E, H, ff, seed=17) / math.sqrt(ff)).to(dtype)
    ids = torch.stack([torch.randperm(E, generator=torch.Generator().manual_seed(t))[:top] for t in range(T)]).int()
    if T > 4:
        ids[:, 0] = torch.where((ids == 0).any(-1), ids[:, 0], torch.zeros_like(ids[:, 0]))     # one expert gets most rows
    wt = torch.rand(T, top, generator=torch.Generator().manual_seed(18))
    xd, upd, dnd = x.double(), up.double(), down.double()
    want = torch.zeros(T, H, dtype=F64)
    for e in range(E):
        tok, slot = (ids == e).nonzero(as_tuple=True)
        if len(tok):
            want[tok] += wt[tok, slot, None].double() * (torch.clamp(xd[tok] @ upd[e].T, min=0) ** 2 @ dnd[e].T)
    got = ops.fused_moe(x.cuda(), up.cuda(), down.cuda(), wt.cuda(), ids.cuda(), "relu2", None, gated=False)
    _close(got, want, 2e-2 if dtype == BF else 1e-5)
    stream, nw = _rand(T, H, seed=19), _rand(H, seed=20, size=0.2).to(dtype)
    xs = stream.cuda()
    ops.fused_moe_post_norm(xs, x.cuda(), up.cuda(), down.cuda(), wt.cuda(), ids.cuda(), "relu2", None, nw.cuda(), 1e-5, True)
    _close(xs, stream.double() + po.centred_norm(want, nw.double(), 1e-5), 2e-2 if dtype == BF else 1e-5)


# ------------------------------------------------------------------------------------------------ attention kernels
def _paged(seqs, R, dtype, BS=64, seed=0):
    """Latents of sequences of the given lengths on scattered pages."""
    pages = [math.ceil(n / BS) for n in seqs]
    total = sum(pages) + 3
    perm = torch.randperm(total - 1, generator=torch.Generator().manual_seed(seed)) + 1
    cache = torch.full((total, BS, R), 3.0, dtype=dtype)
    bt = torch.zeros(len(seqs), max(pages) + 2, dtype=torch.int32)
    lats, at = [], 0
    for b, n in enumerate(seqs):
        c = _rand(n, R, seed=seed + 31 * b + 1).to(dtype)
        for j in range(pages[b]):
            bt[b, j] = perm[at]
            part = c[j * BS:(j + 1) * BS]
            cache[perm[at], :len(part)] = part
            at += 1
        lats.append(c)
    return cache.cuda(), bt.cuda(), lats


def _latent_attention(q, c, first, scale):
    """q [n, H, R] at positions first.., latents c: float64."""
    s = torch.einsum("qhr,kr->hqk", q.double(), c.double()) * scale
    vis = torch.arange(c.shape[0])[None, :] <= torch.arange(first, first + q.shape[0])[:, None]
    return torch.einsum("hqk,kr->qhr", s.masked_fill(~vis, -math.inf).softmax(-1), c.double())


@pytest.mark.parametrize("R", [8, 48, 64, 72, 128, 136, 192, 264, 320, 400, 448, 512])
@pytest.mark.parametrize("H", [1, 4, 16, 20, 40])
def test_mla_decode_any_width(R, H):
    from vllm_b200.ops import cuda_ops
    seqs = [1, 63, 64, 65, 200, 700]
    cache, bt, lats = _paged(seqs, R, BF, seed=R + H)
    q = _rand(H, len(seqs), R, seed=5, size=2.0).to(BF).cuda().transpose(0, 1)       # head-major, as the layer hands it over
    scale = 1.0 / math.sqrt(R)
    sl = torch.tensor(seqs, dtype=torch.int32).cuda()
    for splits in (1, 3):
        out = cuda_ops().mla_decode_tc(q, None, cache, bt, sl, scale, max(seqs), splits)
        for b, c in enumerate(lats):
            _close(out[b:b + 1], _latent_attention(q[b:b + 1].cpu(), c, len(c) - 1, scale), 2e-2)


@pytest.mark.parametrize("dtype", [BF, F32, torch.float16])
@pytest.mark.parametrize("R,H,BS", [(18, 3, 64), (64, 4, 32), (130, 9, 64), (512, 16, 64), (1000, 2, 16)])
def test_mla_simt(R, H, BS, dtype):
    from vllm_b200.ops import cuda_ops
    seqs, lens = [1, 40, 64, 129, 300], [1, 2, 64, 1, 37]
    cache, bt, lats = _paged(seqs, R, dtype, BS, seed=R)
    qsl = torch.tensor([0] + lens).cumsum(0).int()
    q = _rand(int(qsl[-1]), H, R, seed=6, size=2.0).to(dtype)
    scale = 1.0 / math.sqrt(R)
    out = cuda_ops().mla_simt(q.cuda(), None, cache, bt, torch.tensor(seqs, dtype=torch.int32).cuda(), qsl.cuda(), scale)
    for b, c in enumerate(lats):
        s, e = int(qsl[b]), int(qsl[b + 1])
        _close(out[s:e], _latent_attention(q[s:e], c, len(c) - lens[b], scale), 2e-5 if dtype == F32 else 1e-2)


@pytest.mark.parametrize("dim,vdim,H", [(64, 64, 2), (24, 40, 3), (128, 128, 4), (8, 128, 1), (128, 8, 2), (72, 104, 5)])
@pytest.mark.parametrize("dtype", [BF, torch.float16])
def test_mla_prefill(dim, vdim, H, dtype):
    from vllm_b200.ops import cuda_ops
    seqs, lens = [17, 128, 129, 400, 700, 256], [17, 128, 20, 300, 130, 129]
    gap = 3                                                    # rows between the portions belong to other requests
    q_start, at = [], 0
    for n in lens:
        q_start.append(at)
        at += n + gap
    kv_start = [0] + torch.tensor(seqs).cumsum(0).tolist()
    q = _rand(at, H, dim, seed=7, size=2.0).to(dtype)
    k, v = _rand(kv_start[-1], H, dim, seed=8).to(dtype), _rand(kv_start[-1], H, vdim, seed=9).to(dtype)
    out = torch.full((at, H, vdim), 5.0, dtype=dtype).cuda()
    dev = lambda x: torch.tensor(x, dtype=torch.int32).cuda()  # noqa: E731
    scale = dim ** -0.5
    args = (dev(q_start), dev(lens), dev(seqs), dev(kv_start))
    cut = max(1, H // 2)                                       # two launches with half of the heads each
    for h0, h1 in ((0, cut), (cut, H)):
        if h1 > h0:
            cuda_ops().mla_prefill(q.cuda(), k[:, h0:h1].contiguous().cuda(), v[:, h0:h1].contiguous().cuda(), out, *args, h0,
                                   max(lens), scale)
    for b in range(len(seqs)):
        s, n, k0, m = q_start[b], lens[b], kv_start[b], seqs[b]
        att = torch.einsum("qhd,khd->hqk", q[s:s + n].double(), k[k0:k0 + m].double()) * scale
        vis = torch.arange(m)[None, :] <= torch.arange(m - n, m)[:, None]
        want = torch.einsum("hqk,khd->qhd", att.masked_fill(~vis, -math.inf).softmax(-1), v[k0:k0 + m].double())
        _close(out[s:s + n], want, 1.5e-2)
        assert (out[s + n:s + n + gap] == 5.0).all()           # nothing is written outside the portions
