"""Gizilorn on the device: every kernel it adds or extends against the plain float64 implementation."""
import math
from types import SimpleNamespace

import pytest
import torch

from tests import gizilorn_oracle as go

pytestmark = pytest.mark.gpu
BF, F16, F32 = torch.bfloat16, torch.float16, torch.float32


def _rand(*shape, seed=0, size=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * size


def _close(got, want, tol):
    got, want = got.double().cpu(), want.double().cpu()
    assert torch.isfinite(got).all()
    err = float((got - want).abs().max() / want.abs().max().clamp_min(1e-9))
    assert err < tol, err


def _cu():
    from vllm_b200.ops import cuda_ops
    return cuda_ops()


def _pages(n_seqs, lens, BS=64, seed=0, extra=2):
    """(block table, pages in all): sequences of these lengths on scattered pages."""
    pages = [math.ceil(n / BS) for n in lens]
    total = sum(pages) + 3
    perm = (torch.randperm(total - 1, generator=torch.Generator().manual_seed(seed)) + 1).tolist()
    bt = torch.zeros(n_seqs, max(pages) + extra, dtype=torch.int32)
    for b, n in enumerate(pages):
        for j in range(n):
            bt[b, j] = perm.pop()
    return bt, total


def _md(q_lens, lens, table, vt=False):
    qsl = torch.tensor([0] + torch.tensor(q_lens).cumsum(0).tolist(), dtype=torch.int32, device="cuda")
    return SimpleNamespace(num_reqs=len(q_lens), query_start_loc=qsl, seq_lens=torch.tensor(lens, dtype=torch.int32, device="cuda"),
                           block_table=table.cuda(), max_query_len=max(q_lens), max_seq_len=max(lens), decode_only=max(q_lens) == 1, flat=False,
                           kv_vt=vt, num_splits=0, num_actual_tokens=sum(q_lens))


def _table(base, dims, n):
    a = torch.arange(n, dtype=torch.float64)[:, None] * base ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    return torch.cat((a.cos(), a.sin()), -1).float().cuda()


# ------------------------------------------------------------------------------------------------ streams, activation
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("S", [1, 2, 3, 4, 5, 16])
@pytest.mark.parametrize("T,H", [(1, 50), (7, 96), (4, 2048), (3, 4096), (2, 9000), (130, 1000)])
def test_hyper_step(T, H, S, dtype):
    from vllm_b200 import ops
    x, y = _rand(T, S, H, seed=1, size=3.0) + 1.0, (_rand(T, H + 8, seed=2) + 0.5).to(dtype)
    into, out, mix, w = _rand(S, seed=3), _rand(S, seed=4), _rand(S, S, seed=5), (_rand(H, seed=6, size=0.3) + 1).to(dtype)
    p = {"h.in": into.double(), "h.out": out.double(), "h.mix": mix.double()}
    want = go.hyper(x.double().transpose(0, 1), p, "h.", lambda u: y[:, :H].double())
    u = sum(into[s].double() * want[s] for s in range(S))
    xs = x.cuda()
    h = ops.hyper_step(xs, y.cuda()[:, :H], torch.cat([out, mix.flatten()]).cuda(), into.cuda(), w.cuda(), 1e-3)
    _close(xs.transpose(0, 1), want, 1e-6)                   # the streams are never rounded to 16 bits
    assert h.dtype == dtype
    _close(h, go.rms_norm(u, w.double(), 1e-3), 6e-3 if dtype == BF else 1e-5)
    keep = xs.clone()
    h = ops.hyper_step(xs, None, None, into.cuda(), w.cuda(), 1e-3, dtype)
    assert torch.equal(xs, keep)
    _close(h, go.rms_norm(u, w.double(), 1e-3), 6e-3 if dtype == BF else 1e-5)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,H,S", [(1, 50, 3), (9, 96, 1), (5, 4096, 4), (3, 72, 7)])
def test_hyper_entry(T, H, S, dtype):
    from vllm_b200 import ops
    table, we, w = _rand(33, H, seed=1, size=2.0).to(dtype), (_rand(H, seed=2) + 1).to(dtype), (_rand(H, seed=3) + 1).to(dtype)
    ids = torch.randint(0, 33, (T,), generator=torch.Generator().manual_seed(4), dtype=torch.int32)
    into = _rand(S, seed=5) + 0.5
    e = go.rms_norm(table[ids.long()].double(), we.double(), 1e-3)
    x, h = ops.hyper_entry(ids.cuda(), table.cuda(), S, we.cuda(), into.cuda(), w.cuda(), 1e-3)
    assert x.shape == (T, S, H)
    for s in range(S):
        _close(x[:, s], e, 1e-6)
    _close(h, go.rms_norm(into.double().sum() * e, w.double(), 1e-3), 6e-3 if dtype == BF else 1e-5)
    x, h = ops.hyper_entry(None, table.cuda()[:T], S, None, into.cuda(), w.cuda(), 1e-3)
    _close(x[:, S - 1], table[:T], 1e-9)
    _close(h, go.rms_norm(into.double().sum() * table[:T].double(), w.double(), 1e-3), 6e-3 if dtype == BF else 1e-5)


@pytest.mark.parametrize("dtype", [BF, F16, F32])
@pytest.mark.parametrize("T,n", [(1, 7), (5, 64), (130, 1000), (3, 4096)])
def test_xielu(T, n, dtype):
    from vllm_b200 import ops
    x = _rand(T, n, seed=1, size=4.0).to(dtype)
    x.view(-1)[0], x.view(-1)[-1] = -60.0, 1e-4
    got = ops.xielu(x.cuda(), torch.tensor([0.7, 1.3]).cuda())
    z = x.double()
    want = torch.where(z > 0, 0.7 * z * z, 1.3 * (torch.expm1(z.clamp(max=0)) - z.clamp(max=0))) + z / 2
    _close(got, want, 6e-3 if dtype != F32 else 1e-6)


def test_apertus_runs_the_same_activation():
    from vllm_b200.models.llama_variants import _XIELU
    act = _XIELU(F32)
    act.alpha_p.data.fill_(0.4)
    act.alpha_n.data.fill_(-0.9)
    x = _rand(7, 300, seed=1, size=3.0)
    want = act(x)                                              # its plain operations, on the CPU
    _close(act.cuda()(x.cuda()), want, 1e-6)
    act.beta.data.fill_(0.25)
    act.half = None
    _close(act(x.cuda()), act.cpu()(x), 1e-6)


@pytest.mark.parametrize("dtype", [BF, F16, F32])
@pytest.mark.parametrize("M,N,K", [(1, 320, 192), (7, 4096, 1024), (64, 1000, 2048), (200, 512, 4096), (256, 22, 64), (300, 640, 256), (5, 36, 40)])
def test_projection_with_xielu(M, N, K, dtype):
    """Split over a cluster or not, by our kernel or the library's."""
    from vllm_b200 import ops
    x, w, b = _rand(M, K, seed=1).to(dtype), (_rand(N, K, seed=2) * 2 / math.sqrt(K)).to(dtype), _rand(N, seed=3).to(dtype)
    got = ops.linear_xielu(x.cuda(), w.cuda(), b.cuda(), torch.tensor([0.9, 1.1]).cuda())
    z = x.double() @ w.double().T + b.double()
    want = torch.where(z > 0, 0.9 * z * z, 1.1 * (torch.expm1(z.clamp(max=0)) - z.clamp(max=0))) + z / 2
    _close(got, want, 1.5e-2 if dtype != F32 else 1e-5)


# ------------------------------------------------------------------------------------------------ prologues
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("H,G,D,DV,rot,neox,vt", [(4, 2, 24, 40, 16, True, False), (3, 1, 10, 6, 6, True, False), (8, 2, 128, 128, 64, True, True),
                                                  (8, 2, 128, 128, 128, True, True), (4, 4, 64, 64, 32, True, False),
                                                  (2, 1, 64, 32, 64, False, False), (4, 2, 128, 128, 128, False, True)])
def test_rotated_keys_and_values_reach_the_cache(H, G, D, DV, rot, neox, vt, dtype):
    if vt and dtype == F32:
        pytest.skip("the tensor-core layout is a 16-bit one")
    T, BS, DC = 70, 64, max(D, DV)
    proj = _rand(T, H * D + G * (D + DV) + 24, seed=1).to(dtype)
    x = proj.cuda()
    q, k, v = x[:, :H * D], x[:, H * D + 8:H * D + 8 + G * D], x[:, H * D + 16 + G * D:H * D + 16 + G * (D + DV)]
    pos = torch.arange(900, 900 + T)
    slots = torch.randperm(4 * BS, generator=torch.Generator().manual_seed(2))[:T]
    slots[5] = -1
    cache = torch.full((4, 2, G, BS, DC), 7.0, dtype=dtype).cuda()
    _cu().fused_qk_norm_rope(pos.cuda(), q, k, None, None, _table(3000.0, rot, 1000), D, 0.0, neox, v=v, kv_cache=cache,
                             slot_mapping=slots.cuda(), vt=vt, v_head_dim=DV, keep32=True, v_cos_sin=_table(3000.0, DV, 1000))
    parts = [proj[:, a:a + n].double().view(T, -1, d) for a, n, d in
             ((0, H * D, D), (H * D + 8, G * D, D), (H * D + 16 + G * D, G * DV, DV))]
    wq, wk, wv = [go.turn(t, 3000.0, r, neox, first=900) for t, r in zip(parts, (rot, rot, DV))]
    tol = 6e-3 if dtype == BF else 1e-6
    _close(q.view(T, H, D), wq, tol)
    ck = cache[:, 0]
    cv = cache[:, 1].reshape(4, G, DC, BS).transpose(2, 3) if vt else cache[:, 1]
    for t in range(T):
        s = int(slots[t])
        if s >= 0:
            _close(ck[s // BS, :, s % BS, :D], wk[t], tol)
            _close(cv[s // BS, :, s % BS, :DV], wv[t], tol)
    left = torch.ones(4 * BS, dtype=torch.bool)
    left[slots[slots >= 0]] = False
    assert (ck.transpose(1, 2).reshape(4 * BS, -1)[left.cuda()] == 7.0).all()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("H,D,P,R,neox", [(4, 20, 12, 48, False), (1, 7, 2, 9, False), (8, 128, 64, 512, False), (3, 16, 16, 40, True), (2, 24, 0, 32, False),
                                          (20, 64, 32, 128, True)])
@pytest.mark.parametrize("own", [True, False])
def test_latent_prologue(H, D, P, R, neox, own, dtype):
    from vllm_b200 import ops
    T, BS = 33, 64
    q_off, kv_off = 8, 8 + -(-H * (D + P) // 8) * 8
    proj = _rand(T, kv_off + -(-(R + P) // 8) * 8, seed=1, size=2.0).to(dtype)
    w = (_rand(R, seed=2, size=0.3) + 1).to(dtype)
    pos = torch.randint(0, 500, (T,), generator=torch.Generator().manual_seed(3))
    slots = torch.randperm(2 * BS, generator=torch.Generator().manual_seed(4))[:T]
    slots[3] = -1
    cache = torch.full((2, BS, R + P), 7.0, dtype=dtype).cuda()
    x = proj.cuda()
    ops.latent_rope_cache(x, q_off, H, D, P, kv_off, R if own else 0, w.cuda() if own else None, 1e-3, pos.cuda(),
                          _table(700.0, P, 500) if P else None, neox, cache if own else None, slots.cuda() if own else None)

    def turned(t):
        return torch.cat([go.turn(t[i:i + 1], 700.0, P, neox, first=int(pos[i])) for i in range(T)]) if P else t
    tol = 6e-3 if dtype == BF else 2e-6
    q = proj[:, q_off:q_off + H * (D + P)].double().view(T, H, D + P)
    got = x[:, q_off:q_off + H * (D + P)].reshape(T, H, D + P)
    assert torch.equal(got[..., :D].cpu(), proj[:, q_off:q_off + H * (D + P)].view(T, H, D + P)[..., :D])
    if P:
        _close(got[..., D:], turned(q[..., D:]), tol)
    if not own:
        return
    c = go.rms_norm(proj[:, kv_off:kv_off + R].double(), w.double(), 1e-3)
    kr = turned(proj[:, kv_off + R:kv_off + R + P].double()[:, None])[:, 0]
    rows = cache.view(2 * BS, R + P)
    ok = slots >= 0
    _close(rows[slots[ok].cuda()], torch.cat([c, kr], 1)[ok], tol)
    left = torch.ones(2 * BS, dtype=torch.bool)
    left[slots[ok]] = False
    assert (rows[left.cuda()] == 7.0).all()


# ------------------------------------------------------------------------------------------------ attention with mixed heads
def _talk_case(H, G, D, DV, lens, q_lens, window, cap, scale, dtype, vt, seed=0, turned=False, size=1.0):
    """Runs ops.talking_attention on paged random keys; returns (got, want) per sequence."""
    from vllm_b200 import ops
    bt, total = _pages(len(lens), lens, seed=seed)
    DC = max(D, DV)
    cache = torch.zeros(total, 2, G, 64, DC, dtype=dtype)
    q_all, want = [], []
    talk = _rand(H, H, seed=seed + 1) / math.sqrt(H) + 0.5 * torch.eye(H)
    sinks = torch.zeros(H)
    for b, (n, ql) in enumerate(zip(lens, q_lens)):
        q, k, v = [_rand(n, h, d, seed=seed + 10 * b + i + 2, size=s).to(dtype) for i, (h, d, s) in
                   enumerate(((H, D, size), (G, D, 1.0), (G, DV, 1.0)))]
        for j in range(n):
            blk = int(bt[b, j // 64])
            cache[blk, 0, :, j % 64, :D] = k[j]
            if vt:
                cache[blk, 1].view(G, DV, 64)[:, :, j % 64] = v[j]
            else:
                cache[blk, 1, :, j % 64, :DV] = v[j]
        o = go.talking_attention(q.double(), k.double(), v.double(), scale, cap, window, talk.double())
        want.append((go.turn(o, 40.0, DV, True, back=True) if turned else o)[n - ql:])
        q_all.append(q[n - ql:])
    md = _md(q_lens, lens, bt, vt)
    pos = torch.cat([torch.arange(n - ql, n) for n, ql in zip(lens, q_lens)]).cuda()
    rope = SimpleNamespace(cos_sin_cache=_table(40.0, DV, max(lens)), is_neox_style=True) if turned else None
    x = torch.cat(q_all)
    buf = torch.zeros(x.shape[0], H * D + 16, dtype=dtype)
    buf[:, 8:8 + H * D] = x.view(-1, H * D)
    got = ops.talking_attention(buf.cuda()[:, 8:8 + H * D].unflatten(1, (H, D)), cache.cuda(), md, scale, window, cap, talk.cuda(), sinks.cuda(), DV,
                                rope, pos)
    _cu().check_kernel_error(torch.device("cuda", 0))
    return got, torch.cat(want)


SHAPES = [(6, 2, 24, 40), (3, 1, 10, 6), (4, 4, 64, 64), (2, 1, 200, 300), (8, 2, 128, 128), (12, 3, 48, 32)]


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("H,G,D,DV", SHAPES)
@pytest.mark.parametrize("turned", [True, False])
def test_mixed_heads_of_every_shape(H, G, D, DV, turned, dtype):
    lens, q_lens = [1, 64, 65, 150, 333], [1, 64, 3, 1, 70]
    for w, cap in ((40, 3.0), (1000, 80.0)):
        got, want = _talk_case(H, G, D, DV, lens, q_lens, w, cap, 2.0 / math.sqrt(D), dtype, False, seed=H, turned=turned)
        _close(got, want, 1.5e-2 if dtype == BF else 1e-5)
    got, want = _talk_case(H, G, D, DV, lens, [1] * 5, 100, 3.0, 2.0 / math.sqrt(D), dtype, False, seed=D, turned=turned)
    _close(got, want, 1.5e-2 if dtype == BF else 1e-5)


# heads per KV head of 1, 2, 4, 8, 16, 32; odd and even numbers of value heads; more heads than the decode kernel takes
TC = [(8, 8), (8, 4), (16, 4), (32, 8), (8, 1), (16, 1), (24, 3), (32, 4), (32, 2), (32, 1), (4, 1), (12, 3), (40, 5), (64, 8), (1, 1)]


@pytest.mark.parametrize("H,G", TC)
@pytest.mark.parametrize("window", [100, 700])
def test_prompts_on_the_tensor_cores(H, G, window):
    lens, q_lens = [300, 64, 65, 129, 1, 517], [300, 64, 3, 1, 1, 200]
    got, want = _talk_case(H, G, 128, 128, lens, q_lens, window, 20.0, 0.1, BF, True, seed=H, turned=True)
    _close(got, want, 1.5e-2)


@pytest.mark.parametrize("H,G", TC)
@pytest.mark.parametrize("window", [1, 100, 128, 700])
def test_decode_on_the_tensor_cores(H, G, window):
    lens = [1, 2, 63, 64, 65, 128, 129, 300, 517]
    got, want = _talk_case(H, G, 128, 128, lens, [1] * len(lens), window, 20.0, 0.1, BF, True, seed=G, turned=True)
    _close(got, want, 1.5e-2)


@pytest.mark.parametrize("cap,scale,size", [(0.5, 0.1, 1.0), (5.0, 0.5, 3.0), (60.0, 0.3, 4.0), (50.0, 0.02, 1.0), (60.0, 3.0, 8.0)])
def test_scores_far_below_and_far_above_the_cap(cap, scale, size):
    for lens, q_lens in (([200, 90], [200, 90]), ([200, 90, 1], [1, 1, 1])):
        got, want = _talk_case(8, 2, 128, 128, lens, q_lens, 120, cap, scale, BF, True, seed=3, size=size)
        _close(got, want, 2e-2)


def test_value_heads_in_several_passes(monkeypatch):
    """A batch whose unmixed outputs exceed the buffer is done some value heads at a time."""
    monkeypatch.setattr(_cu(), "TALK_BYTES", 1 << 18)
    for G, vt, dtype in ((5, True, BF), (3, False, F32)):
        got, want = _talk_case(4 * G, G, 128, 128, [130, 70], [130, 70], 90, 10.0, 0.1, dtype, vt, seed=5, turned=True)
        _close(got, want, 1.5e-2 if dtype == BF else 1e-5)


def test_splits_of_the_keys_add_up(monkeypatch):
    for splits in (1, 2, 3, 16):
        monkeypatch.setattr(_cu(), "talk_splits", lambda *a: splits)
        got, want = _talk_case(16, 4, 128, 128, [1, 130, 900], [1, 1, 1], 600, 30.0, 0.1, BF, True, seed=6)
        _close(got, want, 1.5e-2)


# ------------------------------------------------------------------------------------------------ latents with a rotated part and a window
def _latents(lens, W, dtype, seed=0):
    bt, total = _pages(len(lens), lens, seed=seed)
    cache = torch.full((total, 64, W), 3.0, dtype=dtype)
    rows = []
    for b, n in enumerate(lens):
        c = _rand(n, W, seed=seed + 31 * b + 1).to(dtype)
        for j in range(n):
            cache[bt[b, j // 64], j % 64] = c[j]
        rows.append(c)
    return cache.cuda(), bt.cuda(), rows


def _latent_attention(q, c, R, first, scale, window):
    """q [n, H, R + P] at positions first.., rows c [m, R + P]: float64 [n, H, R]."""
    s = torch.einsum("qhr,kr->hqk", q.double(), c.double()) * scale
    at, kp = torch.arange(first, first + q.shape[0])[:, None], torch.arange(c.shape[0])[None]
    ok = (kp <= at) & (at - kp < window)
    return torch.einsum("hqk,kr->qhr", s.masked_fill(~ok, -math.inf).softmax(-1), c[:, :R].double())


@pytest.mark.parametrize("R,P", [(8, 8), (48, 16), (64, 64), (128, 32), (136, 24), (264, 40), (400, 8), (512, 64), (512, 32)])
@pytest.mark.parametrize("H", [1, 6, 16, 20, 40])
def test_latent_decode_with_a_rotated_part_and_a_window(R, P, H):
    lens = [1, 63, 64, 65, 200, 700]
    cache, bt, rows = _latents(lens, R + P, BF, seed=R + H)
    q = _rand(len(lens), H, R + P, seed=5, size=2.0).to(BF)
    scale, sl = 1.0 / math.sqrt(R + P), torch.tensor(lens, dtype=torch.int32).cuda()
    qn = q[..., :R].transpose(0, 1).contiguous().cuda().transpose(0, 1)              # head-major, as the layer hands it over
    full = q.cuda()
    for window in (1, 64, 65, 300, 5000):
        for splits in (0, 3):
            out = _cu().mla_decode_tc(qn, full[..., R:], cache, bt, sl, scale, max(lens), splits, sliding_window=window)
            for b, c in enumerate(rows):
                _close(out[b:b + 1], _latent_attention(q[b:b + 1], c, R, len(c) - 1, scale, window), 2e-2)
    _cu().check_kernel_error(torch.device("cuda", 0))


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("R,P,H", [(9, 2, 3), (48, 12, 4), (512, 64, 5)])
def test_generic_latent_attention_with_a_window(R, P, H, dtype):
    lens, q_lens = [1, 40, 64, 129, 300], [1, 2, 64, 1, 37]
    cache, bt, rows = _latents(lens, R + P, dtype, seed=R)
    qsl = torch.tensor([0] + q_lens).cumsum(0).int()
    q = _rand(int(qsl[-1]), H, R + P, seed=6, size=2.0).to(dtype)
    scale = 1.0 / math.sqrt(R + P)
    for window in (1, 33, 100, 1000):
        out = _cu().mla_simt(q[..., :R].cuda(), q[..., R:].cuda(), cache, bt, torch.tensor(lens, dtype=torch.int32).cuda(), qsl.cuda(), scale, window)
        for b, c in enumerate(rows):
            s, e = int(qsl[b]), int(qsl[b + 1])
            _close(out[s:e], _latent_attention(q[s:e], c, R, len(c) - q_lens[b], scale, window), 2e-5 if dtype == F32 else 1e-2)


@pytest.mark.parametrize("dim,rot,vdim,H", [(64, 32, 64, 2), (24, 8, 40, 3), (128, 64, 128, 4), (8, 64, 128, 1), (128, 16, 8, 2), (72, 40, 104, 5)])
@pytest.mark.parametrize("dtype", [BF, F16])
def test_latent_prompts_with_a_rotated_part_and_a_window(dim, rot, vdim, H, dtype):
    lens, q_lens = [17, 128, 129, 400, 700, 256], [17, 128, 20, 300, 130, 129]
    qsl = [0] + torch.tensor(q_lens).cumsum(0).tolist()
    kv_rank = 32
    q = _rand(qsl[-1], H, dim + rot, seed=7, size=2.0).to(dtype)
    scale = (dim + rot) ** -0.5

    def dev(x):
        return torch.tensor(x, dtype=torch.int32).cuda()
    for window in (0, 1, 50, 128, 333, 5000):
        first = [max(0, n - ql + 1 - window) if window else 0 for n, ql in zip(lens, q_lens)]      # keys before it are not gathered
        kv = [n - f for n, f in zip(lens, first)]
        start = [0] + torch.tensor(kv).cumsum(0).tolist()
        ks, vs, rs = [_rand(sum(lens), *s, seed=8 + i).to(dtype) for i, s in enumerate(((H, dim), (H, vdim), (kv_rank + rot,)))]
        at = [0] + torch.tensor(lens).cumsum(0).tolist()
        keep = torch.cat([torch.arange(a + f, a + n) for a, f, n in zip(at, first, lens)])
        out = torch.full((qsl[-1], H, vdim), 5.0, dtype=dtype).cuda()
        rows = rs[keep].cuda()
        _cu().mla_prefill(q.cuda(), ks[keep].cuda(), vs[keep].cuda(), out, dev(qsl[:-1]), dev(q_lens), dev(kv), dev(start), 0, max(q_lens), scale,
                          rows[:, kv_rank:], window)
        for b, (n, ql) in enumerate(zip(lens, q_lens)):
            s = slice(qsl[b], qsl[b] + ql)
            k, v, r = ks[at[b]:at[b + 1]].double(), vs[at[b]:at[b + 1]].double(), rs[at[b]:at[b + 1], kv_rank:].double()
            sc = (torch.einsum("qhd,khd->hqk", q[s, :, :dim].double(), k) + torch.einsum("qhr,kr->hqk", q[s, :, dim:].double(), r)) * scale
            pos, kp = torch.arange(n - ql, n)[:, None], torch.arange(n)[None]
            ok = (kp <= pos) & ((pos - kp < window) if window else True)
            _close(out[s], torch.einsum("hqk,khd->qhd", sc.masked_fill(~ok, -math.inf).softmax(-1), v), 1.5e-2)
    _cu().check_kernel_error(torch.device("cuda", 0))
