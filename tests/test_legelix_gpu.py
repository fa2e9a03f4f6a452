"""Legelix on the device: every kernel it adds or extends against the plain float64 implementation."""
from types import SimpleNamespace

import pytest
import torch

from tests import legelix_oracle as lo

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


# ------------------------------------------------------------------------------------------------ stream
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,H", [(1, 50), (7, 96), (4, 2048), (2, 9000), (130, 1000)])
@pytest.mark.parametrize("bias,nxt", [(True, True), (False, False)])
def test_norm_add(T, H, dtype, bias, nxt):
    from vllm_b200 import ops
    x, y = _rand(T, H, seed=1, size=4.0) + 1.5, (_rand(T, H, seed=2) + 0.7).to(dtype)
    w, b, w2, b2 = [(_rand(H, seed=s, size=0.3) + c).to(dtype) for s, c in ((3, 1.0), (4, 0.0), (5, 1.0), (6, 0.0))]
    yb = _rand(H, seed=7) if bias else None
    yd = y.double() + (yb.double() if bias else 0)
    want = x.double() + 0.4 * lo.layer_norm(yd, w.double(), b.double(), 1e-3)
    xs = x.cuda()
    out = ops.norm_add(xs, y.cuda(), yb.cuda() if bias else None, (w.cuda(), b.cuda()), 0.4, (w2.cuda(), b2.cuda()) if nxt else None, 1e-3)
    _close(xs, want, 2e-6)                                   # the stream itself is never rounded to 16 bits
    assert out.dtype == dtype
    _close(out, lo.layer_norm(want, w2.double(), b2.double(), 1e-3) if nxt else want, 6e-3 if dtype == BF else 3e-6)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,H", [(3, 50), (33, 1024)])
def test_embed_norm(T, H, dtype):
    from vllm_b200 import ops
    table, ids = _rand(70, H, seed=1).to(dtype), torch.randint(0, 70, (T,))
    w, b = (_rand(H, seed=2, size=0.3) + 1).to(dtype), _rand(H, seed=3, size=0.3).to(dtype)
    x, h = ops.embed_norm(ids.int().cuda(), table.cuda(), (w.cuda(), b.cuda()), 1e-5)
    _close(x, table.double()[ids], 1e-7)
    _close(h, lo.layer_norm(table.double()[ids], w.double(), b.double(), 1e-5), 6e-3 if dtype == BF else 3e-6)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("groups,W,first,shared", [(3, 20, True, False), (8, 128, False, True), (1, 2048, True, False), (2, 700, True, False),
                                                   (5, 7, False, True), (1, 6000, True, False)])
def test_gated_norm(groups, W, first, shared, dtype):
    from vllm_b200 import ops
    T, n = 5, groups * W
    y, buf = _rand(T, n, seed=1, size=2.0), _rand(T, n + 24, seed=2).to(dtype).cuda()
    z, w = buf[:, 8:8 + n], (_rand(W if shared else n, seed=3, size=0.3) + 1).to(dtype)
    zd, wd = z.double().cpu(), w.double().repeat(n // w.numel())
    g = lo.silu(zd)
    want = lo.unit_rms((y.double() * (g if first else 1)).view(T, groups, W), 1e-4).view(T, n) * wd * (1 if first else g) * 1.7
    out = torch.zeros(T, n + 16, dtype=dtype, device="cuda")
    ops.gated_norm(y.cuda(), z, w.cuda(), groups, 1e-4, first, out[:, 16:], 1.7)
    _close(out[:, 16:], want, 8e-3 if dtype == BF else 3e-6)
    assert not out[:, :16].any()


# ------------------------------------------------------------------------------------------------ recurrences
# (tokens of each request in successive steps; 0: left out)
STEPS = [([5, 1, 40], [1, 0, 1], [1, 1, 1], [3, 17, 2]), ([70, 0, 1], [33, 2, 16]), ([1, 1, 1], [1, 1, 1])]


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
def test_short_conv_over_steps(taps, dtype):
    C, rows = 70, [3, 1, 4]
    w, b = _rand(C, taps, seed=1, size=0.6).to(dtype), _rand(C, seed=2, size=0.2).to(dtype)
    for steps in STEPS:
        pool = torch.full((6, C * (taps - 1) + 5), float("nan"), device="cuda")
        x = [_rand(sum(s[i] for s in steps), C, seed=10 + i).to(dtype) for i in range(3)]
        got, at = [[], [], []], [0, 0, 0]
        for s in steps:
            live = [i for i in range(3) if s[i]]
            md = _md([s[i] for i in live], [at[i] for i in live], _slots([rows[i] for i in live]))
            wide = torch.zeros(sum(s), C + 10, dtype=dtype)
            wide[:, 4:4 + C] = torch.cat([x[i][at[i]:at[i] + s[i]] for i in live])
            out = _cu().causal_conv1d(wide.cuda()[:, 4:4 + C], w.cuda(), b.cuda(), pool, md)
            for i, part in zip(live, out.split([s[i] for i in live])):
                got[i].append(part)
                at[i] += s[i]
        for i in range(3):
            _close(torch.cat(got[i]), lo.silu(lo.short_conv(x[i].double(), w.double(), b.double())), 2e-6)
        assert pool[[0, 2, 5]].isnan().all() and pool[:, C * (taps - 1):].isnan().all()


@pytest.mark.parametrize("H,P,N,G", [(3, 16, 16, 1), (4, 40, 24, 2), (6, 64, 128, 2), (2, 5, 10, 1), (2, 128, 256, 1), (2, 12, 300, 2), (1, 1, 1, 1)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_ssd_scan_over_steps(H, P, N, G, dtype):
    from vllm_b200 import ops
    rows, off = [3, 1, 4], 8
    A_log, D, dtb = _rand(H, seed=1, size=0.5), _rand(H, seed=2), _rand(H, seed=3, size=0.5)
    width = H * P + 2 * G * N
    for steps in STEPS:
        pool = torch.full((6, off + H * ops.scan_state_elems(N, P)), float("nan"), device="cuda")
        n = [sum(s[i] for s in steps) for i in range(3)]
        x = [_rand(n[i], width, seed=10 + i) for i in range(3)]
        dt = [_rand(n[i], H, seed=20 + i).to(dtype) for i in range(3)]
        got, at = [[], [], []], [0, 0, 0]
        for s in steps:
            live = [i for i in range(3) if s[i]]
            md = _md([s[i] for i in live], [at[i] for i in live], _slots([rows[i] for i in live]))
            xs = torch.cat([x[i][at[i]:at[i] + s[i]] for i in live])
            wide = torch.zeros(sum(s), H + 3, dtype=dtype)
            wide[:, 1:1 + H] = torch.cat([dt[i][at[i]:at[i] + s[i]] for i in live])
            y = _cu().ssd_scan(xs.cuda(), wide.cuda()[:, 1:1 + H], dtb.cuda(), A_log.cuda(), D.cuda(), pool, off, md, H, P, G, N)
            for i, part in zip(live, y.split([s[i] for i in live])):
                got[i].append(part)
                at[i] += s[i]
        for i in range(3):
            xx, B, C = x[i].double().split([H * P, G * N, G * N], -1)
            step = torch.nn.functional.softplus(dt[i].double() + dtb.double(), threshold=1e9)
            want, _ = lo.ssd(xx.reshape(n[i], H, P), B.reshape(n[i], G, N), C.reshape(n[i], G, N), step, A_log.double(), D.double())
            _close(torch.cat(got[i]), want.reshape(n[i], H * P), 5e-6)
        assert pool[[0, 2, 5]].isnan().all()


@pytest.mark.parametrize("H,d,dv,rank", [(3, 16, 16, 4), (2, 20, 36, 8), (4, 64, 64, 16), (2, 6, 5, 3), (2, 128, 128, 16), (1, 200, 96, 16), (1, 1, 1, 1)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_gla_scan_over_steps(H, d, dv, rank, dtype):
    from vllm_b200 import ops
    rows = [3, 1, 4]
    a2, a2b = _rand(H * d, rank, seed=1).to(dtype), _rand(H * d, seed=2).to(dtype)
    sizes = [H * d, H * d, H * dv, rank]
    tau = 5.0
    for steps in STEPS:
        pool = torch.full((6, H * ops.scan_state_elems(d, dv)), float("nan"), device="cuda")
        n = [sum(s[i] for s in steps) for i in range(3)]
        x = [_rand(n[i], sum(sizes) + 8, seed=10 + i).to(dtype) for i in range(3)]
        got, at = [[], [], []], [0, 0, 0]
        for s in steps:
            live = [i for i in range(3) if s[i]]
            md = _md([s[i] for i in live], [at[i] for i in live], _slots([rows[i] for i in live]))
            xs = torch.cat([x[i][at[i]:at[i] + s[i]] for i in live]).cuda()
            q, k, v, a1, _ = xs.split(sizes + [8], -1)
            o = _cu().gla_scan(q, k, v, a1, a2.cuda(), a2b.cuda(), tau, d ** -0.5, pool, md, H, d, dv)
            for i, part in zip(live, o.split([s[i] for i in live])):
                got[i].append(part)
                at[i] += s[i]
        for i in range(3):
            q, k, v, a1, _ = x[i].double().split(sizes + [8], -1)
            z = (a1 @ a2.double().T + a2b.double()).view(n[i], H, d)
            want, _ = lo.gated_scan(q.reshape(n[i], H, d) * d ** -0.5, k.reshape(n[i], H, d), v.reshape(n[i], H, dv),
                                    torch.sigmoid(z) ** (1 / tau))
            _close(torch.cat(got[i]), want.reshape(n[i], H * dv), 5e-6)
        assert pool[[0, 2, 5]].isnan().all()


@pytest.mark.parametrize("R", [12, 32, 60, 128, 200])
@pytest.mark.parametrize("ssd", [True, False])
def test_scan_forms_agree(R, ssd):
    """Lanes hold few or many rows depending on how much runs at once: sequences alone, all together and token by token."""
    from vllm_b200 import ops
    C, dtype, B, n = 40, BF, 48, 21
    for H in (1, 24):
        width = H * C + 2 * R if ssd else 2 * H * R + H * C + 4
        x = _rand(B * n, width, seed=1).to(F32 if ssd else dtype).cuda()
        dt, A, D, tb = _rand(B * n, H, seed=2).cuda(), _rand(H, seed=3).cuda(), _rand(H, seed=4).cuda(), _rand(H, seed=5).cuda()
        a2, a2b = _rand(H * R, 4, seed=6).to(dtype).cuda(), (_rand(H * R, seed=7) + 2).to(dtype).cuda()

        def run(pool, rows, q_len, at, pick):
            md = _md([q_len] * len(rows), [at] * len(rows), _slots([r + 1 for r in rows]))
            if ssd:
                return _cu().ssd_scan(x[pick], dt[pick], tb, A, D, pool, 0, md, H, C, 1, R)
            q, k, v, a1 = x[pick].split([H * R, H * R, H * C, 4], -1)
            return _cu().gla_scan(q, k, v, a1, a2, a2b, 8.0, 0.3, pool, md, H, R, C)

        def pool():
            return torch.full((B + 1, H * ops.scan_state_elems(R, C)), float("nan"), device="cuda")
        everything = torch.arange(B * n).view(B, n)
        many = run(pool(), range(B), n, 0, everything.flatten()).view(B, n, H * C)
        one = run(pool(), [7], n, 0, everything[7])
        _close(one, many[7], 3e-6)
        p = pool()
        first = run(p, range(B), n - 3, 0, everything[:, :n - 3].flatten()).view(B, n - 3, H * C)      # and decode from there
        rest = [run(p, range(B), 1, n - 3 + j, everything[:, n - 3 + j]) for j in range(3)]
        _close(torch.cat([first, torch.stack(rest, 1)], 1), many, 3e-6)


# ------------------------------------------------------------------------------------------------ attention
def _paged(k, v, lens, page, vt):
    """Scatter per-request keys [n, G, D] and values [n, G, DV] over shuffled pages: (cache, block table)."""
    G, D, DV = k[0].shape[1], k[0].shape[2], v[0].shape[2]
    W = max(D, DV)
    need = [-(-n // page) for n in lens]
    order = torch.randperm(sum(need), generator=torch.Generator().manual_seed(5)) + 1
    cache = torch.full((sum(need) + 1, 2, G, page, W), 3.0, dtype=k[0].dtype)       # stale, finite
    table = torch.zeros(len(lens), max(need) + 1, dtype=torch.int32)
    at = 0
    for i, n in enumerate(lens):
        for j in range(need[i]):
            b = int(order[at])
            at += 1
            table[i, j] = b
            kk, vv = k[i][j * page:(j + 1) * page], v[i][j * page:(j + 1) * page]
            cache[b, 0, :, :kk.shape[0], :D] = kk.transpose(0, 1)
            cache[b, 1, :, :vv.shape[0], :DV] = vv.transpose(0, 1)
    if vt:
        cache[:, 1] = cache[:, 1].transpose(-1, -2).contiguous().view(cache[:, 1].shape)
    return cache.cuda(), table.cuda()


SHAPES = [(6, 2, 48, 48), (4, 4, 16, 40), (5, 1, 40, 16), (3, 3, 7, 9), (8, 2, 128, 128), (12, 4, 80, 80), (2, 1, 192, 160), (6, 2, 128, 128), (8, 2, 64, 64), (4, 4, 32, 32),
          (6, 2, 64, 64)]


@pytest.mark.parametrize("H,G,D,DV", SHAPES)
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("sinks,factor", [(True, 0.6), (False, 0.6), (True, 1.0)])
def test_chunk_local_attention(H, G, D, DV, dtype, sinks, factor):
    """Portions that start anywhere, chunks of several sizes, one-token steps, pages in any order."""
    from vllm_b200 import ops
    vt = dtype == BF and _cu().tc_attention_ok(D, DV, H // G)
    scale = 1.3 * D ** -0.5
    for size, q_lens, ctx in ((50, [9, 70, 1, 2], [41, 0, 49, 50]), (64, [1, 1, 1, 1], [63, 64, 0, 200]), (1000, [200, 3], [3, 130]),
                              (1, [4, 1], [0, 9]), (130, [1, 1], [259, 260]), (200, [150], [120])):
        lens = [c + q for c, q in zip(ctx, q_lens)]
        q = [(_rand(n, H, D, seed=10 + i) * 1.5).to(dtype) for i, n in enumerate(lens)]
        k = [_rand(n, G, D, seed=20 + i).to(dtype) for i, n in enumerate(lens)]
        v = [_rand(n, G, DV, seed=30 + i).to(dtype) for i, n in enumerate(lens)]
        sink = _rand(H, seed=40) + 1.0 if sinks else None
        cache, table = _paged(k, v, lens, 64, vt)
        md = _md(q_lens, ctx, table, vt)
        wide = torch.zeros(sum(q_lens), H * D + 16, dtype=dtype, device="cuda")
        wide[:, 8:8 + H * D] = torch.cat([x[c:] for x, c in zip(q, ctx)]).reshape(-1, H * D).cuda()
        buf = torch.zeros(sum(q_lens), H * DV + 24, dtype=dtype, device="cuda")
        ops.paged_attention(wide[:, 8:8 + H * D].view(-1, H, D), cache, md, scale, out=buf[:, 8:8 + H * DV].view(-1, H, DV),
                            sinks=None if sink is None else sink.cuda(), chunk_size=size, v_head_size=DV, out_scale=factor)
        want = torch.cat([lo.attend(a.double(), b.double(), c.double(), scale, size, None if sink is None else sink.double())[n:]
                          for a, b, c, n in zip(q, k, v, ctx)]) * factor
        _close(buf[:, 8:8 + H * DV], want, 2e-2 if dtype == BF else 5e-6)
        assert not buf[:, :8].any() and not buf[:, 8 + H * DV:].any()


@pytest.mark.parametrize("window,cap,causal", [(None, 0.0, True), (37, 0.0, True), (None, 8.0, True), (None, 0.0, False), (21, 0.0, False)])
def test_generic_attention_masks(window, cap, causal):
    """The generic kernel's other features, against the framework's plain op."""
    from vllm_b200 import ops
    from vllm_b200.ops import ref
    H, G, D = 6, 2, 40
    q_lens, ctx = [33, 1, 5], [10, 80, 0]
    lens = [c + q for c, q in zip(ctx, q_lens)]
    k, v = [_rand(n, G, D, seed=20 + i) for i, n in enumerate(lens)], [_rand(n, G, D, seed=30 + i) for i, n in enumerate(lens)]
    cache, table = _paged(k, v, lens, 32, False)
    md = _md(q_lens, ctx, table)
    q, slopes = _rand(sum(q_lens), H, D, seed=1).cuda(), _rand(H, seed=2).abs().cuda() * 0.1
    got, lse = ops.paged_attention(q, cache, md, 0.2, window, cap, causal, alibi_slopes=slopes, return_lse=True)
    want, lse_w = ref.paged_attention(q, cache, table, md.seq_lens, md.query_start_loc, 0.2, causal=causal, sliding_window=window,
                                      logits_soft_cap=cap, alibi_slopes=slopes, return_lse=True)
    _close(got, want, 1e-5)
    _close(lse, lse_w, 1e-5)


@pytest.mark.parametrize("H,G,D,DV,rot", [(6, 2, 48, 48, 48), (4, 4, 16, 40, 8), (5, 1, 40, 16, 40), (3, 3, 7, 9, 2), (8, 2, 128, 128, 128),
                                          (8, 2, 128, 128, 64), (4, 2, 64, 64, 32)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_norm_rotate_and_cache(H, G, D, DV, rot, dtype):
    from vllm_b200.layers.rotary import get_rope
    T, page = 7, 64
    spec = dict(base=9000.0, dims=rot, scaling=dict(factor=3.0, low=1.0, high=4.0, original=512))
    with torch.device("cuda"):
        rope = get_rope(D, rot, 700, 9000.0, False, dict(rope_type="llama3", factor=3.0, low_freq_factor=1.0, high_freq_factor=4.0,
                                                        original_max_position_embeddings=512))
    pos = torch.tensor([0, 1, 5, 63, 64, 300, 699])
    sizes = [H * D, G * D, G * DV]
    offs = [0, (H * D + 7) // 8 * 8]
    offs.append(offs[1] + (G * D + 7) // 8 * 8)
    x = torch.zeros(T, offs[2] + sizes[2] + 8)
    x = (x + _rand(*x.shape, seed=1)).to(dtype)
    q, k, v = [x.cuda()[:, o:o + n] for o, n in zip(offs, sizes)]
    qw, kw = [(_rand(D, seed=s, size=0.3) + 1).to(dtype) for s in (2, 3)]
    vt = dtype == BF and _cu().tc_attention_ok(D, DV, H // G)
    cache = torch.zeros(5, 2, G, page, max(D, DV), dtype=dtype, device="cuda")
    slots = torch.tensor([64, 130, -1, 200, 255, 319, 90], device="cuda")
    _cu().fused_qk_norm_rope(pos.cuda(), q, k, qw.cuda(), kw.cuda(), rope.cos_sin_cache, D, 1e-4, False, v=v, kv_cache=cache,
                             slot_mapping=slots, vt=vt, v_head_dim=DV, keep32=True)
    f = lo.frequencies(spec)

    def want(part, n, w):
        y = lo.unit_rms(part.double().view(T, n, D), 1e-4) * w.double()
        full = torch.zeros(700, n, D, dtype=F64)
        full[pos] = y
        return lo.rotate(full, f)[pos]
    tol = 6e-3 if dtype == BF else 3e-5
    wq, wk = [want(x[:, o:o + n], h, w) for o, n, h, w in zip(offs, sizes, (H, G), (qw, kw))]
    _close(q.reshape(T, H, D), wq, tol)
    flat_k = cache[:, 0].transpose(1, 2).reshape(-1, G, max(D, DV))
    vals = cache[:, 1]
    flat_v = (vals.reshape(5, G, DV, page).permute(0, 3, 1, 2) if vt else vals.transpose(1, 2)).reshape(5 * page, G, -1)
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            _close(flat_k[s][:, :D], wk[t], tol)
            _close(flat_v[s][:, :DV], x[t, offs[2]:offs[2] + sizes[2]].view(G, DV), 1e-9)
    used = {s for s in slots.tolist() if s >= 0}
    assert not flat_k[[s for s in range(5 * page) if s not in used]].any()
