"""Launch each hot kernel a few times so that `ncu --set full -k regex:<name> -s 3 -c 1` can capture it in isolation.

    ncu --set full --clock-control none -k regex:gemm_fp8_kernel -s 3 -c 1 -o ncu_fp8 \
        python scripts/ncu_targets.py fp8
"""
import sys

import torch

sys.path.insert(0, ".")
from vllm_b200.ops import cuda as cu  # noqa: E402
from vllm_b200.ops import ref  # noqa: E402

which = sys.argv[1] if len(sys.argv) > 1 else "all"
torch.manual_seed(0)
dt = torch.bfloat16


def rep(fn, n=5):
    for _ in range(n):
        fn()
    torch.cuda.synchronize()


if which in ("fp8", "all"):
    M, N, K = 64, 7168, 16384
    x = torch.randn(M, K, device="cuda", dtype=dt) * 0.1
    wq, ws = ref.block_quant_weight_fp8(torch.randn(N, K, device="cuda") * 0.02, 128)
    xq, xs = cu.per_token_group_quant_fp8(x, 128, col_major=True)
    ws = ws.contiguous()
    rep(lambda: cu.gemm_fp8_block(xq, xs, wq, ws))
if which in ("gemm", "all"):
    x = torch.randn(64, 4096, device="cuda", dtype=dt) * 0.1
    for N, K in ((6144, 4096), (28672, 4096), (4096, 14336)):
        w = torch.randn(N, K, device="cuda", dtype=dt) * 0.02
        xx = torch.randn(64, K, device="cuda", dtype=dt) * 0.1
        rep(lambda: cu.gemm_tc(xx, w))
if which in ("attn", "mla", "all"):
    from vllm_b200.benchmarks.kernels import _mk_paged
    from vllm_b200.forward_context import AttentionMetadata
    B, BS, ctx = 64, 64, 1040
    if which in ("attn", "all"):
        Hq, Hkv, D = 32, 8, 128
        NB, bt, sl = _mk_paged(B, Hkv, D, BS, ctx)
        cache = (torch.randn(NB, 2, Hkv, BS, D, device="cuda") * 0.3).to(dt)
        q = (torch.randn(B, Hq, D, device="cuda") * 0.3).to(dt)
        md = AttentionMetadata(num_reqs=B, num_actual_tokens=B, max_query_len=1, max_seq_len=ctx,
                               query_start_loc=torch.arange(B + 1, dtype=torch.int32, device="cuda"), seq_lens=sl,
                               block_table=bt, slot_mapping=torch.empty(0), decode_only=True)
        md.kv_vt = True
        rep(lambda: cu.paged_attention(q, cache, md, D ** -0.5))
    if which in ("mla", "all"):
        NB, bt, sl = _mk_paged(B, 1, 576, BS, 4096)
        cache = (torch.randn(NB, BS, 576, device="cuda") * 0.3).to(dt)
        qn = (torch.randn(B, 16, 512, device="cuda") * 0.3).to(dt)
        qp = (torch.randn(B, 16, 64, device="cuda") * 0.3).to(dt)
        rep(lambda: cu.mla_decode_tc(qn, qp, cache, bt, sl, 0.07, 4096))
if which in ("latent", "all"):
    # latent attention and ungated experts: prompt attention, decode over the latents, grouped products of a prompt step
    from vllm_b200.benchmarks.latent_layers import _pages, _routing
    from vllm_b200.ops import moe
    n, ctx, h, D = 4, 1024, 16, 128
    i32 = dict(dtype=torch.int32, device="cuda")
    q, k, v = (torch.randn(n * ctx, h, D, device="cuda", dtype=dt) * 0.3 for _ in range(3))
    out = torch.empty_like(q)
    start, lens = torch.arange(0, n * ctx, ctx, **i32), torch.full((n,), ctx, **i32)
    rep(lambda: cu.mla_prefill(q, k, v, out, start, lens, lens, start, 0, ctx, D ** -0.5))
    cache, bt, sl = _pages(64, 4096, 512)
    qa = torch.randn(64, 16, 512, device="cuda", dtype=dt) * 0.3
    rep(lambda: cu.mla_decode_tc(qa, None, cache, bt, sl, 0.07, 4096))
    x = torch.randn(4096, 2048, device="cuda", dtype=dt) * 0.1
    up, down = (torch.randn(*s, device="cuda", dtype=dt) * 0.02 for s in ((32, 1408, 2048), (32, 2048, 1408)))
    wt, ids = _routing(4096, 32, 6)
    rep(lambda: moe.expert_rows_plain(x, up, down, ids, "relu2", None))
if which in ("scan", "all"):
    # Legelix: scans of prompts (1024 tokens each) and of a decode batch, at the sizes of a 2048-wide model
    from vllm_b200.forward_context import AttentionMetadata
    from vllm_b200.ops import scan_state_elems
    MH, GH, i32 = 64, 8, dict(dtype=torch.int32, device="cuda")
    for n, q in ((4, 1024), (64, 1)):
        T = n * q
        md = AttentionMetadata(num_reqs=n, num_actual_tokens=T, max_query_len=q, max_seq_len=q, query_start_loc=torch.arange(0, T + 1, q, **i32),
                               seq_lens=torch.full((n,), q + (q == 1), **i32), block_table=(torch.arange(n, **i32) + 1).view(-1, 1),
                               slot_mapping=None, decode_only=q == 1)
        xa, dts = torch.randn(T, MH * 64 + 256, device="cuda") * 0.3, torch.randn(T, MH, device="cuda").to(dt)
        A, D, b = [torch.randn(MH, device="cuda") * 0.3 for _ in range(3)]
        pool = torch.zeros(n + 1, MH * scan_state_elems(128, 64), device="cuda")
        rep(lambda: cu.ssd_scan(xa, dts, b, A, D, pool, 0, md, MH, 64, 1, 128))
        x = (torch.randn(T, GH * (128 + 128 + 256) + 16, device="cuda") * 0.3).to(dt)
        qq, kk, vv, a1 = x.split([GH * 128, GH * 128, GH * 256, 16], -1)
        a2, a2b = torch.randn(GH * 128, 16, device="cuda").to(dt), torch.randn(GH * 128, device="cuda").to(dt)
        pool2 = torch.zeros(n + 1, GH * scan_state_elems(128, 256), device="cuda")
        rep(lambda: cu.gla_scan(qq, kk, vv, a1, a2, a2b, 16.0, 0.09, pool2, md, GH, 128, 256))
if which in ("memory", "all"):
    # Kopadra: gates, scan and norm of a matrix memory (prompts of 1024 tokens each, a decode batch), experts of a prompt step with
    # identity experts and the step that combines them, at the sizes of a 2048-wide model
    from vllm_b200.forward_context import AttentionMetadata
    from vllm_b200.ops import moe, scan_state_elems
    MH, R, C, W, i32 = 8, 128, 256, 2048, dict(dtype=torch.int32, device="cuda")
    m_off = MH * scan_state_elems(R, C + 4)
    for n, q in ((4, 1024), (64, 1)):
        T = n * q
        md = AttentionMetadata(num_reqs=n, num_actual_tokens=T, max_query_len=q, max_seq_len=q, query_start_loc=torch.arange(0, T + 1, q, **i32),
                               seq_lens=torch.full((n,), q + (q == 1), **i32), block_table=(torch.arange(n, **i32) + 1).view(-1, 1),
                               slot_mapping=None, decode_only=q == 1)
        h, w, b = (torch.randn(T, W, device="cuda") * 0.3).to(dt), (torch.randn(2 * MH, W, device="cuda") * 0.02).to(dt), torch.randn(2 * MH, device="cuda")
        x, nw = (torch.randn(T, MH * (2 * R + 2 * C), device="cuda") * 0.3).to(dt), torch.ones(MH * C, device="cuda", dtype=dt)
        qq, kk, vv, gg = x.split([MH * R, MH * R, MH * C, MH * C], -1)
        pool3 = torch.zeros(n + 1, m_off + MH, device="cuda")
        rep(lambda: cu.gated_norm(cu.memory_scan(qq, kk, vv, cu.memory_gates(h, w, b, 15.0, pool3, m_off, md), 0.09, pool3, md, MH, R, C),
                                  gg, nw, MH, 1e-6, False, gate="sigmoid",
                                  gates=cu.memory_gates(h, w, b, 15.0, pool3, m_off, md)))
    x = torch.randn(4096, W, device="cuda", dtype=dt) * 0.1
    w13, w2 = (torch.randn(*s, device="cuda", dtype=dt) * 0.02 for s in ((48, 2 * 768, W), (48, W, 768)))
    ids = torch.rand(4096, 64, device="cuda").topk(8, -1).indices.int()
    pw, emap = torch.rand(4096, 8, device="cuda"), torch.cat([torch.arange(48, **i32), torch.full((16,), -1, **i32)])
    stream, nw = torch.zeros(4096, W, device="cuda"), torch.ones(W, device="cuda", dtype=dt)

    def experts():
        rows, inv = moe.expert_rows_gated(x, w13, w2, ids, "silu", emap)
        cu.add_norm(stream, x, (nw, None), 1e-6, dt, rows, inv, pw, ids, 48, x)
    rep(experts)
if which in ("talk", "all"):
    # Gizilorn: attention with mixed heads (prompts, a decode batch), streams, latent attention with a rotated part and a window, at the
    # sizes of a 2048-wide model
    from vllm_b200.benchmarks.latent_layers import _pages
    from vllm_b200.forward_context import AttentionMetadata
    H, G, D, W, i32 = 16, 4, 128, 2048, dict(dtype=torch.int32, device="cuda")
    talk, sinks = torch.randn(H, H, device="cuda") * 0.2, torch.zeros(H, device="cuda")
    for n, q, seq, window in ((2, 4096, 4096, 2048), (64, 1, 4096, 4096)):
        per = seq // 64
        kv = (torch.randn(n * per + 1, 2, G, 64, D, device="cuda") * 0.3).to(dt)
        md = AttentionMetadata(num_reqs=n, num_actual_tokens=n * q, max_query_len=q, max_seq_len=seq,
                               query_start_loc=torch.arange(0, n * q + 1, q, **i32), seq_lens=torch.full((n,), seq, **i32),
                               block_table=(torch.randperm(n * per, device="cuda").int() + 1).view(n, per), slot_mapping=None, kv_vt=True,
                               decode_only=q == 1)
        x = torch.randn(n * q, H, D, device="cuda").to(dt)
        rep(lambda: cu.talking_attention(x, kv, md, D ** -0.5, window, 50.0, talk, sinks, D))
        del kv
    xs, y, w = torch.randn(8192, 4, W, device="cuda"), torch.randn(8192, W, device="cuda").to(dt), torch.ones(W, device="cuda", dtype=dt)
    coef, into = torch.randn(20, device="cuda") * 0.3, torch.ones(4, device="cuda")
    rep(lambda: cu.hyper_step(xs, y, coef, into, w, 1e-6, dt))
    cache, bt, sl = _pages(64, 4096, 576)
    qn, qp = (torch.randn(64, H, m, device="cuda") * 0.3 for m in (512, 64))
    qn, qp = qn.to(dt), qp.to(dt)
    rep(lambda: cu.mla_decode_tc(qn, qp, cache, bt, sl, 0.07, 4096, sliding_window=2048))
    q, k, v = ((torch.randn(8192, H, m, device="cuda") * 0.3).to(dt) for m in (192, 128, 128))
    lat, out = (torch.randn(8192, 576, device="cuda") * 0.3).to(dt), torch.empty(8192, H, 128, device="cuda", dtype=dt)
    start, lens = torch.arange(0, 8192, 4096, **i32), torch.full((2,), 4096, **i32)
    rep(lambda: cu.mla_prefill(q, k, v, out, start, lens, lens, start, 0, 4096, 0.07, lat[:, 512:], 2048))
