"""Kopadra beside the closest model of the framework at equal sizes: Qwen3-Next (gated full attention and a gated delta rule in turn,
experts with a shared one in every layer).  Prefill and decode throughput of a few layers through the engine, and every kernel
against its roofline next to the like kernel.

    python bench.py --design kopadra [--design-part model|kernels|all] [--design-sizes 1k,2k,4k] [--steps K]

Method and roofline as in ``benchmarks/latent_layers.py``.  A scan's FLOPs are those of the recurrence (six per element of the
state and token) over the tensor-core rate, although it runs on the CUDA cores.
"""
from __future__ import annotations

import json

import torch

from vllm_b200.benchmarks.kernels import timeit
from vllm_b200.benchmarks.latent_layers import BF, LAYERS, MAX_LEN, VOCAB, _peaks, bench_model

# (width, query heads, kv heads, memory heads, expert width, experts, top, groups, kept groups, shared width); head sizes below
SIZES = {"1k": (1024, 8, 2, 4, 512, 16, 4, 4, 2, 512), "2k": (2048, 16, 4, 8, 768, 64, 8, 8, 4, 768),
         "4k": (4096, 32, 8, 16, 1536, 64, 8, 8, 4, 1536)}
HEAD, ROT, MEM_K, MEM_V = 128, 64, 128, 256


def configs(size: str) -> dict[str, dict]:
    from vllm_b200.config.model import kopadra_config
    W, H, G, MH, ff, E, k, groups, keep, sh = SIZES[size]

    def own(layers, experts, identity):
        c = kopadra_config(vocab=VOCAB, width=W, heads=H, kv_heads=G, dim=HEAD, mem_heads=MH, mem_dim=MEM_K, mem_vdim=MEM_V, ff=sh,
                           expert_ff=ff, experts=experts, identity=identity, top=k, groups=groups, keep=keep, shared_ff=sh, layers=layers,
                           max_position_embeddings=MAX_LEN, torch_dtype="bfloat16")
        for l in c["layers"]:
            if "rot" in l["mixer"]:
                l["mixer"]["rot"]["dims"] = ROT
        return c
    like = dict(architectures=["Qwen3NextForCausalLM"], model_type="qwen3_next", vocab_size=VOCAB, hidden_size=W, intermediate_size=sh,
                num_hidden_layers=LAYERS, num_attention_heads=H, num_key_value_heads=G, head_dim=HEAD, linear_num_value_heads=MH,
                linear_num_key_heads=MH, linear_key_head_dim=MEM_K, linear_value_head_dim=MEM_V, linear_conv_kernel_dim=4,
                full_attention_interval=2, layer_types=["linear_attention", "full_attention"] * (LAYERS // 2), num_experts=E,
                num_experts_per_tok=k, moe_intermediate_size=ff, shared_expert_intermediate_size=sh, decoder_sparse_step=1,
                norm_topk_prob=True, mlp_only_layers=[], rms_norm_eps=1e-6, hidden_act="silu", max_position_embeddings=MAX_LEN,
                attention_bias=False, rope_parameters=dict(rope_type="default", rope_theta=10000.0, partial_rotary_factor=ROT / HEAD),
                partial_rotary_factor=ROT / HEAD, torch_dtype="bfloat16", tie_word_embeddings=False)
    return {"kopadra": own(["mlstm+moe", "attention+moe"] * (LAYERS // 2), E, 0),
            "kopadra, a quarter identity experts, shared keys": own(["mlstm+moe", "attention+moe", "mlstm+moe", "reuse+moe"], E * 3 // 4, E // 4),
            "qwen3-next layers": like}


def bench_kernels(size: str = "2k", batch: int = 64, prompts: int = 8, ctx: int = 1024) -> list[dict]:
    """Rows: operation, time and roofline fraction of this design's kernel and of the like kernel."""
    from vllm_b200 import ops
    from vllm_b200.forward_context import AttentionMetadata
    from vllm_b200.ops import cuda as cu
    from vllm_b200.ops import moe as moe_ops
    from vllm_b200.ops import scan_state_elems
    W, H, G, MH, ff, E, k, groups, keep, sh = SIZES[size]
    bw, fl = _peaks()
    rows: list[dict] = []
    i32 = dict(dtype=torch.int32, device="cuda")

    def rnd(*shape, s=0.3, dtype=BF):
        return (torch.randn(*shape, device="cuda") * s).to(dtype)

    def row(op, own, own_bytes, own_flops, like_name=None, like=None, like_bytes=0, like_flops=0):
        t = timeit(own)
        best = max(own_bytes / bw, own_flops / fl) * 1e6
        r = {"op": op, "us": t, "of_roofline": best / t}
        if like is not None:
            tl = timeit(like)
            bl = max(like_bytes / bw, like_flops / fl) * 1e6
            r.update(like=like_name, like_us=tl, like_of_roofline=bl / tl, farther_by=(bl / tl) / (best / t))
        rows.append(r)

    qk, vv = MH * MEM_K, MH * MEM_V
    cols = MEM_V + 4
    m_off = MH * scan_state_elems(MEM_K, cols)
    for n_req, q_len in ((batch, 1), (prompts, ctx), (1, prompts * ctx)):
        T = n_req * q_len
        name = f"{T} tokens" + ("" if q_len == 1 else f" in {n_req} prompt{'s' if n_req > 1 else ''}")
        start = ctx if q_len == 1 else 0
        slots = (torch.arange(n_req, **i32) + 1).view(-1, 1).contiguous()
        md = AttentionMetadata(num_reqs=n_req, num_actual_tokens=T, max_query_len=q_len, max_seq_len=start + q_len,
                               query_start_loc=torch.arange(0, T + 1, q_len, **i32), seq_lens=torch.full((n_req,), start + q_len, **i32),
                               block_table=slots, slot_mapping=None, decode_only=q_len == 1)
        # ---- matrix memory
        pool = torch.zeros(n_req + 1, m_off + -(-MH // 4) * 4, device="cuda")
        h, gw, gb = rnd(T, W), rnd(2 * MH, W), rnd(2 * MH, dtype=torch.float32)
        # (whole prompts: one product with 32-bit results, then the gates)
        row(f"memory gates, {name}", lambda: cu.memory_gates(h, gw, gb, 15.0, pool, m_off, md), T * W * 2 + T * MH * 16 + 2 * MH * W * 2,
            4.0 * T * MH * W, "router logits and scores", lambda: cu.router_topk(h, gw, 1, 1, 1, False, "softmax"),
            T * W * 2 + T * 8 + 2 * MH * W * 2, 4.0 * T * MH * W)
        x = rnd(T, 2 * qk + 2 * vv)
        q, kk, v, g = x.split([qk, qk, vv, vv], -1)
        gates = cu.memory_gates(h, gw, gb, 15.0, pool, m_off, md)
        q32, k32, v32 = [rnd(T, MH, d, dtype=torch.float32) for d in (MEM_K, MEM_K, MEM_V)]
        dec, beta = -torch.rand(T, MH, device="cuda"), torch.rand(T, MH, device="cuda")
        st_bytes = n_req * MH * MEM_K * MEM_V * 4 * (2 if start else 1)
        own_bytes = T * ((2 * qk + vv) * 2 + MH * 16 + vv * 4) + st_bytes
        row(f"memory scan, {name}", lambda: cu.memory_scan(q, kk, v, gates, 0.09, pool, md, MH, MEM_K, MEM_V), own_bytes,
            6.0 * T * MH * MEM_K * MEM_V, "gated delta rule scan", lambda: cu.gdn_scan(q32, k32, v32, dec, beta, pool, 0, md),
            T * (2 * qk + 2 * vv) * 4 + st_bytes, 8.0 * T * MH * MEM_K * MEM_V)
        a1, a2, a2b = rnd(T, 16), rnd(qk, 16), rnd(qk)
        row(f"memory scan, {name} (again)", lambda: cu.memory_scan(q, kk, v, gates, 0.09, pool, md, MH, MEM_K, MEM_V), own_bytes,
            6.0 * T * MH * MEM_K * MEM_V, "gated-linear scan with its decays (legelix)",
            lambda: cu.gla_scan(q, kk, v, a1, a2, a2b, 16.0, 0.09, pool, md, MH, MEM_K, MEM_V),
            T * ((2 * qk + vv + 16) * 2 + vv * 4) + st_bytes, 6.0 * T * MH * MEM_K * MEM_V)
        o, nw = cu.memory_scan(q, kk, v, gates, 0.09, pool, md, MH, MEM_K, MEM_V), rnd(vv)
        y, hw = rnd(T, vv, dtype=torch.float32), rnd(MEM_V)
        row(f"divide, head norm, gate, {name}", lambda: cu.gated_norm(o, g, nw, MH, 1e-6, False, gate="sigmoid", gates=gates),
            T * vv * 8 + T * MH * 16, 0, "head norm, then gate (legelix)", lambda: cu.gated_norm(y, g, hw, MH, 1e-6, False), T * vv * 8, 0)
        del pool, x, q, kk, v, g, q32, k32, v32, o, y
        # ---- attention prologue and gate
        sizes = [H * HEAD, G * HEAD, G * HEAD, H * HEAD]
        x = rnd(T, sum(sizes))
        q, kk, v, g = x.split(sizes, -1)
        cs, pos = rnd(MAX_LEN, ROT, dtype=torch.float32), torch.arange(T, device="cuda") % ctx
        cache, where = rnd(T // 64 + 2, 2, G, 64, HEAD), torch.arange(T, device="cuda")
        qw, kw, hn = rnd(H * HEAD), rnd(G * HEAD), rnd(HEAD)
        nb = 2 * T * (H + 2 * G) * HEAD * 2
        kw_ = dict(v=v, kv_cache=cache, slot_mapping=where, vt=True)
        row(f"whole norms, rotation, cache write, {name}",
            lambda: cu.fused_qk_norm_rope(pos, q, kk, qw, kw, cs, HEAD, 1e-6, True, whole=True, **kw_), nb, 0,
            "head norms, rotation, cache write (qwen3-next)", lambda: cu.fused_qk_norm_rope(pos, q, kk, hn, hn, cs, HEAD, 1e-6, True, **kw_), nb, 0)
        a = rnd(T, H * HEAD)
        gu = rnd(T, 2 * H * HEAD)
        row(f"attention gate, {name}", lambda: cu.sigmoid_mul_(a, g), T * H * HEAD * 6, 0, "silu(gate) * up", lambda: cu.act_and_mul(gu, "silu"),
            T * H * HEAD * 6, 0)
        del x, q, kk, v, g, cache, a, gu
        # ---- router, experts, combine
        if n_req > 1:
            real, ident = E * 3 // 4, E // 4
            rw, corr = rnd(E, W, s=0.05), rnd(E, dtype=torch.float32, s=0.02)
            lg = rnd(T, E)
            row(f"router, {name}", lambda: cu.router_topk(h, rw, k, groups, keep, True, "softmax", corr, 1.0, group_score="max"),
                T * W * 2 + E * W * 2, 2.0 * T * E * W, "router product and top-k (qwen3-next)",
                lambda: cu.topk_softmax(ops.linear(h, rw), k, True), T * W * 2 + E * W * 2, 2.0 * T * E * W)
            del lg
            w13, w2 = rnd(E, 2 * ff, W, s=0.02), rnd(E, W, ff, s=0.02)
            ids = torch.rand(T, E, device="cuda").topk(k, -1).indices.int()
            pw = torch.rand(T, k, device="cuda")
            wb, flops = E * 3 * ff * W * 2, 6.0 * T * k * ff * W
            nb = wb + T * W * 2 + T * k * W * 2
            row(f"experts, {name}", lambda: moe_ops.expert_rows_gated(h, w13, w2, ids, "silu", None), nb, flops, "experts (qwen3-next)",
                lambda: cu.fused_moe(h, w13, w2, pw, ids, "silu"), nb, flops)
            emap = torch.cat([torch.arange(real, **i32), torch.full((ident,), -1, **i32)])
            erows, inv = moe_ops.expert_rows_gated(h, w13[:real], w2[:real], ids, "silu", emap)
            stream, res, n1 = rnd(T, W, dtype=torch.float32), rnd(T, W, dtype=torch.float32), rnd(W)
            shared = rnd(T, W)
            live = int((inv >= 0).sum())
            row(f"combine, identities, shared expert, norm, {name}",
                lambda: cu.add_norm(stream, shared, (n1, None), 1e-6, BF, erows, inv, pw, ids, real, h), live * W * 2 + T * W * 14, 0,
                "combine, norm, residual (pomipel)", lambda: cu.post_norm_add(res, erows, n1, 1e-6, True, None, False, inv, pw),
                live * W * 2 + T * W * 10, 0)
            del w13, w2, erows, stream, res, shared
        # ---- stream
        stream, y, res, n1 = rnd(T, W, dtype=torch.float32), rnd(T, W), rnd(T, W), rnd(W)
        row(f"residual, layer norm, {name}", lambda: cu.add_norm(stream, y, (n1, None), 1e-6), T * W * 12, 0, "residual + norm (16-bit stream)",
            lambda: cu.fused_add_rms_norm(y, res, n1, 1e-6), T * W * 8, 0)
        del stream, y, res, h
    lg = rnd(batch, VOCAB)
    row(f"logit cap, {batch} x {VOCAB}", lambda: cu.soft_cap_(lg, 30.0), batch * VOCAB * 4, 0, "silu(gate) * up",
        lambda: cu.act_and_mul(lg, "silu"), batch * VOCAB * 3, 0)
    return rows


def run(part: str = "all", sizes=None, steps: int = 20) -> dict:
    out: dict = {"design": "kopadra", "layers": LAYERS, "dtype": "bf16", "models": [], "kernels": []}
    if part in ("all", "model"):
        for s in sizes or SIZES:
            for name, cfg in configs(s).items():
                r = bench_model(name, cfg, steps=steps)
                out["models"].append({"size": s, **r})
                print(json.dumps(out["models"][-1]), flush=True)
    if part in ("all", "kernels"):
        for s in sizes or ("2k",):
            for r in bench_kernels(s):
                out["kernels"].append({"size": s, **r})
                print(json.dumps(out["kernels"][-1]), flush=True)
    return out
