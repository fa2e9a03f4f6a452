"""Pomipel beside the closest model of the framework (DeepSeek-V3: latent attention with a rotated part, gated experts) at
equal sizes: prefill and decode throughput of a few layers through the engine, and every kernel against its roofline next
to the like kernel of that model.

    python bench.py --design pomipel [--design-part model|kernels|all] [--steps K]

Random weights and token ids.  Model numbers: CUDA events around K replays of the captured decode step, and around whole
prompt steps.  Kernel numbers: median of calls with the L2 flushed before each (benchmarks/kernels.py).  Roofline of an
operation = the larger of its bytes over the measured copy bandwidth and its FLOPs over the measured bf16 rate.
"""
from __future__ import annotations

import json
import math
import os
import statistics
import tempfile

import torch

from vllm_b200.benchmarks.kernels import timeit

BF = torch.bfloat16
# layers that resemble a real model's: (width, heads, q_rank, kv_rank, expert width, experts, top, groups, kept groups)
SIZES = {"1k": (1024, 16, 384, 512, 512, 16, 4, 4, 2), "2k": (2048, 16, 1024, 512, 1408, 64, 6, 8, 3),
         "4k": (4096, 32, 1536, 512, 1536, 64, 8, 8, 4)}
HEAD_DIM, ROPE_DIM, VOCAB, LAYERS, MAX_LEN = 128, 64, 32000, 4, 2048


def _peaks() -> tuple[float, float]:
    root = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    try:
        with open(os.path.join(root, "MEASURED_PEAKS.json")) as f:
            d = json.load(f)
        return d["hbm_gbs"] * 1e9, d["bf16_tflops"] * 1e12
    except (OSError, KeyError, ValueError):
        return 6.65e12, 1.59e15


def configs(size: str) -> dict[str, dict]:
    from vllm_b200.config.model import pomipel_config
    H, h, qr, kr, ff, E, k, G, keep = SIZES[size]
    own = pomipel_config(vocab=VOCAB, width=H, layers=LAYERS, heads=h, dim=HEAD_DIM, vdim=HEAD_DIM, q_rank=qr, kv_rank=kr, ff=ff,
                         experts=E, top=k, groups=G, keep=keep, max_positions=MAX_LEN, torch_dtype="bfloat16")
    like = dict(architectures=["DeepseekV3ForCausalLM"], model_type="deepseek_v3", vocab_size=VOCAB, hidden_size=H,
                intermediate_size=ff, moe_intermediate_size=ff, num_hidden_layers=LAYERS, num_attention_heads=h, num_key_value_heads=h,
                q_lora_rank=qr, kv_lora_rank=kr, qk_nope_head_dim=HEAD_DIM, qk_rope_head_dim=ROPE_DIM, v_head_dim=HEAD_DIM,
                n_routed_experts=E, n_shared_experts=0, num_experts_per_tok=k, n_group=G, topk_group=keep, routed_scaling_factor=1.0,
                first_k_dense_replace=0, moe_layer_freq=1, norm_topk_prob=False, scoring_func="sigmoid", topk_method="noaux_tc",
                max_position_embeddings=MAX_LEN, rms_norm_eps=1e-6, rope_theta=10000.0, hidden_act="silu", torch_dtype="bfloat16",
                tie_word_embeddings=False)
    shared = pomipel_config(vocab=VOCAB, width=H, layers=LAYERS, heads=h, dim=HEAD_DIM, vdim=HEAD_DIM, q_rank=qr, kv_rank=kr, ff=ff,
                            experts=E, top=k, groups=G, keep=keep, max_positions=MAX_LEN, share_every=2, torch_dtype="bfloat16")
    return {"pomipel": own, "pomipel, every second latent shared": shared, "deepseek-v3 layers": like}


def bench_model(name: str, cfg: dict, batch: int = 64, ctx: int = 1024, prompts: int = 8, steps: int = 20) -> dict:
    from vllm_b200 import LLM, SamplingParams
    with tempfile.TemporaryDirectory() as d:
        with open(os.path.join(d, "config.json"), "w") as f:
            json.dump(cfg, f)
        llm = LLM(d, load_format="dummy", dtype="bfloat16", skip_tokenizer_init=True, max_model_len=MAX_LEN, max_num_seqs=batch,
                  max_num_batched_tokens=prompts * ctx, enable_prefix_caching=False, cudagraph_capture_sizes=[batch],
                  gpu_memory_utilization=0.5, multiprocess_mode=False, disable_log_stats=True)
    engine = llm.llm_engine
    runner = engine.engine_core.engine_core.model_executor.worker.runner
    g = torch.Generator().manual_seed(0)

    def ev() -> torch.cuda.Event:
        e = torch.cuda.Event(enable_timing=True)
        e.record()
        return e
    # prefill: one engine step runs `prompts` whole prompts
    sp1 = SamplingParams(max_tokens=1, temperature=0.0, ignore_eos=True, detokenize=False)
    times = []
    for it in range(6):
        for i in range(prompts):
            engine.add_request(f"p{it}-{i}", {"prompt_token_ids": torch.randint(0, VOCAB, (ctx,), generator=g).tolist()}, sp1)
        torch.cuda.synchronize()
        a = ev()
        engine.step()
        b = ev()
        torch.cuda.synchronize()
        while engine.has_unfinished_requests():
            engine.step()
        if it >= 3:
            times.append(a.elapsed_time(b))
    prefill_ms = statistics.median(times)
    # decode: the batch at `ctx` tokens each, then replays of the captured step
    sp = SamplingParams(max_tokens=64, temperature=0.0, ignore_eos=True, detokenize=False)
    for i in range(batch):
        engine.add_request(f"d{i}", {"prompt_token_ids": torch.randint(0, VOCAB, (ctx,), generator=g).tolist()}, sp)
    graph = runner.graphs.get(batch)
    for _ in range(batch // prompts + 12):
        engine.step()
    decode_ms = launches = None
    if graph is not None and getattr(graph, "replays", 0):
        runner.finalize_pending()
        for _ in range(5):
            graph.graph.replay()
        torch.cuda.synchronize()
        a = ev()
        for _ in range(steps):
            graph.graph.replay()
        b = ev()
        torch.cuda.synchronize()
        decode_ms, launches = a.elapsed_time(b) / steps, graph.num_launches
    while engine.has_unfinished_requests():
        engine.step()
    llm.shutdown()
    del llm, engine, runner, graph
    torch.cuda.empty_cache()
    return {"model": name, "prefill_ms": prefill_ms, "prefill_tokens_per_s": prompts * ctx / prefill_ms * 1e3,
            "decode_ms": decode_ms, "decode_tokens_per_s": batch / decode_ms * 1e3 if decode_ms else None,
            "own_launches_per_decode_step": launches, "prefill_tokens": prompts * ctx, "decode_batch": batch, "context": ctx}


# ------------------------------------------------------------------------------------------------ kernels
def _pages(B: int, ctx: int, row: int, BS: int = 64):
    n = math.ceil(ctx / BS)
    cache = torch.randn(B * n + 1, BS, row, device="cuda", dtype=BF) * 0.3
    bt = (torch.randperm(B * n, device="cuda").int() + 1).view(B, n)
    return cache, bt, torch.full((B,), ctx, dtype=torch.int32, device="cuda")


def _routing(T: int, E: int, k: int):
    ids = torch.rand(T, E, device="cuda").topk(k, -1).indices.int()
    return torch.rand(T, k, device="cuda"), ids


def bench_kernels(size: str = "2k", batch: int = 64, prompts: int = 8, ctx: int = 1024) -> list[dict]:
    """Rows: operation, time and roofline fraction of this design's kernel and of the like kernel."""
    from vllm_b200 import ops
    from vllm_b200.forward_context import AttentionMetadata
    from vllm_b200.ops import cuda as cu
    from vllm_b200.ops import moe
    H, h, qr, kr, ff, E, k, G, keep = SIZES[size]
    D, P, T = HEAD_DIM, ROPE_DIM, prompts * ctx
    bw, fl = _peaks()
    rows: list[dict] = []

    def rnd(*shape, s=0.1):
        return torch.randn(*shape, device="cuda", dtype=BF) * s

    def row(op, own, own_bytes, own_flops, like_name, like, like_bytes, like_flops):
        t = timeit(own)
        best = max(own_bytes / bw, own_flops / fl) * 1e6
        r = {"op": op, "us": t, "of_roofline": best / t}
        if like is not None:
            tl = timeit(like)
            bl = max(like_bytes / bw, like_flops / fl) * 1e6
            r.update(like=like_name, like_us=tl, like_of_roofline=bl / tl, farther_by=(bl / tl) / (best / t))
        rows.append(r)

    # ---- attention
    for c in (ctx, 4 * ctx):
        qn, qp = rnd(batch, h, kr), rnd(batch, h, P)
        cache, bt, sl = _pages(batch, c, kr)
        cache_r, bt_r, _ = _pages(batch, c, kr + P)
        row(f"latent decode, {batch} x {c} tokens, {h} heads", lambda: cu.mla_decode_tc(qn, None, cache, bt, sl, 0.08, c), batch * c * kr * 2,
            2.0 * batch * c * h * 2 * kr, "MLA decode with rope", lambda: cu.mla_decode_tc(qn, qp, cache_r, bt_r, sl, 0.08, c),
            batch * c * (kr + P) * 2, 2.0 * batch * c * h * (2 * kr + P))
        del cache, cache_r
    i32 = dict(dtype=torch.int32, device="cuda")
    q, kk, vv, out = rnd(T, h, D), rnd(T, h, D), rnd(T, h, D), torch.empty(T, h, D, device="cuda", dtype=BF)
    start, lens = torch.arange(0, T, ctx, **i32), torch.full((prompts,), ctx, **i32)
    att_fl = 2.0 * 2 * h * D * prompts * ctx * (ctx + 1) / 2
    kv_pages = rnd(T // 64 + 1, 2, h, 64, D)
    md = AttentionMetadata(num_reqs=prompts, num_actual_tokens=T, max_query_len=ctx, max_seq_len=ctx,
                           query_start_loc=torch.arange(0, T + 1, ctx, **i32), seq_lens=lens,
                           block_table=(torch.arange(T // 64, **i32) + 1).view(prompts, -1), slot_mapping=None, kv_vt=True)
    row(f"prompt attention, {prompts} x {ctx} tokens, {h} heads", lambda: cu.mla_prefill(q, kk, vv, out, start, lens, lens, start, 0, ctx, D ** -0.5),
        4 * T * h * D * 2, att_fl, "paged prompt attention (llama)", lambda: cu.paged_attention(q, kv_pages, md, D ** -0.5),
        4 * T * h * D * 2, att_fl)
    del q, kk, vv, out, kv_pages

    # ---- experts
    up, down, w13 = rnd(E, ff, H, s=0.02), rnd(E, H, ff, s=0.02), rnd(E, 2 * ff, H, s=0.02)
    for n in (batch, T):
        x = rnd(n, H)
        wt, ids = _routing(n, E, k)
        R = n * k
        used = int(ids.unique().numel())
        act = 2 * (2 * R * H + 2 * R * ff)
        row(f"experts, {n} tokens (sort, gather, both products, activation)", lambda: moe.expert_rows_plain(x, up, down, ids, "relu2", None),
            used * 2 * ff * H * 2 + act, 2.0 * R * 2 * ff * H, "gated experts (+ combine)",
            lambda: cu.fused_moe(x, w13, down, wt, ids, "silu"), used * 3 * ff * H * 2 + act, 2.0 * R * 3 * ff * H)
        st, res = torch.randn(n, H, device="cuda"), rnd(n, H)
        nw = rnd(H)
        y, inv = moe.expert_rows_plain(x, up, down, ids, "relu2", None)

        def like_combine():
            o = cu.moe_combine(y, inv, wt, n)
            cu.fused_add_rms_norm(o, res, nw, 1e-6)
        row(f"combine + norm + residual, {n} tokens", lambda: cu.post_norm_add(st, y, nw, 1e-6, True, inv=inv, pair_w=wt),
            R * H * 2 + n * H * 10, 0, "combine, then residual + norm", like_combine, R * H * 2 + n * H * 2 * 6, 0)
        o = rnd(n, H)
        row(f"norm + residual, {n} tokens", lambda: cu.post_norm_add(st, o, nw, 1e-6, True), n * H * 12, 0, "residual + norm (16-bit stream)",
            lambda: cu.fused_add_rms_norm(o, res, nw, 1e-6), n * H * 8, 0)
        gate, corr = rnd(E, H, s=0.02), torch.randn(E, device="cuda")

        def like_router():
            ops.topk_softmax(ops.linear(x, gate).float(), k, True)
        row(f"router, {n} tokens", lambda: cu.router_topk(st, gate, k, G, keep, False, "sigmoid", corr, 1.0, x),
            n * H * (4 if n <= cu.ROUTER_FUSED_TOKENS else 2) + E * H * 2, 2.0 * n * E * H, "gate product + softmax top-k (no groups)", like_router,
            n * H * 2 + E * H * 2, 2.0 * n * E * H)
        lat = rnd(n, qr + kr + P)
        cache = torch.zeros(n // 64 + 1, 64, kr, device="cuda", dtype=BF)
        cache_r = torch.zeros(n // 64 + 1, 64, kr + P, device="cuda", dtype=BF)
        slots = torch.arange(n, device="cuda")
        gq, gk = rnd(qr), rnd(kr)

        def like_latent():
            cu.rms_norm(lat[:, :qr], gq, 1e-6)
            c = cu.rms_norm(lat[:, qr:qr + kr], gk, 1e-6)
            cu.concat_and_cache_mla(c, lat[:, qr + kr:].contiguous(), cache_r, slots)
        row(f"latent norms + cache write, {n} tokens",
            lambda: cu.latent_norm_cache(lat[:, :qr + kr], qr, gq, kr, gk, 1e-6, cache, slots, want_kv=False), n * (qr + kr) * 4, 0,
            "two norms, then cache write", like_latent, n * (qr + kr + P) * 4, 0)
        table, pos = rnd(VOCAB, H), rnd(MAX_LEN, H)
        tok, where = torch.randint(0, VOCAB, (n,), device="cuda").int(), torch.randint(0, MAX_LEN, (n,), device="cuda")
        row(f"embedding, {n} tokens", lambda: cu.embed_stream(tok, where, table, pos, 3.0), n * H * 10, 0, "embedding (16-bit)",
            lambda: torch.nn.functional.embedding(tok, table), n * H * 4, 0)
    return rows


def run(part: str = "all", sizes=None, steps: int = 20) -> dict:
    out: dict = {"design": "pomipel", "layers": LAYERS, "dtype": "bf16", "models": [], "kernels": []}
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
