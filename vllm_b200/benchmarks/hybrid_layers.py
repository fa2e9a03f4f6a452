"""Legelix beside the closest models of the framework at equal sizes: Falcon-H1 (attention and Mamba-2 side by side) for the
parallel layers, the gated delta rule of Qwen3-Next for the gated-linear ones.  Prefill and decode throughput of a few layers
through the engine, and every kernel against its roofline next to the like kernel.

    python bench.py --design legelix [--design-part model|kernels|all] [--design-sizes 1k,2k,4k] [--steps K]

Method and roofline as in ``benchmarks/latent_layers.py``.  A scan's FLOPs are those of the recurrence (six per element of the
state and token) over the tensor-core rate, although it runs on the CUDA cores.
"""
from __future__ import annotations

import json

import torch

from vllm_b200.benchmarks.kernels import timeit
from vllm_b200.benchmarks.latent_layers import BF, LAYERS, MAX_LEN, VOCAB, _peaks, bench_model

# (width, query heads, kv heads, Mamba-2 heads, B/C groups, gated-linear heads, feed-forward); head sizes below
SIZES = {"1k": (1024, 8, 2, 32, 1, 4, 2816), "2k": (2048, 16, 4, 64, 1, 8, 5632), "4k": (4096, 32, 8, 128, 8, 16, 14336)}
HEAD, SSM_HEAD, STATE, TAPS, GLA_K, GLA_V, RANK, CHUNK = 128, 64, 128, 4, 128, 256, 16, 8192


def configs(size: str) -> dict[str, dict]:
    from vllm_b200.config.model import legelix_config
    W, H, G, MH, MG, GH, ff = SIZES[size]
    kw = dict(vocab=VOCAB, width=W, heads=H, kv_heads=G, dim=HEAD, chunk=CHUNK, ssm_heads=MH, ssm_dim=SSM_HEAD, state=STATE, groups=MG,
              conv=TAPS, gla_heads=GH, gla_dim=GLA_K, gla_vdim=GLA_V, ff=ff, max_position_embeddings=MAX_LEN, torch_dtype="bfloat16")
    like = dict(architectures=["FalconH1ForCausalLM"], model_type="falcon_h1", vocab_size=VOCAB, hidden_size=W, intermediate_size=ff,
                num_hidden_layers=LAYERS, num_attention_heads=H, num_key_value_heads=G, head_dim=HEAD, max_position_embeddings=MAX_LEN,
                mamba_d_ssm=MH * SSM_HEAD, mamba_n_heads=MH, mamba_d_head=SSM_HEAD, mamba_n_groups=MG, mamba_d_state=STATE,
                mamba_d_conv=TAPS, mamba_chunk_size=128, mamba_conv_bias=True, mamba_proj_bias=False, mamba_norm_before_gate=False,
                mamba_rms_norm=True, rope_theta=10000.0, hidden_act="silu", rms_norm_eps=1e-6, torch_dtype="bfloat16",
                tie_word_embeddings=False)
    return {"legelix": legelix_config(layers=["parallel", "gla"] * (LAYERS // 2), **kw),
            "legelix, parallel layers only": legelix_config(layers=["parallel"] * LAYERS, **kw), "falcon-h1 layers": like}


def bench_kernels(size: str = "2k", batch: int = 64, prompts: int = 8, ctx: int = 1024) -> list[dict]:
    """Rows: operation, time and roofline fraction of this design's kernel and of the like kernel."""
    from vllm_b200.forward_context import AttentionMetadata
    from vllm_b200.ops import cuda as cu
    from vllm_b200.ops import scan_state_elems
    W, H, G, MH, MG, GH, ff = SIZES[size]
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

    def meta(n_req, q_len, total, table):
        return AttentionMetadata(num_reqs=n_req, num_actual_tokens=n_req * q_len, max_query_len=q_len, max_seq_len=total,
                                 query_start_loc=torch.arange(0, n_req * q_len + 1, q_len, **i32), seq_lens=torch.full((n_req,), total, **i32),
                                 block_table=table, slot_mapping=None, kv_vt=True, decode_only=q_len == 1)

    # ---- attention: chunk mask and sinks against the plain causal form of the same kernels
    sinks = torch.randn(H, device="cuda")
    for n_req, q_len, total in ((batch, 1, ctx), (batch, 1, 4 * ctx), (prompts, ctx, ctx)):
        pages = -(-total // 64)
        cache = rnd(n_req * pages + 1, 2, G, 64, HEAD)
        md = meta(n_req, q_len, total, (torch.randperm(n_req * pages, device="cuda").int() + 1).view(n_req, pages))
        q = rnd(n_req * q_len, H, HEAD)
        out = torch.empty(n_req * q_len, H * HEAD + 64, device="cuda", dtype=BF)[:, :H * HEAD].view(-1, H, HEAD)
        nbytes = n_req * total * 2 * G * HEAD * 2 + 2 * n_req * q_len * H * HEAD * 2
        flops = 2.0 * 2 * H * HEAD * n_req * (total if q_len == 1 else q_len * (q_len + 1) / 2)
        name = f"{n_req} x {total}" + ("" if q_len == 1 else " prompt")
        row(f"attention, chunk and sinks, {name}", lambda: cu.paged_attention(q, cache, md, 0.09, out=out, sinks=sinks, chunk_size=CHUNK, out_scale=0.8),
            nbytes, flops, "attention (llama)", lambda: cu.paged_attention(q, cache, md, 0.09), nbytes, flops)
        del cache, q, out
    inner, bc = MH * SSM_HEAD, 2 * MG * STATE
    for n_req, q_len in ((batch, 1), (prompts, ctx), (1, prompts * ctx)):
        T = n_req * q_len
        name = f"{T} tokens" + ("" if q_len == 1 else f" in {n_req} prompt{'s' if n_req > 1 else ''}")
        slots = (torch.arange(n_req, **i32) + 1).view(-1, 1).contiguous()
        start = ctx if q_len == 1 else 0
        md = meta(n_req, q_len, start + q_len, slots)
        # ---- prologue
        if n_req > 1:
            qkv = rnd(T, (H + 2 * G) * HEAD)
            q, k, v = qkv.split([H * HEAD, G * HEAD, G * HEAD], -1)
            cs, pos = rnd(MAX_LEN, HEAD, dtype=torch.float32), torch.arange(T, device="cuda") % ctx
            cache, where, nw = rnd(T // 64 + 2, 2, G, 64, HEAD), torch.arange(T, device="cuda"), rnd(HEAD)
            nb = 2 * T * (H + 2 * G) * HEAD * 2
            row(f"head norms, rotation, cache write, {name}",
                lambda: cu.fused_qk_norm_rope(pos, q, k, nw, nw, cs, HEAD, 1e-6, False, v=v, kv_cache=cache, slot_mapping=where, vt=True, keep32=True),
                nb, 0, "rotation, cache write (llama)", lambda: cu.rope_and_cache(pos, q, k, v, cs, HEAD, True, cache, where, vt=True), nb, 0)
            del qkv, cache
        # ---- Mamba-2
        state_off = (inner + bc) * (TAPS - 1)
        pool = torch.zeros(n_req + 1, state_off + MH * scan_state_elems(STATE, SSM_HEAD), device="cuda")
        xbc, w, b = rnd(T, inner + bc), rnd(inner + bc, TAPS), rnd(inner + bc)
        row(f"short convolution, {name}", lambda: cu.causal_conv1d(xbc, w, b, pool, md), T * (inner + bc) * 6 + n_req * 2 * state_off * 4, 0)
        xa, dt = rnd(T, inner + bc, dtype=torch.float32), rnd(T, MH)
        A, D, tb = [torch.randn(MH, device="cuda") * 0.3 for _ in range(3)]
        st_bytes = n_req * MH * STATE * SSM_HEAD * 4 * (2 if start else 1)
        row(f"Mamba-2 scan, {name}", lambda: cu.ssd_scan(xa, dt, tb, A, D, pool, state_off, md, MH, SSM_HEAD, MG, STATE),
            T * (2 * inner + bc) * 4 + st_bytes, 6.0 * T * MH * STATE * SSM_HEAD)
        y, z, gw = rnd(T, inner, dtype=torch.float32), rnd(T, inner), rnd(inner)
        x16, res = rnd(T, inner), rnd(T, inner)
        row(f"gate, then group norm, {name}", lambda: cu.gated_norm(y, z, gw, MG, 1e-6, True), T * inner * 8, 0, "norm + residual (16-bit)",
            lambda: cu.fused_add_rms_norm(x16, res, gw, 1e-6), T * inner * 8, 0)
        del pool, xbc, xa, y, z, x16, res
        # ---- gated linear attention
        qk, vv = GH * GLA_K, GH * GLA_V
        pool = torch.zeros(n_req + 1, GH * scan_state_elems(GLA_K, GLA_V), device="cuda")
        x = rnd(T, 2 * qk + vv + RANK)
        q, k, v, a1 = x.split([qk, qk, vv, RANK], -1)
        a2, a2b = rnd(qk, RANK), rnd(qk)
        q32, k32, v32 = [rnd(T, GH, d, dtype=torch.float32) for d in (GLA_K, GLA_K, GLA_V)]
        dec, beta = -torch.rand(T, GH, device="cuda"), torch.rand(T, GH, device="cuda")
        st_bytes = n_req * GH * GLA_K * GLA_V * 4 * (2 if start else 1)
        row(f"gated-linear scan with its decays, {name}", lambda: cu.gla_scan(q, k, v, a1, a2, a2b, 16.0, 0.09, pool, md, GH, GLA_K, GLA_V),
            T * ((2 * qk + vv + RANK) * 2 + vv * 4) + st_bytes, 6.0 * T * GH * GLA_K * GLA_V, "gated delta rule scan",
            lambda: cu.gdn_scan(q32, k32, v32, dec, beta, pool, 0, md), T * (2 * qk + 2 * vv) * 4 + st_bytes, 8.0 * T * GH * GLA_K * GLA_V)
        y, g, hw = rnd(T, vv, dtype=torch.float32), rnd(T, vv), rnd(GLA_V)
        x16, res = rnd(T, vv), rnd(T, vv)
        nv = rnd(vv)
        row(f"head norm, then gate, {name}", lambda: cu.gated_norm(y, g, hw, GH, 1e-6, False), T * vv * 8, 0, "norm + residual (16-bit)",
            lambda: cu.fused_add_rms_norm(x16, res, nv, 1e-6), T * vv * 8, 0)
        del pool, x, q32, k32, v32, y, g, x16, res
        # ---- stream
        stream, y, res = rnd(T, W, dtype=torch.float32), rnd(T, W), rnd(T, W)
        n1 = [rnd(W) for _ in range(4)]
        row(f"layer norm, residual, layer norm, {name}", lambda: cu.norm_add(stream, y, None, (n1[0], n1[1]), 0.7, (n1[2], n1[3]), 1e-6),
            T * W * 12, 0, "residual + norm (16-bit stream)", lambda: cu.fused_add_rms_norm(y, res, n1[0], 1e-6), T * W * 8, 0)
    return rows


def run(part: str = "all", sizes=None, steps: int = 20) -> dict:
    out: dict = {"design": "legelix", "layers": LAYERS, "dtype": "bf16", "models": [], "kernels": []}
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
