"""Gizilorn beside the closest models of the framework at equal sizes: Mistral (sliding-window attention; gated feed-forward of as many
parameters), Gemma-2 (capped scores beside a window) and DeepSeek-V2 with dense feed-forwards (latent attention with a rotated part).
Prefill and decode throughput of a few layers through the engine, and every kernel against its roofline next to the like kernel.

    python bench.py --design gizilorn [--design-part model|kernels|all] [--design-sizes 1k,2k,4k] [--steps K]

Method and roofline as in ``benchmarks/latent_layers.py``.  The FLOPs of attention with mixed heads are those of the mechanism as it is
written (scores, mixed weights, values: 2 (dim + heads + vdim) per head and visible pair), not those of the form the kernels use.
"""
from __future__ import annotations

import json

import torch

from vllm_b200.benchmarks.kernels import timeit
from vllm_b200.benchmarks.latent_layers import BF, LAYERS, MAX_LEN, VOCAB, _pages, _peaks, bench_model

# (width, query heads, kv heads, latent heads, feed-forward); sizes that all share below
SIZES = {"1k": (1024, 8, 2, 8, 4096), "2k": (2048, 16, 4, 16, 8192), "4k": (4096, 32, 8, 32, 16384)}
HEAD, ROT, RANK, WINDOW, STREAMS = 128, 64, 512, 512, 4


def _gated(ff: int) -> int:
    """Width of a gated feed-forward with as many parameters."""
    return ff * 2 // 3 // 128 * 128


def configs(size: str) -> dict[str, dict]:
    from vllm_b200.config.model import gizilorn_config
    W, H, G, LH, ff = SIZES[size]

    def own(layers):
        return gizilorn_config(vocab=VOCAB, width=W, layers=layers, heads=H, kv_heads=G, dim=HEAD, latent_heads=LH, latent_dim=HEAD, rot_dim=ROT,
                               latent_vdim=HEAD, kv_rank=RANK, window=WINDOW, latent_window=WINDOW, ff=ff, streams=STREAMS,
                               max_position_embeddings=MAX_LEN, torch_dtype="bfloat16")
    common = dict(vocab_size=VOCAB, hidden_size=W, num_hidden_layers=LAYERS, max_position_embeddings=MAX_LEN, rms_norm_eps=1e-6,
                  torch_dtype="bfloat16", tie_word_embeddings=False, rope_theta=10000.0)
    mistral = dict(architectures=["MistralForCausalLM"], model_type="mistral", intermediate_size=_gated(ff), num_attention_heads=H,
                   num_key_value_heads=G, head_dim=HEAD, sliding_window=WINDOW, hidden_act="silu", **common)
    gemma = dict(architectures=["Gemma2ForCausalLM"], model_type="gemma2", intermediate_size=_gated(ff), num_attention_heads=H,
                 num_key_value_heads=G, head_dim=HEAD, sliding_window=WINDOW, hidden_activation="gelu_pytorch_tanh", query_pre_attn_scalar=HEAD,
                 attn_logit_softcapping=50.0, final_logit_softcapping=None, **common)
    deepseek = dict(architectures=["DeepseekV2ForCausalLM"], model_type="deepseek_v2", intermediate_size=_gated(ff), moe_intermediate_size=_gated(ff),
                    num_attention_heads=LH, num_key_value_heads=LH, q_lora_rank=None, kv_lora_rank=RANK, qk_nope_head_dim=HEAD,
                    qk_rope_head_dim=ROT, v_head_dim=HEAD, n_routed_experts=None, first_k_dense_replace=LAYERS, hidden_act="silu", **common)
    return {"gizilorn": own(["attention", "latent", "reuse", "attention"]), "gizilorn, attention only": own(["attention"] * LAYERS),
            "mistral layers": mistral, "gemma-2 layers": gemma, "gizilorn, latent only": own(["latent"] * LAYERS), "deepseek-v2 dense layers": deepseek}


def bench_kernels(size: str = "2k", batch: int = 64, prompts: int = 8, ctx: int = 1024) -> list[dict]:
    """Rows: operation, time and roofline fraction of this design's kernel and of the like kernel."""
    from vllm_b200 import ops
    from vllm_b200.forward_context import AttentionMetadata
    from vllm_b200.layers.rotary import get_rope
    from vllm_b200.ops import cuda as cu
    W, H, G, LH, ff = SIZES[size]
    bw, fl = _peaks()
    rows: list[dict] = []
    i32 = dict(dtype=torch.int32, device="cuda")

    def rnd(*shape, s=0.3, dtype=BF):
        return (torch.randn(*shape, device="cuda") * s).to(dtype)

    def row(op, own, own_bytes, own_flops, like_name=None, like=None, like_bytes=0, like_flops=0, note=None):
        t = timeit(own)
        best = max(own_bytes / bw, own_flops / fl) * 1e6
        r = {"op": op, "us": t, "of_roofline": best / t}
        if note is not None:
            r["of_executed_flops"] = note / fl * 1e6 / t
        if like is not None:
            tl = timeit(like)
            bl = max(like_bytes / bw, like_flops / fl) * 1e6
            r.update(like=like_name, like_us=tl, like_of_roofline=bl / tl, farther_by=(bl / tl) / (best / t))
        rows.append(r)

    def pairs(n_req, q_len, seq, window):
        return n_req * sum(min(p + 1, window) for p in range(seq - q_len, seq))

    # ---- attention with mixed heads
    talk = torch.randn(H, H, device="cuda") * 0.2
    sinks = torch.zeros(H, device="cuda")
    with torch.device("cuda"):
        rope = get_rope(HEAD, HEAD, 16384, 10000.0, True, dict(exact=True))
        lrope = get_rope(ROT, ROT, 16384, 10000.0, False, dict(exact=True))
    for n_req, q_len, seq, window in ((batch, 1, ctx, WINDOW), (batch, 1, 4 * ctx, 4 * ctx), (4 * batch, 1, ctx, WINDOW), (prompts, ctx, ctx, WINDOW),
                                      (2, 4 * ctx, 4 * ctx, 2 * ctx)):
        T = n_req * q_len
        per = -(-seq // 64)
        kv = rnd(n_req * per + 1, 2, G, 64, HEAD)
        bt = (torch.randperm(n_req * per, device="cuda").int() + 1).view(n_req, per)
        md = AttentionMetadata(num_reqs=n_req, num_actual_tokens=T, max_query_len=q_len, max_seq_len=seq,
                               query_start_loc=torch.arange(0, T + 1, q_len, **i32), seq_lens=torch.full((n_req,), seq, **i32), block_table=bt,
                               slot_mapping=None, kv_vt=True, decode_only=q_len == 1)
        q, pos = rnd(T, H, HEAD, s=1.0), torch.arange(seq - q_len, seq, device="cuda").repeat(n_req)
        n = pairs(n_req, q_len, seq, window)
        seen = min(seq, window + q_len - 1) * n_req
        byts = seen * G * 2 * HEAD * 2 + 2 * T * H * HEAD * 2
        name = f"{n_req} x {q_len} tokens at {seq}, window {window}"
        fold = 2.0 * n * H * (HEAD + G * HEAD)
        own = lambda: cu.talking_attention(q, kv, md, HEAD ** -0.5, window, 50.0, talk, sinks, HEAD, rope, pos)  # noqa: E731
        row(f"attention with mixed heads, {name}", own, byts, 2.0 * n * H * (2 * HEAD + H), "paged attention with a window (mistral)",
            lambda: cu.paged_attention(q, kv, md, HEAD ** -0.5, window), byts, 4.0 * n * H * HEAD, note=fold)
        kv32, md32 = kv.view(-1, 2, G, 64, HEAD), AttentionMetadata(**{**md.__dict__, "kv_vt": False})
        row(f"attention with mixed heads, {name} (again)", own, byts, 2.0 * n * H * (2 * HEAD + H), "capped attention with a window (gemma-2)",
            lambda: cu.paged_attention(q, kv32, md32, HEAD ** -0.5, window, 50.0), byts, 4.0 * n * H * HEAD, note=fold)
        if q_len > 1:
            o, out = rnd(T, H, G, HEAD), torch.empty(T, H, HEAD, device="cuda", dtype=BF)

            def mix():
                cu._check(cu._talk_mix(o.data_ptr(), 0, None, None, talk.data_ptr(), pos.data_ptr(), rope.cos_sin_cache.data_ptr(), 1, out.data_ptr(),
                                       out.stride(0), T, H, H // G, HEAD, 1, 0, G, 0, cu._st()), "talk_mix")
            row(f"  of it: mix and turn back, {T} tokens", mix, T * H * (G + 1) * HEAD * 2, 0)
            del o, out
        del kv, kv32

    # ---- prologues, streams, feed-forward
    for n in (batch, prompts * ctx):
        slots, pos = torch.arange(n, device="cuda"), torch.arange(n, device="cuda") % 8192
        qkv = rnd(n, (H + 2 * G) * HEAD)
        q, k, v = qkv.split([H * HEAD, G * HEAD, G * HEAD], -1)
        cache = torch.zeros(n // 64 + 2, 2, G, 64, HEAD, device="cuda", dtype=BF)
        b = n * (2 * H + 4 * G) * HEAD * 2
        row(f"rotation of queries, keys and values, cache write, {n} tokens",
            lambda: cu.fused_qk_norm_rope(pos, q, k, None, None, rope.cos_sin_cache, HEAD, 0.0, True, v=v, kv_cache=cache, slot_mapping=slots, vt=True,
                                          keep32=True, v_cos_sin=rope.cos_sin_cache), b, 0, "rotation of queries and keys, cache write (mistral)",
            lambda: cu.rope_and_cache(pos, q, k, v, rope.cos_sin_cache, HEAD, True, cache, slots, vt=True), b, 0)
        proj = rnd(n, LH * (HEAD + ROT) + LH * HEAD + RANK + ROT)
        off = LH * (2 * HEAD + ROT)
        lat = torch.zeros(n // 64 + 2, 64, RANK + ROT, device="cuda", dtype=BF)
        nw = rnd(RANK)

        def like_latent():
            c = cu.rms_norm(proj[:, off:off + RANK], nw, 1e-6)
            qp = proj[:, :LH * (HEAD + ROT)].view(n, LH, HEAD + ROT)[..., HEAD:].reshape(n, LH * ROT)
            kp = proj[:, off + RANK:].contiguous()
            cu.rotary_embedding(pos, qp, kp, lrope.cos_sin_cache, ROT, False)
            cu.concat_and_cache_mla(c, kp, lat, slots)
        row(f"latent norm, rotations, cache write, {n} tokens",
            lambda: cu.latent_rope_cache(proj, 0, LH, HEAD, ROT, off, RANK, nw, 1e-6, pos, lrope.cos_sin_cache, False, lat, slots),
            n * (2 * LH * ROT + 2 * (RANK + ROT)) * 2, 0, "norm, rotation, cache write (deepseek)", like_latent,
            n * (2 * LH * ROT + 2 * (RANK + ROT)) * 2, 0)
        x, y, w = torch.randn(n, STREAMS, W, device="cuda"), rnd(n, W), rnd(W)
        coef, into = torch.randn(STREAMS + STREAMS ** 2, device="cuda") * 0.3, torch.ones(STREAMS, device="cuda")
        st, res = torch.randn(n, W, device="cuda"), rnd(n, W)
        row(f"hyper-connections ({STREAMS} streams) + norm, {n} tokens", lambda: cu.hyper_step(x, y, coef, into, w, 1e-6, BF),
            n * W * (8 * STREAMS + 4), 0, "residual + norm, fp32 stream (kopadra)", lambda: cu.add_norm(st, y, (w, None), 1e-6), n * W * 12, 0)
        row(f"hyper-connections ({STREAMS} streams) + norm, {n} tokens (again)", lambda: cu.hyper_step(x, y, coef, into, w, 1e-6, BF),
            n * W * (8 * STREAMS + 4), 0, "residual + norm, 16-bit stream (mistral)", lambda: cu.fused_add_rms_norm(y, res, w, 1e-6), n * W * 8, 0)
        ids, table = torch.randint(0, VOCAB, (n,), **i32), rnd(VOCAB, W)
        row(f"entry: embedding, norm, streams, norm, {n} tokens", lambda: cu.hyper_entry(ids, table, STREAMS, w, into, w, 1e-6),
            n * W * (4 + 4 * STREAMS), 0, "embedding + norm, fp32 stream (kopadra)",
            lambda: cu.norm_add(st, table, None, None, 1.0, (w, None), 1e-6, ids=ids), n * W * 8, 0)
        gff = _gated(ff)
        up, bias, act, gu = rnd(ff, W, s=0.02), rnd(ff), torch.tensor([0.7, 1.2], device="cuda"), rnd(2 * gff, W, s=0.02)
        h = rnd(n, W)
        row(f"projection with xIELU, {n} tokens", lambda: cu.linear_xielu(h, up, bias, act), (ff * W + n * (W + ff)) * 2, 2.0 * n * W * ff,
            "gated projection with SiLU (mistral)", lambda: ops.gated_silu_linear(h, gu), (2 * gff * W + n * (W + gff)) * 2, 4.0 * n * W * gff)
        if n > 256:
            a, g2 = rnd(n, ff), rnd(n, 2 * gff)
            row(f"  of it: xIELU, {n} tokens", lambda: cu.xielu(a, act, out=a), n * ff * 4, 0, "SiLU x gate", lambda: cu.act_and_mul(g2, "silu"),
                n * gff * 6, 0)
            del a, g2
        del x, cache, lat, qkv, proj

    # ---- latent attention
    for c, window in ((ctx, WINDOW), (4 * ctx, 4 * ctx)):
        qn, qp = rnd(batch, LH, RANK), rnd(batch, LH, ROT)
        cache, bt, sl = _pages(batch, c, RANK + ROT)
        s = min(c, window)
        row(f"latent decode, {batch} tokens at {c}, window {window}, {LH} heads",
            lambda: cu.mla_decode_tc(qn, qp, cache, bt, sl, 0.07, c, sliding_window=window), batch * s * (RANK + ROT) * 2,
            2.0 * batch * s * LH * (2 * RANK + ROT), "latent decode without a window (deepseek)",
            lambda: cu.mla_decode_tc(qn, qp, cache, bt, sl, 0.07, c), batch * c * (RANK + ROT) * 2, 2.0 * batch * c * LH * (2 * RANK + ROT))
        del cache
    for n_req, q_len, window in ((prompts, ctx, WINDOW), (2, 4 * ctx, 2 * ctx)):
        T = n_req * q_len
        q, k, v, out = rnd(T, LH, HEAD + ROT), rnd(T, LH, HEAD), rnd(T, LH, HEAD), torch.empty(T, LH, HEAD, device="cuda", dtype=BF)
        rows_, start, lens = rnd(T, RANK + ROT), torch.arange(0, T, q_len, **i32), torch.full((n_req,), q_len, **i32)
        qs = rnd(T, LH, HEAD)
        n = pairs(n_req, q_len, q_len, window)
        full = pairs(n_req, q_len, q_len, q_len)
        row(f"latent prompt attention, {n_req} x {q_len} tokens, window {window}, {LH} heads",
            lambda: cu.mla_prefill(q, k, v, out, start, lens, lens, start, 0, q_len, 0.07, rows_[:, RANK:], window), T * LH * (4 * HEAD + ROT) * 2,
            2.0 * n * LH * (2 * HEAD + ROT), "latent prompt attention without a rotated part or a window (pomipel)",
            lambda: cu.mla_prefill(qs, k, v, out, start, lens, lens, start, 0, q_len, 0.09), T * LH * 4 * HEAD * 2, 2.0 * full * LH * 2 * HEAD)
        o, g = rnd(T, LH * HEAD), rnd(T, LH * HEAD)
        row(f"output gate, {T} tokens", lambda: cu.sigmoid_mul_(o, g), T * LH * HEAD * 6, 0, "SiLU x gate", lambda: cu.act_and_mul(g, "silu"),
            T * LH * HEAD * 3, 0)
        del q, k, v, out
    return rows


def run(part: str = "all", sizes=None, steps: int = 20) -> dict:
    out: dict = {"design": "gizilorn", "layers": LAYERS, "dtype": "bf16", "models": [], "kernels": []}
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
