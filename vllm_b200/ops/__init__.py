"""Op dispatch: CUDA tensors → our sm_100a kernels (``ops/cuda.py`` → ``_C.so``),
CPU tensors → the PyTorch reference (``ops/ref.py``).

There is deliberately no multi-backend registry (the reference has
``CustomOp`` + IR providers: model_executor/custom_op.py:103-210, vllm/ir/op.py);
this framework targets exactly one device.  A CUDA tensor with the extension
missing raises — it never silently falls back to eager PyTorch.
"""
from __future__ import annotations

from typing import Optional

import torch

from vllm_b200 import envs
from vllm_b200.ops import ref

_cuda_mod = None


def cuda_ops():
    global _cuda_mod
    if _cuda_mod is None:
        from vllm_b200.ops import cuda as _m
        _cuda_mod = _m
    return _cuda_mod


def _use_cuda(x: torch.Tensor) -> bool:
    return x.is_cuda and not envs.VLLM_B200_FORCE_REF_OPS


def _vec_ok(x: torch.Tensor) -> bool:
    """The row kernels move 16-byte vectors: the row width must be a multiple of 16 bytes."""
    return (x.shape[-1] * x.element_size()) % 16 == 0


def rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float, gemma: bool = False) -> torch.Tensor:
    if _use_cuda(x) and _vec_ok(x):
        return cuda_ops().rms_norm(x, weight, eps, gemma)
    return ref.rms_norm(x, weight, eps, gemma)


def fused_add_rms_norm(x: torch.Tensor, residual: torch.Tensor, weight: torch.Tensor, eps: float,
                       gemma: bool = False) -> tuple[torch.Tensor, torch.Tensor]:
    """Returns (normed, new_residual). The CUDA path updates ``residual`` in place and
    writes the normed result into ``x``'s storage."""
    if _use_cuda(x) and _vec_ok(x):
        return cuda_ops().fused_add_rms_norm(x, residual, weight, eps, gemma)
    return ref.fused_add_rms_norm(x, residual, weight, eps, gemma)


def layer_norm(x, weight, bias, eps):
    if _use_cuda(x):
        return cuda_ops().layer_norm(x, weight, bias, eps)
    return ref.layer_norm(x, weight, bias, eps)


def silu_and_mul(x: torch.Tensor) -> torch.Tensor:
    if _use_cuda(x):
        return cuda_ops().act_and_mul(x, "silu")
    return ref.silu_and_mul(x)


def silu_and_mul_interleaved(x: torch.Tensor) -> torch.Tensor:
    """silu(x[..., 0::2]) * x[..., 1::2]: the activation for gate_up weights stored as interleaved (gate_i, up_i) rows."""
    if _use_cuda(x):
        return cuda_ops().silu_and_mul_interleaved(x)
    return (torch.nn.functional.silu(x[..., 0::2].float()) * x[..., 1::2].float()).to(x.dtype)


def gated_silu_linear(x: torch.Tensor, weight_il: torch.Tensor) -> torch.Tensor:
    """silu(x Wg^T) * (x Wu^T) for a weight whose rows interleave (gate_i, up_i).  Decode batches on CUDA run ONE
    kernel: the stream-K tcgen05 GEMM applies SiLU·mul in its epilogue (csrc/gemm_sk.cu)."""
    K = x.shape[-1]
    x2 = x.reshape(-1, K)
    if _use_cuda(x):
        cu = cuda_ops()
        if 0 < x2.shape[0] <= 256 and cu._tc_ok(x2, weight_il) and weight_il.shape[0] % 4 == 0:
            fn = cu.gemm_sk if envs.VLLM_B200_GEMM_SK else cu.gemm_tc
            return fn(x2, weight_il, act=True).view(x.shape[:-1] + (weight_il.shape[0] // 2,))
    return silu_and_mul_interleaved(linear(x, weight_il))


def gelu_and_mul(x: torch.Tensor, approximate: str = "none") -> torch.Tensor:
    if _use_cuda(x):
        return cuda_ops().act_and_mul(x, "gelu_tanh" if approximate == "tanh" else "gelu")
    return ref.gelu_and_mul(x, approximate)


def activation(x: torch.Tensor, name: str) -> torch.Tensor:
    if _use_cuda(x):
        return cuda_ops().activation(x, name)
    return ref.ACT_FNS[name](x)


def sigmoid_mul_(x: torch.Tensor, gate: torch.Tensor) -> torch.Tensor:
    """x *= sigmoid(gate) in place, rows of any stride."""
    if _use_cuda(x):
        return cuda_ops().sigmoid_mul_(x, gate)
    return x.copy_(x.float() * torch.sigmoid(gate.float()))


def soft_cap(logits: torch.Tensor, cap: float) -> torch.Tensor:
    """cap tanh(logits / cap) in 32-bit; in place on CUDA."""
    if _use_cuda(logits):
        return cuda_ops().soft_cap_(logits, cap)
    return (torch.tanh(logits.float() / cap) * cap).to(logits.dtype)


_HALF = (torch.bfloat16, torch.float16)


def _rope_ok(q, cos_sin_cache, head_dim) -> bool:
    """Shapes the vectorised RoPE / cache-write kernel covers (16-byte vectors over half-precision heads)."""
    rot = cos_sin_cache.shape[-1]
    return q.dtype in _HALF and head_dim % 8 == 0 and (rot // 2) % 8 == 0 and (head_dim - rot) % 8 == 0


def cuda_attention_supported(D: int, DV: int, BS: int, G: int, dtype, kv_dtype, vt: bool = False) -> bool:
    """Every head shape has a kernel where the cache holds the model dtype (csrc/attention_any.cu takes what the others do
    not); fp8 caches need a shape of csrc/attention_simt.cu."""
    return vt or (kv_dtype == dtype and max(D, DV) <= 512) or cuda_ops()._simt_attention_ok(D, DV, BS, G, dtype)


def cuda_cache_write_supported(D: int, dtype) -> bool:
    """Layers without a fused prologue write their keys and values with the vectorised kernel (no host synchronisation)."""
    return dtype in _HALF and D % 8 == 0


def rotary_embedding(positions, q, k, cos_sin_cache, head_dim, is_neox=True):
    """In place on CUDA; returns (q, k)."""
    if _use_cuda(q) and _rope_ok(q, cos_sin_cache, head_dim):
        return cuda_ops().rotary_embedding(positions, q, k, cos_sin_cache, head_dim, is_neox)
    return ref.rotary_embedding(positions, q, k, cos_sin_cache, head_dim, is_neox)


def reshape_and_cache(key, value, kv_cache, slot_mapping, vt: bool = False) -> None:
    if _use_cuda(key) and (vt or (key.dtype in _HALF and key.shape[-1] % 8 == 0)):
        return cuda_ops().reshape_and_cache(key, value, kv_cache, slot_mapping, vt=vt)
    return ref.reshape_and_cache(key, value, kv_cache, slot_mapping)


def rope_and_cache(positions, q, k, v, cos_sin_cache, head_dim, is_neox, kv_cache, slot_mapping, vt: bool = False):
    """Fused RoPE(q,k) + paged KV write. q/k: [T, H*D] views; returns (q, k) rotated.
    ``vt``: the cache uses the tensor-core layout (V pages transposed), CUDA only."""
    if _use_cuda(q) and (vt or _rope_ok(q, cos_sin_cache, head_dim)):
        return cuda_ops().rope_and_cache(positions, q, k, v, cos_sin_cache, head_dim, is_neox, kv_cache,
                                         slot_mapping, vt=vt)
    q, k = ref.rotary_embedding(positions, q, k, cos_sin_cache, head_dim, is_neox)
    Hkv = kv_cache.shape[2]
    ref.reshape_and_cache(k.reshape(k.shape[0], Hkv, head_dim), v.reshape(v.shape[0], Hkv, head_dim),
                          kv_cache, slot_mapping)
    return q, k


def concat_and_cache_mla(kv_c, k_pe, kv_cache, slot_mapping) -> None:
    if _use_cuda(kv_c):
        return cuda_ops().concat_and_cache_mla(kv_c, k_pe, kv_cache, slot_mapping)
    return ref.concat_and_cache_mla(kv_c, k_pe, kv_cache, slot_mapping)


def paged_attention(q, kv_cache, md, scale, sliding_window=None, logits_soft_cap=0.0, causal=True,
                    out: Optional[torch.Tensor] = None, alibi_slopes: Optional[torch.Tensor] = None,
                    sinks: Optional[torch.Tensor] = None, chunk_size: int = 0, return_lse: bool = False,
                    v_head_size: Optional[int] = None, out_scale: float = 1.0):
    """``md``: AttentionMetadata (see vllm_b200.forward_context).  ``v_head_size``: value width where it is not the keys'.
    ``out``: [T, Hq, value width] to write into; ``out_scale``: its factor."""
    if _use_cuda(q) and cuda_attention_supported(q.shape[2], v_head_size or q.shape[2], kv_cache.shape[3],
                                                 q.shape[1] // kv_cache.shape[2], q.dtype, kv_cache.dtype, md.kv_vt):
        return cuda_ops().paged_attention(q, kv_cache, md, scale, sliding_window, logits_soft_cap, causal, out,
                                          return_lse=return_lse, alibi_slopes=alibi_slopes, sinks=sinks,
                                          chunk_size=chunk_size, v_head_size=v_head_size, out_scale=out_scale)
    sl = md.seq_lens_cpu if md.seq_lens_cpu is not None else md.seq_lens.cpu()
    qsl = md.query_start_loc_cpu if md.query_start_loc_cpu is not None else md.query_start_loc.cpu()
    pad = kv_cache.shape[-1] - q.shape[-1]
    if pad:                                   # cache rows as wide as the wider of key and value
        q = torch.nn.functional.pad(q, (0, pad))
    got = ref.paged_attention(q, kv_cache, md.block_table, sl, qsl, scale,
                              causal=causal, sliding_window=sliding_window, logits_soft_cap=logits_soft_cap,
                              alibi_slopes=alibi_slopes, sinks=sinks, chunk_size=chunk_size, return_lse=return_lse)
    o, lse = got if return_lse else (got, None)
    if v_head_size is not None:
        o = o[..., :v_head_size]
    if out_scale != 1.0:
        o = o * out_scale
    if out is not None:
        o = out.copy_(o)
    return (o, lse) if return_lse else o


def talking_attention(q, kv_cache, md, scale, sliding_window, soft_cap, talk, sinks, v_head_size: int, v_rope=None, positions=None,
                      out: Optional[torch.Tensor] = None):
    """paged_attention whose heads' weights are mixed by ``talk`` [Hq, Hq] behind the softmax (None: not mixed), outputs turned back by
    their position (``v_rope``: the rotation of the cached values)."""
    if _use_cuda(q):
        return cuda_ops().talking_attention(q, kv_cache, md, scale, sliding_window, soft_cap, talk, sinks, v_head_size, v_rope, positions, out)
    if talk is None:
        o = paged_attention(q, kv_cache, md, scale, sliding_window, soft_cap, sinks=sinks, v_head_size=v_head_size).float()
    else:
        sl = md.seq_lens_cpu if md.seq_lens_cpu is not None else md.seq_lens.cpu()
        qsl = md.query_start_loc_cpu if md.query_start_loc_cpu is not None else md.query_start_loc.cpu()
        o = ref.talking_attention(q, kv_cache, md.block_table, sl, qsl, scale, sliding_window, soft_cap, talk, sinks, v_head_size)
    if v_rope is not None:
        half = v_rope.cos_sin_cache.shape[-1] // 2
        back = torch.cat((v_rope.cos_sin_cache[:, :half], -v_rope.cos_sin_cache[:, half:]), dim=-1)
        o = ref.rotary_embedding(positions, o.reshape(o.shape[0], -1), None, back, v_head_size, v_rope.is_neox_style)[0].view(o.shape)
    return o.to(q.dtype) if out is None else out.copy_(o)


def mla_attention(q_nope_abs, q_pe, kv_cache, md, scale, kv_lora_rank, sliding_window: Optional[int] = None):
    """``q_pe`` None: no rope part."""
    if _use_cuda(q_nope_abs):
        return cuda_ops().mla_attention(q_nope_abs, q_pe, kv_cache, md, scale, kv_lora_rank, sliding_window)
    sl = md.seq_lens_cpu if md.seq_lens_cpu is not None else md.seq_lens.cpu()
    qsl = md.query_start_loc_cpu if md.query_start_loc_cpu is not None else md.query_start_loc.cpu()
    if q_pe is None:
        q_pe = q_nope_abs[..., :0]
    return ref.mla_decode_attention(q_nope_abs, q_pe, kv_cache, md.block_table, sl, qsl, scale, kv_lora_rank, sliding_window)


def mla_attention_rows(q_abs, q_pe, kv_cache, block_table, seq_lens, max_len: int, scale, sliding_window: Optional[int] = None):
    """Attention over the latent cache for rows with a block table and a number of visible keys each (CUDA); with a window, of its last
    ones."""
    cu = cuda_ops()
    if cu._mla_tc_ok(q_abs, q_pe, kv_cache):
        return cu.mla_decode_tc(q_abs, q_pe, kv_cache, block_table, seq_lens, scale, max_len, sliding_window=sliding_window)
    return cu.mla_simt(q_abs, q_pe, kv_cache, block_table, seq_lens, None, scale, sliding_window)


def latent_expand_ok(q, dim: int, rot: int, v_dim: int, kv_rank: int) -> bool:
    """Can prompt portions run over expanded keys and values (csrc/mla_prefill.cu)?"""
    return _use_cuda(q) and cuda_ops().mla_prefill_ok(q, dim, rot, v_dim, kv_rank)


def gather_latents(kv_cache, block_table, cu_kv, num_kv: int, max_kv: int, starts=None):
    """Cached rows of a batch of sequences (from position ``starts`` on), contiguous [num_kv, R] (CUDA)."""
    out = torch.empty((num_kv, kv_cache.shape[-1]), dtype=kv_cache.dtype, device=kv_cache.device)
    return cuda_ops().gather_cache(kv_cache, block_table, cu_kv, out, max_kv, starts)


def mla_prefill(q, k, v, out, q_start, q_len, seq_len, kv_start, h0: int, max_q: int, scale, k_pe=None, window: int = 0) -> None:
    cuda_ops().mla_prefill(q, k, v, out, q_start, q_len, seq_len, kv_start, h0, max_q, scale, k_pe, window)


def latent_rope_cache(proj, q_off, heads, dim, rot, kv_off, kv_rank, kv_weight, eps, positions, cos_sin, neox, cache=None, slots=None) -> None:
    """On the columns of a merged projection [T, ...], in place: rotates the last ``rot`` dimensions of every query head, norms the latent,
    rotates the key part behind it and writes both into their cache rows (``kv_rank`` 0: queries alone)."""
    if _use_cuda(proj):
        return cuda_ops().latent_rope_cache(proj, q_off, heads, dim, rot, kv_off, kv_rank, kv_weight, eps, positions, cos_sin, neox, cache, slots)
    return ref.latent_rope_cache(proj, q_off, heads, dim, rot, kv_off, kv_rank, kv_weight, eps, positions, cos_sin, neox, cache, slots)


def latent_norm_cache(lat, q_rank, q_weight, kv_rank, kv_weight, eps, cache=None, slots=None):
    """RMSNorm of both halves of a latent down-projection; the key / value latents go into their cache rows (and are
    returned by themselves where no cache is bound)."""
    if _use_cuda(lat):
        return cuda_ops().latent_norm_cache(lat, q_rank, q_weight, kv_rank, kv_weight, eps, cache, slots, want_kv=cache is None)
    return ref.latent_norm_cache(lat, q_rank, q_weight, kv_rank, kv_weight, eps, cache, slots)


def embed_stream(ids, positions, table, pos_table=None, scale: float = 1.0):
    """Entry of an fp32 residual stream: (table[id] * scale + pos_table[position] in fp32, the same in the table's dtype)."""
    if _use_cuda(table):
        return cuda_ops().embed_stream(ids, positions, table, pos_table, scale)
    return ref.embed_stream(ids, positions, table, pos_table, scale)


def post_norm_add(x, y, weight, eps, gemma=False, next_weight=None, next_gemma=False):
    """In place on the fp32 stream: x += rmsnorm(y) * w.  Returns the next GEMM's input in y's dtype: x, or its norm with
    ``next_weight``."""
    if _use_cuda(x):
        return cuda_ops().post_norm_add(x, y, weight, eps, gemma, next_weight, next_gemma)
    return ref.post_norm_add(x, y, weight, eps, gemma, next_weight, next_gemma)


def norm_add(x, y, y_bias, norm, mult: float, next_norm, eps: float):
    """In place on the fp32 stream: x += mult * norm(y + y_bias), layer norms (weight, bias); ``y_bias`` fp32 or None.  Returns the
    next GEMM's input in y's dtype: next_norm(x), or x where that is None."""
    if _use_cuda(x):
        return cuda_ops().norm_add(x, y, y_bias, norm, mult, next_norm, eps)
    return ref.norm_add(x, y, y_bias, norm, mult, next_norm, eps)


def hyper_entry(ids, table, streams: int, embed_weight, into, weight, eps: float):
    """Entry of ``streams`` equal fp32 streams: (x [T, S, H], rms norm of sum(into) e in the table's dtype), e the rms norm of table[ids],
    or a row of ``table`` where ``ids`` is None."""
    if _use_cuda(table):
        return cuda_ops().hyper_entry(ids, table, streams, embed_weight, into, weight, eps)
    return ref.hyper_entry(ids, table, streams, embed_weight, into, weight, eps)


def hyper_step(x, y, coef, into, weight, eps: float, dtype=None):
    """Hyper-connections, one step of S fp32 streams x [T, S, H] between sublayers: in place x_t = sum_s mix[s, t] x_s + out[t] y (``coef``:
    out [S] and mix [S, S], fp32; y None: unchanged).  Returns the rms norm of sum_s into[s] x_s in ``dtype`` (y's)."""
    if _use_cuda(x):
        return cuda_ops().hyper_step(x, y, coef, into, weight, eps, dtype or y.dtype)
    return ref.hyper_step(x, y, coef, into, weight, eps, dtype or y.dtype)


def xielu(x, coef):
    """a z^2 + z / 2 above zero, b (e^z - 1 - z) + z / 2 below, (a, b) = ``coef`` (fp32)."""
    if _use_cuda(x):
        return cuda_ops().xielu(x, coef)
    return ref.xielu(x, coef)


def linear_xielu(x, weight, bias, coef):
    """xielu(x W^T + b); one kernel for decode batches on CUDA."""
    if _use_cuda(x):
        return cuda_ops().linear_xielu(x, weight, bias, coef)
    return ref.xielu(linear(x, weight, bias), coef)


def add_norm(x, y, next_norm, eps: float, dtype=None):
    """In place on the fp32 stream: x += y.  Returns the next GEMM's input in y's dtype: the layer norm ``next_norm`` (weight, bias or
    None) of x, or x where that is None."""
    if _use_cuda(x):
        return cuda_ops().add_norm(x, y, next_norm, eps)
    return ref.add_norm(x, y, next_norm, eps)


def embed_norm(ids, table, next_norm, eps: float):
    """Entry of an fp32 stream in front of a normed sublayer: (table[ids] fp32, next_norm of it in the table's dtype)."""
    if _use_cuda(table):
        x = torch.empty((ids.numel(), table.shape[1]), dtype=torch.float32, device=table.device)
        return x, cuda_ops().norm_add(x, table, None, None, 1.0, next_norm, eps, ids=ids)
    x = torch.nn.functional.embedding(ids, table).float()
    return x, ref.layer_norm(x, *next_norm, eps).to(table.dtype)


def scan_state_elems(R: int, C: int) -> int:
    """Floats that a head's [R, C] state takes in a slot: the lane layout of csrc/linear_attn.cu."""
    if not 1 <= R <= 512:
        raise ValueError(f"state of {R} rows: the scan kernels hold up to 512")
    rows = max(16, 1 << (R - 1).bit_length())
    return -(-C // 4) * 4 * rows


def gated_norm(y, z, weight, groups: int, eps: float, gate_first: bool, out=None, scale: float = 1.0, gate: str = "silu"):
    """RMS norm of y (fp32) over equal parts with the gate silu(z) or sigmoid(z) before or behind it; in z's dtype."""
    if _use_cuda(y):
        return cuda_ops().gated_norm(y, z, weight, groups, eps, gate_first, out, scale, gate)
    o = ref.gated_norm(y, z, weight, groups, eps, gate_first, gate) * scale
    return o.to(z.dtype) if out is None else out.copy_(o)


def merge_attn_states(o1, lse1, o2, lse2):
    if _use_cuda(o1):
        return cuda_ops().merge_attn_states(o1, lse1, o2, lse2)
    return ref.merge_attn_states(o1, lse1, o2, lse2)


def linear(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """y = x @ weight.T + bias. CUDA: tcgen05 GEMM for the shapes it covers, else cuBLASLt."""
    if _use_cuda(x):
        return cuda_ops().linear(x, weight, bias)
    return torch.nn.functional.linear(x, weight, bias)


def topk_softmax(gating, k, renormalize):
    if _use_cuda(gating):
        return cuda_ops().topk_softmax(gating, k, renormalize)
    return ref.topk_softmax(gating, k, renormalize)


def grouped_topk(scores, k, n_group, topk_group, renormalize, scoring="sigmoid", bias=None,
                 routed_scaling_factor=1.0, group_score=None):
    """``group_score``: a group is ranked by its two best choice scores ("top2") or its best ("max"); None: by two where there is a bias."""
    if _use_cuda(scores):
        return cuda_ops().grouped_topk(scores, k, n_group, topk_group, renormalize, scoring, bias,
                                       routed_scaling_factor, group_score)
    return ref.grouped_topk(scores, k, n_group, topk_group, renormalize, scoring, bias, routed_scaling_factor, group_score)


def router_topk(x, gate, k, n_group, topk_group, renormalize, scoring="sigmoid", bias=None, routed_scaling_factor=1.0,
                x_half=None, group_score=None):
    """Router with 32-bit logits: (weights fp32 [T, k], ids [T, k]) of x [T, H] (fp32 stream or model dtype) with gate [E, H]."""
    if _use_cuda(x):
        return cuda_ops().router_topk(x, gate, k, n_group, topk_group, renormalize, scoring, bias, routed_scaling_factor, x_half,
                                      group_score)
    return ref.grouped_topk(x.float() @ gate.float().t(), k, n_group, topk_group, renormalize, scoring, bias,
                            routed_scaling_factor, group_score)


def fused_moe(x, w13, w2, topk_w, topk_ids, act="silu", expert_map=None, gated: bool = True, on_device: bool = False):
    """``gated`` False: w13 is the plain up projection [E, I, H].  ``on_device``: never synchronise with the host, at any batch size."""
    if _use_cuda(x):
        return cuda_ops().fused_moe(x, w13, w2, topk_w, topk_ids, act, expert_map, gated, on_device)
    return ref.fused_moe(x, w13, w2, topk_w, topk_ids, act, expert_map, gated)


def fused_moe_post_norm(stream, x, w_up, w_down, topk_w, topk_ids, act, expert_map, weight, eps, gemma=False, next_weight=None,
                        next_gemma=False):
    """post_norm_add of the routed sum of ungated experts; on CUDA the combine is the load of that kernel."""
    if _use_cuda(x):
        from vllm_b200.ops.moe import expert_rows_plain
        rows, inv = expert_rows_plain(x, w_up, w_down, topk_ids, act, expert_map)
        return cuda_ops().post_norm_add(stream, rows, weight, eps, gemma, next_weight, next_gemma, inv,
                                        topk_w.to(torch.float32).contiguous())
    return ref.post_norm_add(stream, ref.fused_moe(x, w_up, w_down, topk_w, topk_ids, act, expert_map, False), weight, eps, gemma,
                             next_weight, next_gemma)


def fused_moe_add_norm(stream, x, w13, w2, topk_w, topk_ids, act, expert_map, gated: bool, experts: int, y, next_norm, eps: float):
    """add_norm of the routed sum (identity experts: numbers from ``experts`` on add their weight times x) plus ``y`` (or None); on CUDA
    the combine is the load of that kernel."""
    if _use_cuda(x):
        from vllm_b200.ops.moe import expert_rows
        ids = topk_ids if topk_ids.dtype == torch.int32 else topk_ids.to(torch.int32)
        rows, inv = expert_rows(x, w13, w2, ids, act, expert_map, gated)
        return cuda_ops().add_norm(stream, y, next_norm, eps, x.dtype, rows, inv, topk_w.to(torch.float32).contiguous(), ids, experts,
                                   x if expert_map is not None and expert_map.numel() > experts else None)
    out = ref.fused_moe(x, w13, w2, topk_w, topk_ids, act, expert_map, gated) + ref.identity_experts(x, topk_w, topk_ids, experts)
    return ref.add_norm(stream, out if y is None else out + y, next_norm, eps)


def block_fp8_linear(x, wq, w_scale, block=128, bias=None):
    if _use_cuda(x):
        return cuda_ops().block_fp8_linear(x, wq, w_scale, block, bias)
    return ref.block_fp8_linear(x, wq, w_scale, block, bias)


# -- quantisers, q/k-norm + RoPE, cache maintenance: CUDA kernels (csrc/quant.cu, qknorm_rope.cu, cache_ops.cu), fp32
#    PyTorch reference on the CPU
def scaled_fp8_quant(x, scale=None, per_token: bool = False):
    if _use_cuda(x) and x.dtype in (torch.bfloat16, torch.float16) and x.shape[-1] % 8 == 0:
        return cuda_ops().scaled_fp8_quant(x, scale, per_token)
    return ref.scaled_fp8_quant(x, scale, per_token)


def scaled_int8_quant(x, scale=None):
    if _use_cuda(x) and x.dtype in (torch.bfloat16, torch.float16) and x.shape[-1] % 8 == 0:
        return cuda_ops().scaled_int8_quant(x, scale)
    return ref.scaled_int8_quant(x, scale)


def per_token_group_quant_fp8(x, group: int = 128, col_major: bool = False, ue8m0: bool = False):
    if _use_cuda(x) and x.dtype in (torch.bfloat16, torch.float16):
        return cuda_ops().per_token_group_quant_fp8(x, group, col_major, ue8m0)
    return ref.per_token_group_quant_fp8(x.reshape(-1, x.shape[-1]), group)


def rms_norm_quant(x, weight, eps, *, residual=None, scale=None, mode: str = "static", group: int = 128,
                   gemma: bool = False):
    """(residual add +) RMSNorm + fp8 quant in one pass; returns (q, scale) and updates ``residual`` in place."""
    if _use_cuda(x) and x.dtype in (torch.bfloat16, torch.float16) and x.shape[-1] % 8 == 0:
        return cuda_ops().rms_norm_quant(x, weight, eps, residual=residual, scale=scale, mode=mode, group=group,
                                         gemma=gemma)
    if residual is not None:
        y, _ = ref.fused_add_rms_norm(x, residual, weight, eps, gemma)
    else:
        y = ref.rms_norm(x, weight, eps, gemma)
    if mode == "group":
        return ref.per_token_group_quant_fp8(y.reshape(-1, y.shape[-1]), group)
    return ref.scaled_fp8_quant(y, scale, per_token=(mode == "token"))


def act_mul_quant(x, act: str = "silu", *, scale=None, mode: str = "static", group: int = 128):
    if _use_cuda(x) and x.dtype in (torch.bfloat16, torch.float16) and x.shape[-1] % 16 == 0:
        return cuda_ops().act_mul_quant(x, act, scale=scale, mode=mode, group=group)
    y = ref.silu_and_mul(x) if act == "silu" else ref.gelu_and_mul(x, "tanh" if "tanh" in act else "none")
    if mode == "group":
        return ref.per_token_group_quant_fp8(y.reshape(-1, y.shape[-1]), group)
    return ref.scaled_fp8_quant(y, scale, per_token=(mode == "token"))


def fused_qk_norm_rope(positions, q, k, q_weight, k_weight, cos_sin_cache, head_dim, eps, is_neox=True, **kw):
    if _use_cuda(q) and q.dtype in (torch.bfloat16, torch.float16) and cuda_ops().qknorm_rope_ok(
            head_dim, cos_sin_cache.shape[-1] if cos_sin_cache is not None else 0, is_neox):
        return cuda_ops().fused_qk_norm_rope(positions, q, k, q_weight, k_weight, cos_sin_cache, head_dim, eps, is_neox,
                                             **kw)
    q, k = ref.fused_qk_norm_rope(positions, q, k, q_weight, k_weight, cos_sin_cache, head_dim, eps, is_neox)
    if kw.get("kv_cache") is not None:
        v = kw["v"]
        Hkv = k.shape[-1] // head_dim
        reshape_and_cache(k.reshape(-1, Hkv, head_dim), v.reshape(-1, Hkv, head_dim), kw["kv_cache"],
                          kw["slot_mapping"], vt=kw.get("vt", False))
    return q, k


def swap_blocks(src, dst, mapping) -> None:
    if (src.is_cuda or dst.is_cuda) and not envs.VLLM_B200_FORCE_REF_OPS and (src.is_cuda or src.is_pinned()) \
            and (dst.is_cuda or dst.is_pinned()) and (src[0].numel() * src.element_size()) % 16 == 0 \
            and src.is_contiguous() and dst.is_contiguous() and src.dtype == dst.dtype:
        return cuda_ops().swap_blocks(src, dst, mapping)
    return ref.swap_blocks(src, dst, mapping if not isinstance(mapping, torch.Tensor) else mapping.tolist())


def convert_fp8(x, scale: float = 1.0, to_fp8: bool = True):
    if _use_cuda(x) and (x.dtype in (torch.bfloat16, torch.float16) or not to_fp8):
        return cuda_ops().convert_fp8(x, scale, to_fp8)
    return ref.convert_fp8(x, scale, to_fp8)


def scaled_fp4_quant(x, global_scale=None, mx: bool = False):
    if _use_cuda(x) and x.dtype in (torch.bfloat16, torch.float16) and x.shape[-1] % 32 == 0:
        return cuda_ops().scaled_fp4_quant(x, global_scale, mx)
    raise NotImplementedError("fp4 activation quantisation runs on the device only")


def scaled_mm(a, b, scale_a, scale_b, out_dtype, bias=None):
    """W8A8: (a · bᵀ) * scale_a * scale_b (+bias).  fp8 operands run on the tcgen05 f8f6f4 kernel."""
    if _use_cuda(a):
        return cuda_ops().scaled_mm(a, b, scale_a, scale_b, out_dtype, bias)
    return ref.scaled_mm(a, b, scale_a, scale_b, out_dtype, bias)


# -- ops served by the PyTorch implementations on every device (elementwise / bookkeeping)
mul_and_silu = ref.mul_and_silu
fatrelu_and_mul = ref.fatrelu_and_mul
swigluoai_and_mul = ref.swigluoai_and_mul
fp4_dequant = ref.fp4_dequant
