"""Paged attention layer.

Behavioural reference: vllm/model_executor/layers/attention/attention.py:218
(``Attention.forward`` :478-571 = KV-cache update + unified attention op,
``get_kv_cache_spec`` :597).  Here the layer owns a fused
RoPE + KV-write + attention call sequence over our own cache layout
``[num_blocks, 2, Hkv, block_size, D]``.
"""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn as nn

from vllm_b200 import envs, ops
from vllm_b200.core.kv_cache_manager import (FullAttentionSpec, KVCacheSpec, MLAAttentionSpec, SlidingWindowMLASpec,
                                            SlidingWindowSpec)
from vllm_b200.forward_context import get_forward_context

_LAYER_REGISTRY: dict[str, "Attention"] = {}


def attention_layers() -> dict[str, "Attention"]:
    return _LAYER_REGISTRY


def clear_attention_layers() -> None:
    _LAYER_REGISTRY.clear()


class Attention(nn.Module):
    cascade_calls = 0          # how many layer invocations took the cascade path (tests / debugging)

    def __init__(self, num_heads: int, head_size: int, scale: float, num_kv_heads: Optional[int] = None,
                 sliding_window: Optional[int] = None, logits_soft_cap: float = 0.0, prefix: str = "",
                 causal: bool = True, rope: Optional[nn.Module] = None,
                 alibi_slopes: Optional[torch.Tensor] = None, sinks: Optional[torch.Tensor] = None,
                 chunk_size: int = 0, v_head_size: Optional[int] = None, fused_prologue: bool = False,
                 out_scale: float = 1.0, whole_qk_norm: bool = False, kv_sharing_target: Optional[str] = None,
                 talk: Optional[torch.Tensor] = None, v_rope: Optional[nn.Module] = None, cache_window: Optional[int] = None) -> None:
        """``v_head_size``: value width where it is not ``head_size`` (cache rows are as wide as the wider one).
        ``fused_prologue``: q/k norms, rotation and cache write are one kernel for whatever shape and dtype, 32-bit between norm
        and rotation.  ``out_scale``: factor of the output, applied in 32-bit.  ``whole_qk_norm``: the q/k norms go over all heads of
        the projection at once (weights as long).  ``kv_sharing_target``: name of an earlier layer whose cache this one reads (it owns
        none, writes nothing and is called without keys and values).  ``talk`` [Hq, Hq]: the heads' weights are mixed by it behind the
        softmax, head h then applies sum_g talk[h, g] weights_g to the values of its own KV head (a parameter of the model).  ``v_rope``:
        values are rotated by their position before they are cached, outputs turned back by that of the query.  ``cache_window``: pages
        stay for this many tokens (layers of different windows then share pages and a block table), at least ``sliding_window``."""
        super().__init__()
        self.talk, self.v_rope = talk, v_rope
        self.cache_window = max(cache_window or 0, sliding_window) if sliding_window else None
        if (talk is not None or v_rope is not None) and (kv_sharing_target is not None or not causal or not fused_prologue):
            raise NotImplementedError("mixed heads and rotated values take the fused prologue, causal masks and a cache of their own")
        self.whole_qk_norm, self.kv_sharing_target, self.cache_name = whole_qk_norm, kv_sharing_target, kv_sharing_target or prefix
        self.v_head_size = v_head_size or head_size
        self.cache_head_size = max(head_size, self.v_head_size)
        self.fused_prologue, self.out_scale = fused_prologue, float(out_scale)
        self.chunk_size = int(chunk_size or 0)        # chunked-local attention (Llama-4 rope layers)
        # ALiBi slopes / attention-sink logits of THIS rank's heads (buffers follow the module's device)
        self.register_buffer("alibi_slopes", None if alibi_slopes is None else alibi_slopes.float(), persistent=False)
        # nn.Parameter owned by the model (loaded from the checkpoint), or constants
        if sinks is None or isinstance(sinks, nn.Parameter):
            self.sinks = sinks
        else:
            self.register_buffer("sinks", sinks.float(), persistent=False)
        self.num_heads, self.head_size, self.scale = num_heads, head_size, scale
        self.num_kv_heads = num_kv_heads or num_heads
        self.sliding_window = sliding_window
        self.logits_soft_cap = logits_soft_cap
        self.causal = causal
        self.layer_name = prefix
        self.rope = rope
        if kv_sharing_target is not None:
            owner = _LAYER_REGISTRY.get(kv_sharing_target)
            if not isinstance(owner, Attention) or (owner.num_heads, owner.num_kv_heads, owner.head_size, owner.v_head_size) != (
                    self.num_heads, self.num_kv_heads, head_size, self.v_head_size):
                raise ValueError(f"layer {prefix!r} shares the cache of {kv_sharing_target!r}, which is not an earlier attention layer "
                                 "of the same head shapes on this rank")
            return
        assert prefix not in _LAYER_REGISTRY, f"duplicate attention layer name {prefix}"
        _LAYER_REGISTRY[prefix] = self

    def get_kv_cache_spec(self, block_size: int, dtype_size: int) -> KVCacheSpec:
        from vllm_b200.parallel.state import get_dcp_group
        d = get_dcp_group().world_size
        if d > 1:
            if self.whole_qk_norm or self.talk is not None or self.v_rope is not None:
                raise NotImplementedError("decode context parallelism does not cover norms over whole projections, mixed heads and "
                                          "rotated values")
            if self.sliding_window or self.alibi_slopes is not None or self.sinks is not None or self.chunk_size:
                raise NotImplementedError("decode context parallelism covers full causal attention (no sliding window / "
                                          "ALiBi / sinks / chunked-local layers)")
            return FullAttentionSpec(block_size=block_size * d, num_kv_heads=self.num_kv_heads, head_size=self.cache_head_size,
                                     dtype_size=dtype_size, dcp=d)
        cls = SlidingWindowSpec if self.sliding_window else FullAttentionSpec
        return cls(block_size=block_size, num_kv_heads=self.num_kv_heads, head_size=self.cache_head_size,
                   dtype_size=dtype_size, sliding_window=self.cache_window)

    def _forward_dcp(self, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, positions, md, kv_cache) -> torch.Tensor:
        """Decode context parallelism for GQA / MQA caches (reference: config/parallel.py:342-388, v1/attention/ops/dcp.py:
        241-338).  It applies where tensor parallelism REPLICATES KV heads (tp > num_kv_heads): the d ranks that hold
        replicas of the same heads stop storing the same tokens d times and shard the cache by position instead (token p
        lives on rank p % d), so the group holds d x more context.  Per step: the ranks all-gather their query heads, each
        attends over its shard of the *previous* context for all of them, the partial results are merged by their
        log-sum-exp across the group; the tokens of the current step are attended locally (their K / V were just computed
        on every rank)."""
        from vllm_b200.ops import ref
        from vllm_b200.parallel.state import get_dcp_group
        g = get_dcp_group()
        d, r = g.world_size, g.rank_in_group
        T, D, h, hkv = q.shape[0], self.head_size, self.num_heads, self.num_kv_heads
        if self.rope is not None and positions is not None:
            q, k = self.rope(positions, q, k)
        k3, v3 = k.reshape(T, hkv, D), v.reshape(T, hkv, D)
        ops.reshape_and_cache(k3, v3, kv_cache, md.slot_mapping)               # positions owned elsewhere carry slot -1
        q3 = q.reshape(T, h, D)
        # gathered query heads: [T, d, hkv, h/hkv, D] → regrouped so that the heads of one KV head stay contiguous
        q_all = g.all_gather(q3.reshape(T, 1, hkv, h // hkv, D).contiguous(), dim=1)
        q_all = q_all.permute(0, 2, 1, 3, 4).reshape(T, d * h, D)
        qsl = (md.query_start_loc_cpu if md.query_start_loc_cpu is not None else md.query_start_loc.cpu()).tolist()
        sls = (md.seq_lens_cpu if md.seq_lens_cpu is not None else md.seq_lens.cpu()).tolist()
        bs = kv_cache.shape[3]
        o_ctx = torch.zeros(T, d * h, D, dtype=torch.float32, device=q.device)
        lse_ctx = torch.full((T, d * h), float("-inf"), dtype=torch.float32, device=q.device)
        o_new = torch.zeros(T, h, D, dtype=torch.float32, device=q.device)
        lse_new = torch.full((T, h), float("-inf"), dtype=torch.float32, device=q.device)
        for i in range(md.num_reqs):
            s, e = qsl[i], qsl[i + 1]
            if e <= s:
                continue
            ctx = sls[i] - (e - s)                                             # positions before this step's tokens
            n_loc = (ctx - r + d - 1) // d if ctx > r else 0                   # ... of which this rank stores n_loc
            if n_loc > 0:
                nb = (n_loc + bs - 1) // bs
                blk = kv_cache[md.block_table[i, :nb].long()]                  # [nb, 2, hkv, bs, D]
                kc = blk[:, 0].permute(0, 2, 1, 3).reshape(nb * bs, hkv, D)[:n_loc]
                vc = blk[:, 1].permute(0, 2, 1, 3).reshape(nb * bs, hkv, D)[:n_loc]
                o_ctx[s:e], lse_ctx[s:e] = ref.partial_attention(q_all[s:e], kc, vc, self.scale, None, self.logits_soft_cap)
            o_new[s:e], lse_new[s:e] = ref.partial_attention(q3[s:e], k3[s:e], v3[s:e], self.scale, 0, self.logits_soft_cap)
        # merge the context partials of the d ranks (softmax-weighted by their lse), keep this rank's heads
        lse_all = g.all_gather(lse_ctx[..., None].contiguous(), dim=-1)       # [T, d*h, d]
        lse_tot = torch.logsumexp(lse_all, dim=-1)
        w = torch.exp(lse_ctx - lse_tot).nan_to_num(0.0)                      # ranks without context contribute 0
        o_all = g.all_reduce((o_ctx * w[..., None]).contiguous())
        mine = o_all.reshape(T, hkv, d, h // hkv, D)[:, :, r].reshape(T, h, D)
        lse_c = lse_tot.reshape(T, hkv, d, h // hkv)[:, :, r].reshape(T, h)
        m = torch.maximum(lse_c, lse_new)
        wc, wn = torch.exp(lse_c - m).nan_to_num(0.0), torch.exp(lse_new - m)
        out = (mine * wc[..., None] + o_new * wn[..., None]) / (wc + wn)[..., None]
        return out.to(q.dtype).reshape(T, h * D)

    def forward(self, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor,
                positions: Optional[torch.Tensor] = None, qk_norm: Optional[tuple] = None,
                out: Optional[torch.Tensor] = None, gate: Optional[torch.Tensor] = None) -> torch.Tensor:
        """``_attend``, then times sigmoid(``gate``) [T, Hq*DV] where given."""
        o = self._attend(q, k, v, positions, qk_norm, out)
        return o if gate is None else ops.sigmoid_mul_(o, gate)

    def _attend(self, q: torch.Tensor, k: Optional[torch.Tensor], v: Optional[torch.Tensor], positions: Optional[torch.Tensor],
                qk_norm: Optional[tuple], out: Optional[torch.Tensor]) -> torch.Tensor:
        """q: [T, Hq*D], k: [T, Hkv*D], v: [T, Hkv*DV] → [T, Hq*DV] (``out``: a buffer for it, any token stride). If the layer has a ``rope``,
        rotation and the KV write happen in one fused kernel.  ``qk_norm`` = (q_norm, k_norm) per-head RMSNorm modules
        (Qwen3 / Gemma-3 / OLMo-2 style; over the whole projections with ``whole_qk_norm``): on CUDA they are fused with the rotation
        and the cache insert into ONE launch (csrc/qknorm_rope.cu), otherwise applied here before the rotation.  k and v are None (and
        so is k_norm) in a layer that reads another layer's cache."""
        ctx = get_forward_context()
        T = q.shape[0]
        D = self.head_size
        md = ctx.metadata_for(self.cache_name)
        kv_cache = ctx.kv_caches.get(self.cache_name)
        shared = self.kv_sharing_target is not None
        if md is not None and kv_cache is None:
            raise RuntimeError(f"attention layer {self.layer_name!r} has no KV cache bound (KV-cache config does not "
                               "cover this worker's layers)")
        if md is None or kv_cache is None:
            # memory-profiling run: no cache; keep the data flow (and the GEMM shapes) intact
            if self.v_head_size != D or out is not None or self.fused_prologue:
                return (q.new_empty(T, self.num_heads * self.v_head_size) if out is None else out).zero_()
            if self.rope is not None and positions is not None:
                q, k = self.rope(positions, q, k)
            return q.clone() if q.shape[-1] == self.num_heads * D else q
        from vllm_b200.parallel.state import get_dcp_group
        if get_dcp_group().world_size > 1:
            if qk_norm is not None:
                qn, kn = qk_norm
                q = qn(q.reshape(T, -1, D)).reshape(T, -1)
                k = kn(k.reshape(T, -1, D)).reshape(T, -1)
            return self._forward_dcp(q, k, v, positions, md, kv_cache)
        pcp = ctx.extra.get("pcp")
        if pcp is not None and (shared or self.whole_qk_norm or self.talk is not None or self.v_rope is not None):
            raise NotImplementedError("prefill context parallelism does not cover shared caches, norms over whole projections, mixed heads "
                                      "and rotated values")
        mpos = ctx.extra.get("mrope_positions") if (self.rope is not None and self.rope.mrope_section) else None
        first = positions
        if qk_norm is not None or self.fused_prologue:
            qn, kn = qk_norm or (None, None)
            fused = (md is not None and kv_cache is not None and q.is_cuda and pcp is None and mpos is None
                     and self.rope is not None and positions is not None
                     and kv_cache.dtype == q.dtype
                     and (shared or qn is None or (getattr(qn, "gemma", False) == getattr(kn, "gemma", False) and qn.eps == kn.eps))
                     and not envs.VLLM_B200_FORCE_REF_OPS
                     and (self.fused_prologue or (q.dtype in (torch.bfloat16, torch.float16) and ops.cuda_ops().qknorm_rope_ok(
                         D, self.rope.cos_sin_cache.shape[-1], self.rope.is_neox_style))))
            if fused:
                ops.cuda_ops().fused_qk_norm_rope(positions, q, k, None if qn is None else qn.weight, None if shared or kn is None else
                                                  kn.weight, self.rope.cos_sin_cache, D, 0.0 if qn is None else qn.eps,
                                                  self.rope.is_neox_style, v=v, kv_cache=None if shared else kv_cache,
                                                  slot_mapping=md.slot_mapping, gemma=getattr(qn, "gemma", False),
                                                  vt=md.kv_vt, v_head_dim=self.v_head_size, keep32=self.fused_prologue,
                                                  whole=self.whole_qk_norm,
                                                  v_cos_sin=None if self.v_rope is None else self.v_rope.cos_sin_cache)
                positions = None            # rotation and cache insert are done: skip them below
                skip_cache_write = True
            else:
                whole = self.whole_qk_norm
                if self.v_rope is not None:
                    v, _ = self.v_rope(positions, v, None)
                if qn is not None:
                    q = qn(q.reshape(T, -1, q.shape[-1] if whole else D)).reshape(T, -1)
                    k = k if shared else kn(k.reshape(T, -1, k.shape[-1] if whole else D)).reshape(T, -1)
                skip_cache_write = False
        else:
            skip_cache_write = False
        if skip_cache_write:
            pass
        elif shared:
            if mpos is not None:
                raise NotImplementedError("shared caches with M-RoPE")
            if self.rope is not None and positions is not None:
                q, _ = self.rope(positions, q, None)
        elif self.v_head_size != D:
            if pcp is not None or mpos is not None:
                raise NotImplementedError("unequal key and value widths with prefill context parallelism or M-RoPE")
            if self.rope is not None and positions is not None:
                q, k = self.rope(positions, q, k)
            wide = [torch.nn.functional.pad(x.reshape(T, self.num_kv_heads, -1), (0, self.cache_head_size - w))
                    for x, w in ((k, D), (v, self.v_head_size))]
            ops.reshape_and_cache(*wide, kv_cache, md.slot_mapping, vt=md.kv_vt)
        elif mpos is not None:
            # multimodal rotary ids differ per channel section for image tokens: rotate un-fused, then the ordinary
            # cache write (text-only steps take the fused path below with 1-D positions = index + per-request delta)
            q, k = self.rope.forward_mrope(mpos, q, k)
            ops.reshape_and_cache(k.view(T, self.num_kv_heads, D), v.view(T, self.num_kv_heads, D), kv_cache,
                                  md.slot_mapping, vt=md.kv_vt)
        elif pcp is not None:
            # prefill context parallelism: this rank holds a share of the step's tokens.  Rotate locally, all-gather
            # K / V of the whole step (global token order) so that every rank's cache stays complete, attend for the
            # local queries only (metadata describes them as the tails of shorter sequences).
            if self.rope is not None and positions is not None:
                q, k = self.rope(positions, q, k)
            Tg = pcp["num_tokens"]
            k_all, v_all = pcp["gather"](k.contiguous()), pcp["gather"](v.contiguous())
            ops.reshape_and_cache(k_all.view(Tg, self.num_kv_heads, D), v_all.view(Tg, self.num_kv_heads, D), kv_cache,
                                  pcp["slot_mappings"][ctx.layer_to_group.get(self.layer_name, 0)], vt=md.kv_vt)
        elif self.rope is not None and positions is not None:
            q, k = ops.rope_and_cache(positions, q, k, v, self.rope.cos_sin_cache, D,
                                      self.rope.is_neox_style, kv_cache, md.slot_mapping, vt=md.kv_vt)
        else:
            ops.reshape_and_cache(k.view(T, self.num_kv_heads, D), v.view(T, self.num_kv_heads, D),
                                  kv_cache, md.slot_mapping, vt=md.kv_vt)
        if (md.cascade is not None and self.causal and not self.sliding_window and self.alibi_slopes is None
                and self.sinks is None and not self.chunk_size and self.v_head_size == D and out is None):
            # shared prefix: its K/V are read once for the whole batch (all queries sit after it → no causal mask),
            # the per-request remainders are attended separately, the two partial softmaxes are merged by their LSE
            md_p, md_s = md.cascade
            q3 = q.view(T, self.num_heads, D)
            o1, l1 = ops.paged_attention(q3, kv_cache, md_p, self.scale, None, self.logits_soft_cap, False, return_lse=True)
            o2, l2 = ops.paged_attention(q3, kv_cache, md_s, self.scale, None, self.logits_soft_cap, True, return_lse=True)
            out, _ = ops.merge_attn_states(o1, l1, o2, l2)
            Attention.cascade_calls += 1
            return out.view(T, self.num_heads * D)
        buf = None if out is None else out.view(T, self.num_heads, self.v_head_size)
        if self.talk is not None or self.v_rope is not None:
            o = ops.talking_attention(q.view(T, self.num_heads, D), kv_cache, md, self.scale, self.sliding_window, self.logits_soft_cap,
                                      self.talk, self.sinks, self.v_head_size, self.v_rope, first, out=buf)
            return o.reshape(T, self.num_heads * self.v_head_size) if out is None else out
        o = ops.paged_attention(q.view(T, self.num_heads, D), kv_cache, md, self.scale,
                                self.sliding_window, self.logits_soft_cap, self.causal, out=buf,
                                alibi_slopes=self.alibi_slopes, sinks=self.sinks, chunk_size=self.chunk_size,
                                v_head_size=self.v_head_size, out_scale=self.out_scale)
        return o.reshape(T, self.num_heads * self.v_head_size) if out is None else out


class MLAAttentionCore(nn.Module):
    """Latent-cache attention core for DeepSeek-style MLA (reference algorithm doc:
    layers/attention/mla_attention.py:1-200). Decode and prefill both run as MQA over
    the 576-d latent (absorbed W_UK / W_UV), which is also what the sm_100 CUTLASS-MLA
    decode kernel in the reference does."""

    def __init__(self, num_heads: int, kv_lora_rank: int, qk_rope_head_dim: int, scale: float,
                 prefix: str = "", kv_sharing_target: Optional[str] = None, sliding_window: Optional[int] = None,
                 cache_window: Optional[int] = None) -> None:
        """``kv_sharing_target``: name of an earlier layer whose cache this one reads (it owns none and writes nothing).
        ``sliding_window``: a query sees that many tokens; pages stay for ``cache_window`` tokens (at least the windows of all layers
        that read them)."""
        super().__init__()
        self.num_heads, self.kv_lora_rank, self.qk_rope_head_dim = num_heads, kv_lora_rank, qk_rope_head_dim
        self.scale = scale
        self.layer_name = prefix
        self.head_size = kv_lora_rank + qk_rope_head_dim
        self.num_kv_heads = 1
        self.sliding_window = sliding_window
        self.cache_window = max(cache_window or 0, sliding_window) if sliding_window else None
        self.kv_sharing_target = kv_sharing_target
        self.cache_name = kv_sharing_target or prefix
        if kv_sharing_target is None:
            _LAYER_REGISTRY[prefix] = self  # type: ignore[assignment]
            return
        owner = _LAYER_REGISTRY.get(kv_sharing_target)
        if not isinstance(owner, MLAAttentionCore) or owner.head_size != self.head_size:
            raise ValueError(f"layer {prefix!r} shares the cache of {kv_sharing_target!r}, which is not an earlier latent "
                             f"cache of width {self.head_size} on this rank")
        if owner.cache_window is not None and (self.cache_window is None or self.cache_window > owner.cache_window):
            raise ValueError(f"layer {prefix!r} reads further back than {kv_sharing_target!r} keeps its pages")

    def get_kv_cache_spec(self, block_size: int, dtype_size: int) -> KVCacheSpec:
        from vllm_b200.parallel.state import get_dcp_group
        d = get_dcp_group().world_size
        if self.cache_window is not None:
            if d > 1:
                raise NotImplementedError("decode context parallelism with windows over latents")
            return SlidingWindowMLASpec(block_size=block_size, head_size=self.head_size, dtype_size=dtype_size,
                                        sliding_window=self.cache_window)
        return MLAAttentionSpec(block_size=block_size * d, head_size=self.head_size, dtype_size=dtype_size, dcp=d)

    def _forward_dcp(self, q_nope_abs, q_pe, kv_c, k_pe, md, kv_cache) -> torch.Tensor:
        """Decode context parallelism (reference: config/parallel.py:342-388, v1/attention/ops/dcp.py): the latent
        cache — identical on every TP rank without DCP — is sharded by position (token p lives on rank p % d), so
        the group holds d x more context.  Queries of all ranks are gathered, every rank attends over its shard of
        the *previous* context, partial results are merged with their log-sum-exp across the group; the tokens of
        the current step are attended locally (their latents were just computed on every rank)."""
        from vllm_b200.ops import ref
        from vllm_b200.parallel.state import get_dcp_group
        g = get_dcp_group()
        d, r = g.world_size, g.rank_in_group
        R = self.kv_lora_rank
        ops.concat_and_cache_mla(kv_c, k_pe, kv_cache, md.slot_mapping)       # non-owned positions carry slot -1
        T, h, _ = q_nope_abs.shape
        qn_all = g.all_gather(q_nope_abs.contiguous(), dim=1)                 # [T, d*h, R]
        qp_all = g.all_gather(q_pe.contiguous(), dim=1)
        qsl = (md.query_start_loc_cpu if md.query_start_loc_cpu is not None else md.query_start_loc.cpu()).tolist()
        sls = (md.seq_lens_cpu if md.seq_lens_cpu is not None else md.seq_lens.cpu()).tolist()
        bs = kv_cache.shape[1]
        o_ctx = torch.zeros(T, d * h, R, dtype=torch.float32, device=q_nope_abs.device)
        lse_ctx = torch.full((T, d * h), float("-inf"), dtype=torch.float32, device=q_nope_abs.device)
        o_new = torch.zeros(T, h, R, dtype=torch.float32, device=q_nope_abs.device)
        lse_new = torch.full((T, h), float("-inf"), dtype=torch.float32, device=q_nope_abs.device)
        new_lat = torch.cat((kv_c, k_pe), dim=-1)
        for i in range(md.num_reqs):
            s, e = qsl[i], qsl[i + 1]
            if e <= s:
                continue
            ctx = sls[i] - (e - s)                                             # positions before this step's tokens
            n_loc = (ctx - r + d - 1) // d if ctx > r else 0                   # ... of which this rank stores n_loc
            if n_loc > 0:
                nb = (n_loc + bs - 1) // bs
                lat = kv_cache[md.block_table[i, :nb].long()].reshape(nb * bs, -1)[:n_loc]
                o_ctx[s:e], lse_ctx[s:e] = ref.mla_partial_attention(qn_all[s:e], qp_all[s:e], lat, self.scale, R)
            o_new[s:e], lse_new[s:e] = ref.mla_partial_attention(q_nope_abs[s:e], q_pe[s:e], new_lat[s:e], self.scale, R,
                                                                 causal_offset=0)
        # merge the context partials of the d ranks: softmax-weighted by their lse
        lse_all = g.all_gather(lse_ctx[..., None].contiguous(), dim=-1)       # [T, d*h, d]
        lse_tot = torch.logsumexp(lse_all, dim=-1)
        w = torch.exp(lse_ctx - lse_tot).nan_to_num(0.0)                      # ranks without context contribute 0
        o_all = g.all_reduce((o_ctx * w[..., None]).contiguous())
        o_c, lse_c = o_all[:, r * h:(r + 1) * h], lse_tot[:, r * h:(r + 1) * h]
        # merge context and current-step parts for this rank's heads
        m = torch.maximum(lse_c, lse_new)
        wc, wn = torch.exp(lse_c - m).nan_to_num(0.0), torch.exp(lse_new - m)
        out = (o_c * wc[..., None] + o_new * wn[..., None]) / (wc + wn)[..., None]
        return out.to(q_nope_abs.dtype)

    def bound_cache(self):
        """(metadata, cache) of this step; (None, None) in a profiling run."""
        ctx = get_forward_context()
        md = ctx.metadata_for(self.cache_name)
        kv_cache = ctx.kv_caches.get(self.cache_name)
        if md is not None and kv_cache is None:
            raise RuntimeError(f"MLA layer {self.layer_name!r} has no KV cache bound")
        return (md, kv_cache) if md is not None else (None, None)

    def forward(self, q_nope_abs: torch.Tensor, q_pe: torch.Tensor, kv_c: torch.Tensor, k_pe: torch.Tensor
                ) -> torch.Tensor:
        md, kv_cache = self.bound_cache()
        if md is None:
            return torch.zeros_like(q_nope_abs)
        from vllm_b200.parallel.state import get_dcp_group
        if get_dcp_group().world_size > 1:
            return self._forward_dcp(q_nope_abs, q_pe, kv_c, k_pe, md, kv_cache)
        ops.concat_and_cache_mla(kv_c, k_pe, kv_cache, md.slot_mapping)
        return ops.mla_attention(q_nope_abs, q_pe, kv_cache, md, self.scale, self.kv_lora_rank)
