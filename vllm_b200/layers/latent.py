"""Latent attention, in two forms of its projections.

With a query latent and no rotated part:

    [c_q | c_kv] = W_down h          one GEMM; both halves are RMS-normed, c_kv is what the cache holds
    q = W_uq c_q                     per head: k = W_uk c_kv, v = W_uv c_kv, score = (q . k) * scale
    out = W_o concat(heads)

With direct queries, a rotated part, a window and an output gate (the last three optional):

    [q | g | c_kv | k_r] = W_in h    one GEMM; c_kv is RMS-normed, k_r and the last part q_r of every query head are rotated
    score = (q_n . W_uk c_kv + q_r . k_r) * scale        over the window's keys; k_r is one for all heads
    out = W_o (concat(heads) * sigmoid(g))

Only c_kv (and k_r) are cached (``MLAAttentionCore``), and a layer may own no latent at all and read an earlier layer's
(``kv_sharing_target``) with its own W_uk and W_uv.

Two forms of the same attention serve a step.  *Absorbed* (decode): q is taken into the latent space by W_uk, every head
attends over the latent rows themselves, W_uv maps the result back — nothing but the latents is read.  *Expanded*
(prompt portions): keys and values of the portion's whole context are written out by two GEMMs and a multi-head kernel
runs over them — a score costs ``dim`` multiplications instead of the latent width.  A mixed step is split between the
two by the length of each request's portion, once per step (``LatentPlan``), whatever the batch looks like otherwise.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import numpy as np
import torch
import torch.nn as nn

from vllm_b200 import ops
from vllm_b200.forward_context import AttentionMetadata, get_forward_context
from vllm_b200.layers.attention import MLAAttentionCore
from vllm_b200.layers.common import RMSNorm
from vllm_b200.layers.linear import (ColumnParallelLinear, MergedColumnParallelLinear, MergedMixedLinear, MergedReplicatedLinear,
                                      RowParallelLinear)
from vllm_b200.parallel.state import get_dcp_group, get_tp_group
from vllm_b200.parallel.utils import divide

# portions of at most this many tokens attend in the latent space, one row per token: re-reading the context that often is
# still cheaper than writing its keys and values out
ABSORB_MAX_TOKENS = 16
# bytes of expanded keys and values held at a time; a longer context is done a few heads at a time
EXPAND_BYTES = 1 << 30


@dataclass
class LatentPlan:
    """Device-side index arrays of one step (int32 / int64), shared by all its layers of one window."""
    rows: Optional[torch.Tensor] = None        # absorbed: token rows (None: every token of the step)
    row_block_table: Optional[torch.Tensor] = None
    row_seq_lens: Optional[torch.Tensor] = None
    num_rows: int = 0
    max_row_len: int = 0
    block_table: Optional[torch.Tensor] = None  # expanded: one entry per request
    q_start: Optional[torch.Tensor] = None
    q_len: Optional[torch.Tensor] = None
    seq_len: Optional[torch.Tensor] = None     # keys of each request that some row of its portion sees
    kv_first: Optional[torch.Tensor] = None    # position of the first of them (None: all start at 0)
    cu_kv: Optional[torch.Tensor] = None       # [n + 1] key rows before each request
    num_kv: int = 0
    max_q: int = 0
    max_kv: int = 0

    @classmethod
    def of(cls, md: AttentionMetadata, device: torch.device, window: int) -> "LatentPlan":
        plans = md.latent_plan = md.latent_plan if md.latent_plan is not None else {}
        if window not in plans:
            plans[window] = cls.build(md, device, window)
        return plans[window]

    @classmethod
    def build(cls, md: AttentionMetadata, device: torch.device, window: int = 0) -> "LatentPlan":
        if md.host_lens is not None:
            cu, sl = md.host_lens
        else:
            cu, sl = md.query_start_loc.cpu().numpy(), md.seq_lens.cpu().numpy()
        cu, sl = np.asarray(cu, dtype=np.int64), np.asarray(sl, dtype=np.int64)
        ql = cu[1:] - cu[:-1]
        sl = sl[:len(ql)]
        short = np.nonzero((ql > 0) & (ql <= ABSORB_MAX_TOKENS))[0]
        long = np.nonzero(ql > ABSORB_MAX_TOKENS)[0]
        n_rows, n = int(ql[short].sum()), len(long)
        # token row, request and number of visible keys of every absorbed row
        req = np.repeat(short, ql[short])
        first = np.repeat(np.cumsum(ql[short]) - ql[short], ql[short])
        off = np.arange(n_rows) - first
        vis = sl[req] - ql[req] + off + 1
        kv_first = np.maximum(sl[long] - ql[long] + 1 - window, 0) if window else np.zeros(n, dtype=np.int64)
        kl = sl[long] - kv_first
        cu_kv = np.concatenate([[0], np.cumsum(kl)])
        parts = [cu[req] + off, req, vis, long, cu[long], ql[long], kl, kv_first, cu_kv]
        packed = torch.from_numpy(np.concatenate(parts).astype(np.int32)).to(device, non_blocking=True)
        rows, req_t, vis_t, long_t, q_start, q_len, seq_len, first_t, cu_t = packed.split([len(p) for p in parts])
        plan = cls(num_rows=n_rows)
        if n_rows:
            plan.rows = rows.long() if n else None
            plan.row_block_table = md.block_table.index_select(0, req_t)
            plan.row_seq_lens = vis_t
            plan.max_row_len = int(vis.max())
        if n:
            plan.block_table = md.block_table.index_select(0, long_t)
            plan.q_start, plan.q_len, plan.seq_len, plan.cu_kv = q_start, q_len, seq_len, cu_t
            plan.kv_first = first_t if kv_first.any() else None
            plan.num_kv, plan.max_q, plan.max_kv = int(cu_kv[-1]), int(ql[long].max()), int(kl.max())
        return plan


class LatentAttention(nn.Module):
    def __init__(self, hidden_size: int, num_heads: int, dim: int, v_dim: int, q_rank: int, kv_rank: int, scale: float, eps: float,
                 dtype=None, quant_config=None, prefix: str = "", kv_sharing_target: Optional[str] = None, rope: Optional[nn.Module] = None,
                 window: int = 0, cache_window: int = 0, gated: bool = False) -> None:
        """``q_rank`` 0: direct queries, with the parts that ``rope`` (its width is that of the rotated part), ``window`` and ``gated`` name;
        ``cache_window``: how long pages stay (``MLAAttentionCore``)."""
        super().__init__()
        if get_dcp_group().world_size > 1:
            raise NotImplementedError("decode context parallelism with this form of latent attention")
        if q_rank and (rope is not None or window or gated):
            raise NotImplementedError("a query latent beside a rotated part, a window or a gate")
        self.heads = divide(num_heads, get_tp_group().world_size)
        self.dim, self.v_dim, self.q_rank, self.kv_rank = dim, v_dim, q_rank, kv_rank
        self.rope, self.rot, self.window = rope, 0 if rope is None else rope.rotary_dim, window
        self.scale, self.eps = float(scale), eps
        self.owns_latent = kv_sharing_target is None
        self.kv_norm = RMSNorm(kv_rank, eps, dtype) if self.owns_latent else None
        if q_rank:
            self.down = MergedReplicatedLinear(hidden_size, [q_rank, kv_rank] if self.owns_latent else [q_rank], False, dtype,
                                               quant_config, f"{prefix}.down")
            self.q_norm = RMSNorm(q_rank, eps, dtype)
            self.uq = ColumnParallelLinear(q_rank, num_heads * dim, False, dtype=dtype, quant_config=quant_config,
                                           prefix=f"{prefix}.uq")
        else:
            parts = [(num_heads * (dim + self.rot), True, "q")] + ([(num_heads * v_dim, True, "g")] if gated else []) + (
                [(kv_rank + self.rot, False, "kv")] if self.owns_latent else [])
            self.part = {name: i for i, (_, _, name) in enumerate(parts)}
            self.in_proj = MergedMixedLinear(hidden_size, [p[0] for p in parts], [p[1] for p in parts], False, dtype, quant_config,
                                             f"{prefix}.in_proj", align=8)
        # kept unquantised: consumed as batched absorbed matrices too, not only as a GEMM weight
        self.ukv = MergedColumnParallelLinear(kv_rank, [num_heads * dim, num_heads * v_dim], False, dtype, None, f"{prefix}.ukv")
        self.o = RowParallelLinear(num_heads * v_dim, hidden_size, False, dtype=dtype, quant_config=quant_config,
                                   prefix=f"{prefix}.o")
        self.attn = MLAAttentionCore(self.heads, kv_rank, self.rot, self.scale, prefix=f"{prefix}.attn",
                                     kv_sharing_target=kv_sharing_target, sliding_window=window or None,
                                     cache_window=cache_window or None)

    def _up(self) -> tuple[torch.Tensor, torch.Tensor]:
        """(W_uk [h, dim, R], W_uv [h, v_dim, R]): views of the stacked weight."""
        w, n = self.ukv.weight, self.heads * self.dim
        return w[:n].view(self.heads, self.dim, self.kv_rank), w[n:].view(self.heads, self.v_dim, self.kv_rank)

    def forward(self, h: torch.Tensor, positions: Optional[torch.Tensor] = None) -> torch.Tensor:
        T = h.shape[0]
        md, cache = self.attn.bound_cache()
        gate = None
        if self.q_rank:
            lat = self.down(h)
            if self.owns_latent:
                c_q, c_kv = ops.latent_norm_cache(lat, self.q_rank, self.q_norm.weight, self.kv_rank, self.kv_norm.weight, self.eps,
                                                  cache, None if md is None else md.slot_mapping)
            else:
                c_q, c_kv = ops.latent_norm_cache(lat, self.q_rank, self.q_norm.weight, 0, None, self.eps)
            q = self.uq(c_q).view(T, self.heads, self.dim)
        else:
            proj = self.in_proj(h)
            parts = self.in_proj.parts(proj)
            own = self.owns_latent
            if self.rot or own:
                ops.latent_rope_cache(proj, 0, self.heads, self.dim, self.rot, self.in_proj.offsets[self.part["kv"]] if own else 0,
                                      self.kv_rank if own else 0, self.kv_norm.weight if own else None, self.eps, positions,
                                      None if self.rope is None else self.rope.cos_sin_cache,
                                      self.rope is not None and self.rope.is_neox_style, cache if own else None,
                                      md.slot_mapping if own and md is not None else None)
            q = parts[0].view(T, self.heads, self.dim + self.rot)
            gate = parts[self.part["g"]] if "g" in self.part else None
            c_kv = parts[self.part["kv"]][:, :self.kv_rank] if own else None
        if md is None:
            # memory-profiling run: hold what expanding a batch of prompts would
            if c_kv is not None:
                self.ukv(c_kv)
            return self.o(q.new_zeros(T, self.heads * self.v_dim))
        o = self._attend(q, md, cache).view(T, self.heads * self.v_dim)
        return self.o(o if gate is None else ops.sigmoid_mul_(o, gate))

    def _attend(self, q: torch.Tensor, md: AttentionMetadata, cache: torch.Tensor) -> torch.Tensor:
        T = q.shape[0]
        out = torch.empty(T, self.heads, self.v_dim, dtype=q.dtype, device=q.device)
        window = self.window or None
        if md.decode_only or not ops.latent_expand_ok(q, self.dim, self.rot, self.v_dim, self.kv_rank):
            return self._absorbed(q, out, lambda q_abs, q_pe: ops.mla_attention(q_abs, q_pe, cache, md, self.scale, self.kv_rank, window))
        plan = LatentPlan.of(md, q.device, self.window)
        if plan.num_rows:
            def attend(q_abs, q_pe):
                return ops.mla_attention_rows(q_abs, q_pe, cache, plan.row_block_table, plan.row_seq_lens, plan.max_row_len,
                                              self.scale, window)
            if plan.rows is None:
                return self._absorbed(q, out, attend)
            part = torch.empty(plan.num_rows, self.heads, self.v_dim, dtype=q.dtype, device=q.device)
            out.index_copy_(0, plan.rows, self._absorbed(q.index_select(0, plan.rows), part, attend))
        self._expanded(q, out, plan, cache)
        return out

    def _absorbed(self, q: torch.Tensor, out: torch.Tensor, attend) -> torch.Tensor:
        w_uk, w_uv = self._up()
        q_abs = torch.bmm(q[..., :self.dim].transpose(0, 1), w_uk).transpose(0, 1)   # [T, h, R], head-major in memory
        o_lat = attend(q_abs, q[..., self.dim:] if self.rot else None)
        torch.bmm(o_lat.transpose(0, 1), w_uv.transpose(1, 2), out=out.transpose(0, 1))
        return out

    def _expanded(self, q: torch.Tensor, out: torch.Tensor, plan: LatentPlan, cache: torch.Tensor) -> None:
        # layers that share a cache (and see as much of it) share the gathered rows too
        gathered = get_forward_context().extra.setdefault("latent_rows", {})
        key = self.attn.cache_name, self.window
        rows = gathered.get(key)
        if rows is None:
            rows = gathered[key] = ops.gather_latents(cache, plan.block_table, plan.cu_kv, plan.num_kv, plan.max_kv, plan.kv_first)
        c = rows[:, :self.kv_rank]
        w_uk, w_uv = self._up()
        per_head = plan.num_kv * (self.dim + self.v_dim) * q.element_size()
        step = max(1, min(self.heads, EXPAND_BYTES // max(per_head, 1)))
        for h0 in range(0, self.heads, step):
            h1 = min(self.heads, h0 + step)
            k = ops.linear(c, w_uk[h0:h1].reshape(-1, self.kv_rank)).view(plan.num_kv, h1 - h0, self.dim)
            v = ops.linear(c, w_uv[h0:h1].reshape(-1, self.kv_rank)).view(plan.num_kv, h1 - h0, self.v_dim)
            ops.mla_prefill(q, k, v, out, plan.q_start, plan.q_len, plan.seq_len, plan.cu_kv, h0, plan.max_q, self.scale,
                            rows[:, self.kv_rank:] if self.rot else None, self.window)
