"""Gated linear attention with a per-request state slot.

    S_t = diag(a_t) S_{t-1} + k_t v_t^T        a_t = sigmoid(W_2 W_1 h_t + b)^(1 / tau), a decay per key channel
    o_t = S_t^T q_t                            RMS norm per head, then the gate silu(g_t)

The projections of the layer's input (q, k, v, the gate and the decay's low-rank half) are one GEMM.  On CUDA the second half of
the decay, the recurrence and the state update are ``csrc/linear_attn.cu`` (prompts, portions and decode steps alike; the
state is advanced in its slot), and the norm with the gate is one more kernel.
"""
from __future__ import annotations

import torch
import torch.nn as nn

from vllm_b200 import ops
from vllm_b200.core.kv_cache_manager import KVCacheSpec, MambaSpec
from vllm_b200.forward_context import get_forward_context
from vllm_b200.layers import attention as _attn
from vllm_b200.layers.linear import MergedReplicatedLinear, ReplicatedLinear


class GatedLinearAttention(nn.Module):
    def __init__(self, hidden: int, num_heads: int, dim: int, vdim: int, rank: int, tau: float, eps: float, dtype, prefix: str) -> None:
        super().__init__()
        self.nh, self.dk, self.dv = num_heads, dim, vdim
        self.tau, self.eps, self.q_scale = float(tau), eps, dim ** -0.5
        qk, v = num_heads * dim, num_heads * vdim
        self.in_proj = MergedReplicatedLinear(hidden, [qk, qk, v, v, rank], False, dtype, None, f"{prefix}.in_proj", align=8)
        self.a2 = nn.Parameter(torch.zeros(qk, rank, dtype=dtype), requires_grad=False)
        self.a2_bias = nn.Parameter(torch.zeros(qk, dtype=dtype), requires_grad=False)
        self.norm_weight = nn.Parameter(torch.ones(vdim, dtype=dtype), requires_grad=False)      # shared by the heads
        self.out_proj = ReplicatedLinear(v, hidden, False, dtype, None, f"{prefix}.out_proj")
        self.layer_name = prefix
        self.state_elems = num_heads * ops.scan_state_elems(dim, vdim)
        self.num_kv_heads, self.head_size, self.sliding_window = 1, 0, None
        assert prefix not in _attn._LAYER_REGISTRY, f"duplicate layer name {prefix}"
        _attn._LAYER_REGISTRY[prefix] = self

    def get_kv_cache_spec(self, block_size: int, dtype_size: int) -> KVCacheSpec:
        return MambaSpec(block_size=block_size, state_bytes=self.state_elems * 4)

    def forward(self, hidden: torch.Tensor) -> torch.Tensor:
        q, k, v, g, a1 = self.in_proj.parts(self.in_proj(hidden))
        o = self._recur(q, k, v, a1)
        return self.out_proj(ops.gated_norm(o, g, self.norm_weight, self.nh, self.eps, gate_first=False))

    def _recur(self, q, k, v, a1) -> torch.Tensor:
        """[T, heads * vdim] fp32."""
        ctx = get_forward_context()
        md = ctx.metadata_for(self.layer_name)
        cache = ctx.kv_caches.get(self.layer_name)
        T = q.shape[0]
        if md is None or cache is None:                      # profiling run: no state
            return torch.zeros(T, self.nh * self.dv, dtype=torch.float32, device=q.device)
        if ops._use_cuda(q):
            return ops.cuda_ops().gla_scan(q, k, v, a1, self.a2, self.a2_bias, self.tau, self.q_scale, cache, md,
                                           self.nh, self.dk, self.dv)
        from vllm_b200.ops import ref
        z = a1.float() @ self.a2.float().t() + self.a2_bias.float()
        alpha = torch.exp(torch.nn.functional.logsigmoid(z) / self.tau).view(T, self.nh, self.dk)
        q, k = (q.float() * self.q_scale).reshape(T, self.nh, self.dk), k.float().reshape(T, self.nh, self.dk)
        v = v.float().reshape(T, self.nh, self.dv)
        qsl = (md.query_start_loc_cpu if md.query_start_loc_cpu is not None else md.query_start_loc.cpu()).tolist()
        sls = (md.seq_lens_cpu if md.seq_lens_cpu is not None else md.seq_lens.cpu()).tolist()
        slots = md.block_table[:md.num_reqs, 0].tolist()
        n = self.nh * self.dk * self.dv
        o = torch.zeros(T, self.nh, self.dv, dtype=torch.float32, device=q.device)
        for i in range(md.num_reqs):
            s, e = qsl[i], qsl[i + 1]
            if e <= s:
                continue
            state = cache[slots[i], :n].reshape(self.nh, self.dk, self.dv)
            if sls[i] == e - s:
                state = torch.zeros_like(state)
            o[s:e], state = ref.gated_linear_scan(q[s:e], k[s:e], v[s:e], alpha[s:e], state)
            cache[slots[i], :n] = state.reshape(-1)
        return o.reshape(T, self.nh * self.dv)
