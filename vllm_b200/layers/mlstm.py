"""Matrix memory of xLSTM (mLSTM) with a per-request state slot.

    z' = cap tanh(z / cap), z = W h + b per head        i = z'_i (log input gate),  f = log sigmoid(z'_f) (log forget gate)
    m_t = max(f + m_{t-1}, i),  m_0 = 0                 running maximum: S and n are kept divided by exp(m)
    S_t = exp(f + m_{t-1} - m_t) S_{t-1} + exp(i - m_t) k v^T,   n_t likewise with k alone
    o_t = S_t^T q / (max(|n_t . q|, exp(-m_t)) + 1e-6)  RMS norm per head, then the gate sigmoid(W_g h)

The projections of the layer's input (q, k, v and the output gate) are one GEMM; the gates of the recurrence are products of
their own with 32-bit results.  On CUDA the gates, the recurrence (n is one more column of S) and the norm with both divisions
and the gate are a kernel each (``csrc/linear_attn.cu``), for prompts, portions and decode steps alike; the state is advanced
in its slot, ``[S and n per head | m per head]``.
"""
from __future__ import annotations

import torch
import torch.nn as nn

from vllm_b200 import ops
from vllm_b200.core.kv_cache_manager import KVCacheSpec, MambaSpec
from vllm_b200.forward_context import get_forward_context
from vllm_b200.layers import attention as _attn
from vllm_b200.layers.linear import MergedReplicatedLinear, ReplicatedLinear


class MatrixMemory(nn.Module):
    def __init__(self, hidden: int, num_heads: int, dim: int, vdim: int, gate_cap: float, eps: float, dtype, prefix: str) -> None:
        super().__init__()
        self.nh, self.dk, self.dv = num_heads, dim, vdim
        self.cap, self.eps, self.q_scale = float(gate_cap), eps, dim ** -0.5
        qk, v = num_heads * dim, num_heads * vdim
        self.in_proj = MergedReplicatedLinear(hidden, [qk, qk, v, v], False, dtype, None, f"{prefix}.in_proj", align=8)
        # rows: input gates, forget gates
        self.gate_proj = MergedReplicatedLinear(hidden, [num_heads, num_heads], False, dtype, None, f"{prefix}.gate_proj")
        self.gate_bias = nn.Parameter(torch.zeros(2 * num_heads, dtype=torch.float32), requires_grad=False)
        self.norm_weight = nn.Parameter(torch.ones(v, dtype=dtype), requires_grad=False)
        self.out_proj = ReplicatedLinear(v, hidden, False, dtype, None, f"{prefix}.out_proj")
        self.layer_name = prefix
        self.m_off = num_heads * ops.scan_state_elems(dim, -(-vdim // 4) * 4 + 4)
        self.state_elems = self.m_off + -(-num_heads // 4) * 4
        self.num_kv_heads, self.head_size, self.sliding_window = 1, 0, None
        assert prefix not in _attn._LAYER_REGISTRY, f"duplicate layer name {prefix}"
        _attn._LAYER_REGISTRY[prefix] = self

    def get_kv_cache_spec(self, block_size: int, dtype_size: int) -> KVCacheSpec:
        return MambaSpec(block_size=block_size, state_bytes=self.state_elems * 4)

    def forward(self, hidden: torch.Tensor) -> torch.Tensor:
        q, k, v, g = self.in_proj.parts(self.in_proj(hidden))
        ctx = get_forward_context()
        md = ctx.metadata_for(self.layer_name)
        cache = ctx.kv_caches.get(self.layer_name)
        if md is None or cache is None:                      # profiling run: no state
            return self.out_proj(torch.zeros(hidden.shape[0], self.nh * self.dv, dtype=hidden.dtype, device=hidden.device))
        if ops._use_cuda(hidden):
            cu = ops.cuda_ops()
            gates = cu.memory_gates(hidden, self.gate_proj.weight, self.gate_bias, self.cap, cache, self.m_off, md)
            o = cu.memory_scan(q, k, v, gates, self.q_scale, cache, md, self.nh, self.dk, self.dv)
            return self.out_proj(cu.gated_norm(o, g, self.norm_weight, self.nh, self.eps, False, gate="sigmoid", gates=gates))
        o = self._recur(hidden, q, k, v, cache, md)
        return self.out_proj(ops.gated_norm(o, g, self.norm_weight, self.nh, self.eps, False, gate="sigmoid"))

    def _recur(self, hidden, q, k, v, cache, md) -> torch.Tensor:
        """Plain path: [T, heads * vdim] fp32."""
        from vllm_b200.ops import ref
        T, H, R, C = hidden.shape[0], self.nh, self.dk, self.dv
        z = hidden.float() @ self.gate_proj.weight.float().t() + self.gate_bias
        i, f = (self.cap * torch.tanh(z / self.cap)).split([H, H], dim=-1)
        f = torch.nn.functional.logsigmoid(f)
        q, k, v = (q.float() * self.q_scale).reshape(T, H, R), k.float().reshape(T, H, R), v.float().reshape(T, H, C)
        qsl = (md.query_start_loc_cpu if md.query_start_loc_cpu is not None else md.query_start_loc.cpu()).tolist()
        sls = (md.seq_lens_cpu if md.seq_lens_cpu is not None else md.seq_lens.cpu()).tolist()
        slots = md.block_table[:md.num_reqs, 0].tolist()
        sizes, shapes = [H * R * C, H * R, H], [(H, R, C), (H, R), (H,)]
        o = torch.zeros(T, H, C, dtype=torch.float32, device=hidden.device)
        for j in range(md.num_reqs):
            s, e = qsl[j], qsl[j + 1]
            if e <= s:
                continue
            slot = cache[slots[j], :sum(sizes)]
            state = [t.reshape(sh) for t, sh in zip(slot.split(sizes), shapes)]
            if sls[j] == e - s:
                state = [torch.zeros_like(t) for t in state]
            o[s:e], *state = ref.matrix_memory_scan(q[s:e], k[s:e], v[s:e], i[s:e], f[s:e], *state)
            cache[slots[j], :sum(sizes)] = torch.cat([t.reshape(-1) for t in state])
        return o.reshape(T, H * C)
