"""ctypes bindings to ``vllm_b200/_C.so`` (built by ``vllm_b200/csrc/build.py``).

Every wrapper passes raw device pointers + the current CUDA stream, so the calls are
CUDA-graph capturable.  On a GPU box the kernels are the only path (no silent PyTorch fallback).

A symbol is looked up at its first call.  In a checkout where nothing was built ahead (no ``_C.so``) the source file
that defines it is compiled then, by itself: a process compiles the kernels its model uses and no others
(``prebuild`` does a known set in parallel).
"""
from __future__ import annotations

import ctypes
import os
from typing import Optional

import torch

from vllm_b200 import envs

_LIB_PATH = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "_C.so")


_libs: dict[str, ctypes.CDLL] = {}


def _library_for(name: str) -> ctypes.CDLL:
    """The library that holds symbol ``name``: the full build where there is one, else its source's own."""
    path = _LIB_PATH
    if not os.path.exists(path):
        from vllm_b200.csrc import build as b
        path = b.build_source(b.source_of(name))
    if path not in _libs:
        _libs[path] = ctypes.CDLL(path)
    return _libs[path]


def prebuild(sources) -> None:
    """Compile these sources (names without suffix) in parallel, unless the full library exists."""
    if not os.path.exists(_LIB_PATH):
        from vllm_b200.csrc import build as b
        b.build_sources(sources)


class _Symbol:
    __slots__ = ("name", "argtypes", "fn")

    def __init__(self, name: str, argtypes: tuple) -> None:
        self.name, self.argtypes, self.fn = name, argtypes, None

    def resolve(self):
        fn = getattr(_library_for(self.name), self.name)
        fn.argtypes = list(self.argtypes)
        fn.restype = ctypes.c_int
        self.fn = fn
        return fn

    def __call__(self, *args):
        return (self.fn or self.resolve())(*args)


_symbols: list[_Symbol] = []


def resolve_all() -> None:
    """Look every declared symbol up (a build check: a missing one raises)."""
    for sym in _symbols:
        sym.resolve()


_vp, _i, _i64, _f = ctypes.c_void_p, ctypes.c_int, ctypes.c_int64, ctypes.c_float

_DT = {torch.bfloat16: 0, torch.float16: 1, torch.float32: 2}
_ACT = {"silu": 0, "gelu": 1, "gelu_tanh": 2, "gelu_pytorch_tanh": 2, "relu": 3, "gelu_new": 4, "gelu_fast": 5,
        "quick_gelu": 6, "relu2": 7}


def _sig(name: str, *argtypes) -> _Symbol:
    sym = _Symbol(name, argtypes)
    _symbols.append(sym)
    return sym


_rms_norm = _sig("vb_rms_norm", _vp, _vp, _vp, _vp, _i, _i, _i64, _f, _i, _i, _vp)
_layer_norm = _sig("vb_layer_norm", _vp, _vp, _vp, _vp, _i, _i, _f, _i, _vp)
_act_and_mul = _sig("vb_act_and_mul", _vp, _vp, _i64, _i, _i, _i, _vp)
_activation = _sig("vb_activation", _vp, _vp, _i64, _i, _i, _vp)
_rope_and_cache = _sig("vb_rope_and_cache", _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i64, _i64, _i64, _vp, _vp,
                       _i, _i, _i, _f, _f, _vp, _i, _vp)
_concat_mla = _sig("vb_concat_and_cache_mla", _vp, _vp, _vp, _vp, _i, _i, _i, _i64, _i64, _i, _i, _vp)
_paged_attention = _sig("vb_paged_attention", _vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i,
                        _i64, _i64, _i, _i, _i, _f, _f, _f, _i, _i, _i, _vp)
_paged_attention_ex = _sig("vb_paged_attention_ex", _vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i,
                           _i64, _i64, _i, _i, _i, _f, _f, _f, _i, _i, _i, _vp, _vp, _i, _vp)
_fmha_tc = _sig("vb_fmha_tc2", _vp, _vp, _i64, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i64, _i64, _i,
                _i, _i, _f, _i, _i, _i, _vp, _f, _i, _vp)
_fmha_tc_decode = _sig("vb_fmha_tc_decode", _vp, _vp, _i64, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i64, _i64, _i,
                       _i, _i, _f, _i, _vp, _f, _i, _vp)
_any_attention = _sig("vb_any_attention", _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i, _i, _i64, _i64, _i, _i, _i,
                      _i, _f, _f, _f, _vp, _vp, _i, _vp)
_merge_states = _sig("vb_merge_attn_states", _vp, _vp, _vp, _vp, _vp, _vp, _i64, _i, _i, _vp)
_argmax = _sig("vb_argmax", _vp, _i64, _i, _i, _vp, _i, _vp)
_fused_sample = _sig("vb_fused_sample", _vp, _i64, _i, _i, _vp, _vp, _vp, _vp, _i, _vp)
_topk_topp = _sig("vb_topk_topp", _vp, _i, _i, _vp, _vp, _vp, _vp)
_row_lse = _sig("vb_row_lse", _vp, _i64, _i, _i, _vp, _i, _vp)
_gemm_plan = _sig("vb_gemm_tc_plan", _i, _i, _i, _i, ctypes.POINTER(_i), ctypes.POINTER(_i), ctypes.POINTER(_i),
                  ctypes.POINTER(_i64), ctypes.POINTER(_i))
_gemm_tc = _sig("vb_gemm_tc2", _vp, _vp, _vp, _vp, _i, _i, _i, _i64, _i, _i, _i, _vp, _vp, _i, _vp, _i, _vp)
_any_fold = _sig("vb_any_attention_fold", _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i, _i, _i64, _i, _i, _f, _f, _vp, _i, _i,
                 _i, _vp)
_talk_fold = _sig("vb_talk_fold", _vp, _vp, _i64, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i64, _i, _i, _f, _f, _vp, _i, _i, _vp)
_talk_decode = _sig("vb_talk_decode", _vp, _vp, _i64, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i64, _i, _i, _i, _f, _f, _vp)
_talk_mix = _sig("vb_talk_mix", _vp, _i, _vp, _vp, _vp, _vp, _vp, _i, _vp, _i64, _i, _i, _i, _i, _i, _i, _i, _i, _vp)


def _st() -> int:
    return torch.cuda.current_stream().cuda_stream


def _p(t: Optional[torch.Tensor]) -> Optional[int]:
    return None if t is None else t.data_ptr()


LAUNCHES = 0  # number of our kernels launched through these wrappers (bench.py reports the delta)


def _check(rc: int, name: str, n: int = 1) -> None:
    global LAUNCHES
    LAUNCHES += n
    if rc != 0:
        raise RuntimeError(f"vllm_b200 CUDA op {name} failed (code {rc}"
                           f"{': ' + torch.cuda.get_device_name() if rc > 0 else ''})")


_NUM_SMS: dict[int, int] = {}


def num_sms() -> int:
    d = torch.cuda.current_device()
    if d not in _NUM_SMS:
        _NUM_SMS[d] = torch.cuda.get_device_properties(d).multi_processor_count
    return _NUM_SMS[d]


# ------------------------------------------------------------------ norms / act
def _rows(x: torch.Tensor) -> torch.Tensor:
    """Contiguous and at a 16-byte address, as the vectorised row kernels read it.  (``contiguous`` alone keeps a column slice
    of a single row where it is.)"""
    x = x.contiguous()
    return x if x.data_ptr() % 16 == 0 else x.clone()


def _heads(x: torch.Tensor) -> torch.Tensor:
    """Rows of heads, any row stride, for kernels that read heads in 16-byte vectors."""
    return x if x.data_ptr() % 16 == 0 and (x.stride(0) * x.element_size()) % 16 == 0 else x.clone(memory_format=torch.contiguous_format)


def rms_norm(x, weight, eps, gemma=False):
    H = x.shape[-1]
    x2 = x.reshape(-1, H)
    if x2.stride(-1) != 1 or x2.data_ptr() % 16 or (x2.stride(0) * x2.element_size()) % 16:
        x2 = x2.clone(memory_format=torch.contiguous_format)
    out = torch.empty((x2.shape[0], H), dtype=x.dtype, device=x.device)
    _check(_rms_norm(out.data_ptr(), x2.data_ptr(), None, weight.data_ptr(), x2.shape[0], H, x2.stride(0), eps,
                     int(gemma), _DT[x.dtype], _st()), "rms_norm")
    return out.view(x.shape)


def fused_add_rms_norm(x, residual, weight, eps, gemma=False):
    """In place: residual += x; x = norm(residual). Returns (x, residual)."""
    H = x.shape[-1]
    assert x.is_contiguous() and residual.is_contiguous()
    T = x.numel() // H
    _check(_rms_norm(x.data_ptr(), x.data_ptr(), residual.data_ptr(), weight.data_ptr(), T, H, H, eps, int(gemma),
                     _DT[x.dtype], _st()), "fused_add_rms_norm")
    return x, residual


def layer_norm(x, weight, bias, eps):
    H = x.shape[-1]
    xc = _rows(x)
    out = torch.empty_like(xc)
    _check(_layer_norm(out.data_ptr(), xc.data_ptr(), weight.data_ptr(), _p(bias), xc.numel() // H, H, eps,
                       _DT[x.dtype], _st()), "layer_norm")
    return out


def act_and_mul(x, act: str):
    d = x.shape[-1] // 2
    xc = _rows(x)
    out = torch.empty(x.shape[:-1] + (d,), dtype=x.dtype, device=x.device)
    _check(_act_and_mul(out.data_ptr(), xc.data_ptr(), xc.numel() // (2 * d), d, _ACT[act], _DT[x.dtype], _st()),
           "act_and_mul")
    return out


_silu_mul_il = _sig("vb_silu_mul_interleaved", _vp, _vp, _i64, _i, _i, _vp)


def silu_and_mul_interleaved(x):
    """x[..., 2i] = gate_i, x[..., 2i+1] = up_i → silu(gate) * up."""
    d = x.shape[-1] // 2
    xc = _rows(x)
    out = torch.empty(x.shape[:-1] + (d,), dtype=x.dtype, device=x.device)
    _check(_silu_mul_il(out.data_ptr(), xc.data_ptr(), xc.numel() // (2 * d), d, _DT[x.dtype], _st()), "silu_mul_interleaved")
    return out


_sigmoid_mul = _sig("vb_sigmoid_mul", _vp, _i64, _vp, _i64, _vp, _i64, _i64, _i, _i, _vp)
_soft_cap = _sig("vb_soft_cap", _vp, _i64, _i64, _i, _f, _i, _vp)


def sigmoid_mul_(x, g):
    """x *= sigmoid(g) in place; rows of any stride."""
    assert x.dim() == 2 and x.shape == g.shape and x.dtype == g.dtype and x.stride(1) == g.stride(1) == 1
    _check(_sigmoid_mul(x.data_ptr(), x.stride(0), g.data_ptr(), g.stride(0), x.data_ptr(), x.stride(0), x.shape[0], x.shape[1],
                        _DT[x.dtype], _st()), "sigmoid_mul")
    return x


def soft_cap_(x, cap: float):
    """x = cap tanh(x / cap) in place; rows of any stride."""
    assert x.dim() == 2 and x.stride(1) == 1
    _check(_soft_cap(x.data_ptr(), x.stride(0), x.shape[0], x.shape[1], cap, _DT[x.dtype], _st()), "soft_cap")
    return x


def activation(x, name: str):
    xc = _rows(x)
    out = torch.empty_like(xc)
    _check(_activation(out.data_ptr(), xc.data_ptr(), xc.numel(), _ACT[name], _DT[x.dtype], _st()), "activation")
    return out


# ------------------------------------------------------------------ rope / cache
def _kv_fp8(kv_cache) -> int:
    return int(kv_cache.dtype in (torch.float8_e4m3fn, torch.uint8))


def rope_and_cache(positions, q, k, v, cos_sin_cache, head_dim, is_neox, kv_cache, slot_mapping,
                   k_scale: float = 1.0, v_scale: float = 1.0, vt: bool = False, v_cos_sin=None):
    T = q.shape[0]
    Hq, Hkv = q.shape[-1] // head_dim, k.shape[-1] // head_dim
    assert q.stride(-1) == 1 and k.stride(-1) == 1 and v.stride(-1) == 1
    q, k, v = _heads(q), _heads(k), _heads(v)
    rot = cos_sin_cache.shape[-1]
    flags = _kv_fp8(kv_cache) | (2 if vt else 0)
    _check(_rope_and_cache(positions.data_ptr(), q.data_ptr(), k.data_ptr(), v.data_ptr(), cos_sin_cache.data_ptr(),
                           rot, T, Hq, Hkv, head_dim, q.stride(0), k.stride(0), v.stride(0), kv_cache.data_ptr(),
                           slot_mapping.data_ptr(), kv_cache.shape[3], int(is_neox), flags, k_scale,
                           v_scale, _p(v_cos_sin), _DT[q.dtype], _st()), "rope_and_cache")
    return q, k


def rotary_embedding(positions, q, k, cos_sin_cache, head_dim, is_neox=True):
    T = q.shape[0]
    Hq = q.shape[-1] // head_dim
    Hkv = k.shape[-1] // head_dim if k is not None else 0
    if q.stride(-1) != 1:
        q = q.contiguous()
    q, k = _heads(q), None if k is None else _heads(k)
    rot = cos_sin_cache.shape[-1]
    _check(_rope_and_cache(positions.data_ptr(), q.data_ptr(), _p(k), None, cos_sin_cache.data_ptr(), rot, T, Hq,
                           Hkv, head_dim, q.stride(0), k.stride(0) if k is not None else 0, 0, None, None, 1,
                           int(is_neox), 0, 1.0, 1.0, None, _DT[q.dtype], _st()), "rotary_embedding")
    return q, k


def reshape_and_cache(key, value, kv_cache, slot_mapping, k_scale: float = 1.0, v_scale: float = 1.0,
                      vt: bool = False):
    T, Hkv, D = key.shape
    key, value = _heads(key), _heads(value)
    _check(_rope_and_cache(None, None, key.data_ptr(), value.data_ptr(), None, 0, T, 0, Hkv, D, 0, key.stride(0),
                           value.stride(0), kv_cache.data_ptr(), slot_mapping.data_ptr(), kv_cache.shape[3], 1,
                           _kv_fp8(kv_cache) | (2 if vt else 0), k_scale, v_scale, None, _DT[key.dtype], _st()),
           "reshape_and_cache")


def concat_and_cache_mla(kv_c, k_pe, kv_cache, slot_mapping):
    T, R = kv_c.shape
    P = k_pe.shape[-1]
    _check(_concat_mla(kv_c.data_ptr(), k_pe.data_ptr(), kv_cache.data_ptr(), slot_mapping.data_ptr(), T, R, P,
                       kv_c.stride(0), k_pe.stride(0), kv_cache.shape[1], _DT[kv_c.dtype], _st()),
           "concat_and_cache_mla")


# ------------------------------------------------------------------ attention
class AttnWorkspace:
    """Split-KV partials, sized once for (max_batch, Hq, max_splits, D)."""

    def __init__(self, max_tokens: int, Hq: int, D: int, max_splits: int, device) -> None:
        self.max_splits = max_splits
        self.part_out = torch.empty(max_tokens * Hq * max_splits * D, dtype=torch.float32, device=device)
        self.part_lse = torch.empty(max_tokens * Hq * max_splits, dtype=torch.float32, device=device)


_attn_ws: dict[tuple, AttnWorkspace] = {}


def _get_attn_ws(B: int, Hq: int, D: int, splits: int, device) -> AttnWorkspace:
    key = (device.index, Hq, D)
    ws = _attn_ws.get(key)
    need = B * Hq * splits * D
    if ws is None or ws.part_out.numel() < need:
        if torch.cuda.is_current_stream_capturing():
            raise RuntimeError("attention workspace must be allocated before CUDA-graph capture")
        ws = AttnWorkspace(max(B, 64), Hq, D, max(splits, 16), device)
        if ws.part_out.numel() < need:
            ws = AttnWorkspace(B, Hq, D, splits, device)
        _attn_ws[key] = ws
    return ws


def batch_invariant() -> bool:
    """``VLLM_BATCH_INVARIANT=1``: every dispatch decision that changes a row's floating-point reduction order is
    made from that row's own shape only — never from how many other rows share the launch.  Concretely: no split-K in
    the decode GEMMs (the split factor is otherwise chosen per (N, K) but switches off above 256 rows), no split-KV in
    decode attention (the split count depends on batch × heads), decode-only batches run the same varlen attention
    kernel as mixed batches, collectives reduce in rank order at every size (no in-switch multimem reduction, no
    Lamport fused GEMM + all-reduce), and the MoE combine does not use ``red.add`` epilogues (atomic arrival order).
    Reference: vllm/model_executor/layers/batch_invariant.py (``VLLM_BATCH_INVARIANT`` swaps in fixed-reduction-order
    matmul / softmax / rms-norm kernels, fixes the attention split size and pins NCCL to one algorithm :1105-1180),
    tests/v1/determinism/test_batch_invariance.py."""
    return bool(envs.VLLM_BATCH_INVARIANT)


def decode_splits(B: int, Hkv: int, max_seq_len: int, block_size: int) -> int:
    if batch_invariant():
        return 1
    forced = envs.VLLM_B200_ATTN_SPLITS
    if forced > 0:
        return forced
    ctas = max(B * Hkv, 1)
    target = 2 * num_sms()
    s = max(1, min(16, (target + ctas - 1) // ctas))
    pages = max(1, (max_seq_len + block_size - 1) // block_size)
    # a split costs ~10 us (workspace round trip + reduce kernel): measured on B200 (profiles/README.md §3) it only
    # pays once every split still streams >= ~2k tokens — at 1k-token contexts one CTA per (sequence, kv head) wins
    # even when that leaves SMs idle (14.5 us vs 25.8 us for 64 seqs x 1 kv head)
    s = min(s, max(1, max_seq_len // 2048))
    return max(1, min(s, pages))


_SIMT_SHAPES = {(128, 64), (64, 64), (32, 64), (128, 32), (128, 16), (64, 32), (64, 16), (256, 32), (32, 32), (32, 16)}


def tc_attention_ok(D: int, DV: int, G: int) -> bool:
    """Head shapes of the tensor-core attention kernels (csrc/attention_tc*.cu)."""
    return D == 128 and DV == 128 and G <= 128 and 128 % G == 0


def _simt_attention_ok(D: int, DV: int, BS: int, G: int, dtype) -> bool:
    return (dtype in _HALF_DTYPES and D == DV and (D, BS) in _SIMT_SHAPES and G <= 8 and G & (G - 1) == 0)


def paged_attention(q, kv_cache, md, scale, sliding_window=None, logits_soft_cap=0.0, causal=True, out=None,
                    kv_scale: float = 1.0, return_lse: bool = False, alibi_slopes=None, sinks=None, chunk_size: int = 0,
                    v_head_size: Optional[int] = None, out_scale: float = 1.0):
    """``out``: [T, Hq, DV] (any token stride) to write into."""
    T, Hq, D = q.shape
    Hkv, BS = kv_cache.shape[2], kv_cache.shape[3]
    DV = v_head_size or D
    G = Hq // Hkv
    if out is None:
        # (bucket padding rows are written by no CTA: keep them finite for the row-wise layers that follow)
        out = (torch.zeros if md.flat else torch.empty)((T, Hq, DV), dtype=q.dtype, device=q.device)
    elif md.flat:
        out.zero_()
    assert out.stride(-1) == 1 and out.stride(1) == DV and q.stride(-1) == 1 and q.stride(1) == D
    lse = torch.empty((T, Hq), dtype=torch.float32, device=q.device) if return_lse else None
    bt = md.block_table
    if alibi_slopes is not None:
        alibi_slopes = alibi_slopes.to(device=q.device, dtype=torch.float32).contiguous()
    if sinks is not None:
        sinks = sinks.to(device=q.device, dtype=torch.float32).contiguous()
    chunk_size = int(chunk_size or 0)
    if md.kv_vt:
        # tcgen05 kernel over the tensor-core cache layout
        assert tc_attention_ok(D, DV, G) and BS == 64 and not logits_soft_cap and alibi_slopes is None, \
            "tensor-core attention: D=128, 64-token pages, no soft-cap / ALiBi"
        # batch-invariant mode: a decode row takes the varlen kernel it would take inside a mixed batch
        decode = md.decode_only and not (batch_invariant() and md.query_start_loc is not None)
        splits = (md.num_splits or decode_splits(md.num_reqs, Hkv, md.max_seq_len, 128)) if decode else 1
        if chunk_size and chunk_size <= 4096:
            splits = 1                                   # a chunk is all that a query reads
        ws = _get_attn_ws(md.num_reqs, Hq, D, splits, q.device) if splits > 1 else None
        if decode and G <= 16 and (G & (G - 1)) == 0 and causal:
            # swap-AB decode kernel: KV tokens on the MMA M axis
            rc = _fmha_tc_decode(q.data_ptr(), kv_cache.data_ptr(), kv_cache.shape[0], bt.data_ptr(),
                                 md.seq_lens.data_ptr(), out.data_ptr(), _p(ws.part_out) if ws else None,
                                 _p(ws.part_lse) if ws else None, _p(lse), md.num_reqs, Hq, Hkv, q.stride(0),
                                 out.stride(0), bt.stride(0), splits, sliding_window or 0, scale, chunk_size, _p(sinks),
                                 out_scale, _DT[q.dtype], _st())
            _check(rc, f"fmha_tc_decode(G={G})", 2 if splits > 1 else 1)
            return (out, lse) if return_lse else out
        rc = _fmha_tc(q.data_ptr(), kv_cache.data_ptr(), kv_cache.shape[0], bt.data_ptr(), md.seq_lens.data_ptr(),
                      None if decode else md.query_start_loc.data_ptr(), out.data_ptr(),
                      _p(ws.part_out) if ws else None, _p(ws.part_lse) if ws else None, _p(lse), md.num_reqs, T,
                      md.max_query_len, Hq, Hkv, q.stride(0), out.stride(0), bt.stride(0), splits,
                      sliding_window or 0, scale, int(causal), int(md.flat and not decode), chunk_size, _p(sinks), out_scale,
                      _DT[q.dtype], _st())
        _check(rc, f"fmha_tc(G={Hq // Hkv})", 2 if splits > 1 else 1)
        return (out, lse) if return_lse else out
    if not _simt_attention_ok(D, DV, BS, G, q.dtype) or out_scale != 1.0:
        assert kv_cache.dtype == q.dtype, "the generic attention kernel reads caches of the model dtype"
        # one token per request needs no offsets (and the same arithmetic serves prompts and decode steps)
        rc = _any_attention(q.data_ptr(), kv_cache.data_ptr(), bt.data_ptr(), md.seq_lens.data_ptr(),
                            None if md.decode_only else md.query_start_loc.data_ptr(), out.data_ptr(), _p(lse), md.num_reqs,
                            1 if md.decode_only else md.max_query_len, Hq, Hkv, D, DV, kv_cache.shape[4], BS, q.stride(0),
                            out.stride(0), bt.stride(0), sliding_window or 0, chunk_size, int(causal), scale, logits_soft_cap,
                            out_scale, _p(alibi_slopes), _p(sinks), _DT[q.dtype], _st())
        _check(rc, f"any_attention(D={D}, DV={DV}, G={G})")
        return (out, lse) if return_lse else out
    n_launch = 1
    if md.decode_only and not (batch_invariant() and md.query_start_loc is not None):
        splits = md.num_splits or decode_splits(md.num_reqs, Hkv, md.max_seq_len, BS)
        n_launch = 2 if splits > 1 else 1
        ws = _get_attn_ws(md.num_reqs, Hq, D, splits, q.device) if splits > 1 else None
        rc = _paged_attention_ex(q.data_ptr(), kv_cache.data_ptr(), bt.data_ptr(), md.seq_lens.data_ptr(), None,
                                 out.data_ptr(), _p(ws.part_out) if ws else None, _p(ws.part_lse) if ws else None,
                                 _p(lse), md.num_reqs, 1, Hq, Hkv, D, BS, q.stride(0), out.stride(0), bt.stride(0),
                                 splits, sliding_window or 0, scale, logits_soft_cap, kv_scale, int(causal),
                                 _kv_fp8(kv_cache), _DT[q.dtype], _p(alibi_slopes), _p(sinks), chunk_size, _st())
    else:
        rc = _paged_attention_ex(q.data_ptr(), kv_cache.data_ptr(), bt.data_ptr(), md.seq_lens.data_ptr(),
                                 md.query_start_loc.data_ptr(), out.data_ptr(), None, None, _p(lse), md.num_reqs,
                                 md.max_query_len, Hq, Hkv, D, BS, q.stride(0), out.stride(0), bt.stride(0), 1,
                                 sliding_window or 0, scale, logits_soft_cap, kv_scale, int(causal),
                                 _kv_fp8(kv_cache), _DT[q.dtype], _p(alibi_slopes), _p(sinks), chunk_size, _st())
    _check(rc, f"paged_attention(D={D}, BS={BS}, G={Hq // Hkv})", n_launch)
    return (out, lse) if return_lse else out


# bytes of unmixed head outputs held at a time; larger batches are done some value heads at a time
TALK_BYTES = 1 << 30


def tc_talk_ok(dtype, soft_cap: float) -> bool:
    """Do the tensor-core kernels of mixed heads take these scores (head shapes: ``tc_attention_ok``)?  e^score must fit into 32 bits."""
    return dtype == torch.bfloat16 and 0.0 < soft_cap <= 60.0


def talk_decode_ok(H: int, Hkv: int) -> bool:
    g = H // Hkv
    return H <= 32 and Hkv <= 8 and g in (1, 2, 4, 8, 16) and (g > 2 or H <= 16)


def talk_splits(B: int, max_seq_len: int, window: int) -> int:
    """Key ranges per request in a decode step: one wave of CTAs, two tiles of 128 keys each at least."""
    if batch_invariant():
        return 1
    keys = min(max_seq_len, window) if window else max_seq_len
    return max(1, min(num_sms() // max(B, 1), (keys + 255) // 256, 16))


def talking_attention(q, kv_cache, md, scale, sliding_window, soft_cap, talk, sinks, v_head_size: int, v_rope=None, positions=None,
                      out=None):
    """Attention whose heads' weights are mixed by ``talk`` (csrc/attention_talk.cu); q [T, Hq, D] → [T, Hq, DV]."""
    T, Hq, D = q.shape
    Hkv, BS = kv_cache.shape[2], kv_cache.shape[3]
    DV, G, window, dev = v_head_size, Hq // Hkv, sliding_window or 0, q.device
    back = None if v_rope is None else v_rope.cos_sin_cache
    neox = v_rope is not None and v_rope.is_neox_style
    if talk is None:
        o = paged_attention(q, kv_cache, md, scale, sliding_window, soft_cap, sinks=sinks, v_head_size=DV)
        if v_rope is not None:
            half = back.shape[-1] // 2
            from vllm_b200 import ops
            o = ops.rotary_embedding(positions, o.view(T, Hq * DV), None, torch.cat((back[:, :half], -back[:, half:]), -1), DV, neox)[0]
            o = o.view(T, Hq, DV)
        return o if out is None else out.copy_(o)
    if out is None:
        out = torch.empty((T, Hq, DV), dtype=q.dtype, device=dev)
    assert q.stride(2) == 1 and q.stride(1) == D and out.stride(2) == 1 and out.stride(1) == DV and kv_cache.dtype == q.dtype
    assert talk.dtype == torch.float32 and talk.is_contiguous() and (sinks is None or sinks.dtype == torch.float32) and not md.flat
    bt = md.block_table

    def mix(o, l, S, c0, nc):
        _check(_talk_mix(o.data_ptr(), _DT[o.dtype], _p(l), _p(sinks) if l is not None else None, talk.data_ptr(), _p(positions), _p(back),
                         int(neox), out.data_ptr(), out.stride(0), T, Hq, G, DV, S, c0, nc, _DT[q.dtype], _st()), "talk_mix")
    if md.kv_vt and md.decode_only and talk_decode_ok(Hq, Hkv):
        S = talk_splits(md.num_reqs, md.max_seq_len, window)
        o = torch.empty((S, T, Hq, Hkv, DV), dtype=torch.float32, device=dev)
        l = torch.empty((S, T, Hq), dtype=torch.float32, device=dev)
        _check(_talk_decode(q.data_ptr(), kv_cache.data_ptr(), kv_cache.shape[0], bt.data_ptr(), md.seq_lens.data_ptr(), o.data_ptr(),
                            l.data_ptr(), kernel_error_flag(dev).data_ptr(), md.num_reqs, Hq, Hkv, q.stride(0), bt.stride(0), S, window,
                            scale, soft_cap, _st()), f"talk_decode(H={Hq}, Hkv={Hkv})")
        mix(o, l, S, 0, Hkv)
        return out
    tc = md.kv_vt
    if tc:
        assert tc_attention_ok(D, DV, G) and BS == 64 and tc_talk_ok(q.dtype, soft_cap), "tensor-core layout with another head shape"
    per_head = T * Hq * DV * (2 if tc else 4)
    step = max(2 if tc else 1, min(Hkv, TALK_BYTES // max(per_head, 1) // 2 * 2))
    qsl = md.query_start_loc
    for c0 in range(0, Hkv, step):
        nc = min(step, Hkv - c0)
        # (padding rows are written by no CTA: keep them finite)
        o = (torch.empty if md.num_actual_tokens == T else torch.zeros)((T, Hq, nc, DV), dtype=torch.bfloat16 if tc else torch.float32, device=dev)
        if tc:
            _check(_talk_fold(q.data_ptr(), kv_cache.data_ptr(), kv_cache.shape[0], bt.data_ptr(), md.seq_lens.data_ptr(), qsl.data_ptr(),
                              o.data_ptr(), kernel_error_flag(dev).data_ptr(), md.num_reqs, T, 1 if md.decode_only else md.max_query_len,
                              Hq, Hkv, q.stride(0), bt.stride(0), window, scale, soft_cap, _p(sinks), c0, nc, _st()),
                   f"talk_fold(H={Hq}, Hkv={Hkv})")
        else:
            _check(_any_fold(q.data_ptr(), kv_cache.data_ptr(), bt.data_ptr(), md.seq_lens.data_ptr(),
                             None if md.decode_only else qsl.data_ptr(), o.data_ptr(), md.num_reqs,
                             1 if md.decode_only else md.max_query_len, Hq, Hkv, D, DV, kv_cache.shape[4], BS, q.stride(0), bt.stride(0),
                             window, scale, soft_cap, _p(sinks), c0, nc, _DT[q.dtype], _st()), f"any_attention_fold(D={D}, DV={DV})")
        mix(o, None, 1, c0, nc)
    return out


def merge_attn_states(o1, lse1, o2, lse2):
    T, H, D = o1.shape
    out = torch.empty_like(o1)
    lse = torch.empty_like(lse1)
    _check(_merge_states(out.data_ptr(), lse.data_ptr(), o1.data_ptr(), lse1.data_ptr(), o2.data_ptr(),
                         lse2.data_ptr(), T * H, D, _DT[o1.dtype], _st()), "merge_attn_states")
    return out, lse


_mla_decode = _sig("vb_mla_decode", _vp, _vp, _vp, _i64, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i64, _i64,
                   _i64, _i64, _i64, _i, _i, _i, _f, _i, _vp)
_mla_prefill = _sig("vb_mla_prefill", _vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i64, _i, _i, _i, _i, _i, _i, _i64, _i64,
                    _i64, _i64, _i64, _i, _i, _f, _i, _vp)
_mla_simt = _sig("vb_mla_simt", _vp, _vp, _vp, _vp, _vp, _i64, _vp, _vp, _i, _i, _i, _i, _i, _i, _i64, _i64, _i64, _i64, _i64,
                 _i64, _i, _f, _i, _vp)
_latent_rope = _sig("vb_latent_rope_cache", _vp, _vp, _i64, _i, _i, _i, _i, _vp, _f, _vp, _vp, _i, _vp, _i64, _vp, _i, _i, _vp)
_latent_norm = _sig("vb_latent_norm_cache", _vp, _i64, _i, _vp, _vp, _i, _vp, _vp, _vp, _i64, _vp, _i, _f, _i, _vp)
_mla_ws: dict[int, tuple] = {}
_kernel_error: dict[int, torch.Tensor] = {}


def kernel_error_flag(device: torch.device) -> torch.Tensor:
    """Device int that a kernel with bounded waits raises when one of them ran into its limit."""
    key = device.index or 0
    t = _kernel_error.get(key)
    if t is None:
        if torch.cuda.is_current_stream_capturing():
            raise RuntimeError("the kernel error flag must be allocated before CUDA-graph capture")
        t = _kernel_error[key] = torch.zeros(1, dtype=torch.int32, device=device)
    return t


def check_kernel_error(device: torch.device) -> None:
    """Raise if a kernel gave up on a wait since the last check (synchronises)."""
    t = _kernel_error.get(device.index or 0)
    if t is not None and int(t.item()):
        t.zero_()
        raise RuntimeError("a kernel gave up waiting for a copy or a matrix product; its outputs are not valid")


def mla_decode_splits(B: int, H: int, max_seq_len: int, least: int = 512) -> int:
    if batch_invariant():
        return 1
    forced = envs.VLLM_B200_ATTN_SPLITS
    if forced > 0:
        return forced
    groups = (H + 31) // 32 if H > 16 else 1
    ctas = max(B * groups, 1)
    s = max(1, min(16, num_sms() // ctas))           # one CTA per SM (170 KB smem): stay inside ONE wave
    return max(1, min(s, max_seq_len // least))     # every split should still stream >= 8 tiles (windows: 4)


def mla_decode_tc(q_nope_abs, q_pe, kv_cache, block_table, seq_lens, scale, max_seq_len: int, num_splits: int = 0,
                  return_lse: bool = False, sliding_window: Optional[int] = None):
    """tcgen05 MLA decode (csrc/mla_decode.cu): q_nope_abs [B, H, R], q_pe [B, H, P] or None, cache [blocks, BS, R + P]."""
    B, H, R = q_nope_abs.shape
    P = 0 if q_pe is None else q_pe.shape[-1]
    assert kv_cache.shape[-1] == R + P and q_nope_abs.stride(-1) == 1 and (q_pe is None or q_pe.stride(-1) == 1)
    dev = q_nope_abs.device
    splits = num_splits or (mla_decode_splits(B, H, min(max_seq_len, sliding_window), 256) if sliding_window else
                            mla_decode_splits(B, H, max_seq_len))
    out = torch.empty((B, H, R), dtype=q_nope_abs.dtype, device=dev)
    lse = torch.empty((B, H), dtype=torch.float32, device=dev) if return_lse else None
    po = pl = None
    if splits > 1:
        key = dev.index or 0
        need = B * H * splits
        ws = _mla_ws.get(key)
        if ws is None or ws[1].numel() < need:
            if torch.cuda.is_current_stream_capturing():
                raise RuntimeError("MLA split-KV workspace must be allocated before CUDA-graph capture")
            n = max(need, 64 * 128 * 4)
            ws = _mla_ws[key] = (torch.empty(n * 512, dtype=torch.float32, device=dev),
                                 torch.empty(n, dtype=torch.float32, device=dev))
        po, pl = ws
    err = kernel_error_flag(dev)
    _check(_mla_decode(q_nope_abs.data_ptr(), _p(q_pe), kv_cache.data_ptr(), kv_cache.shape[0],
                       block_table.data_ptr(), seq_lens.data_ptr(), out.data_ptr(), _p(po), _p(pl), _p(lse), err.data_ptr(), B,
                       H, R, P, kv_cache.shape[1], q_nope_abs.stride(0), q_nope_abs.stride(1),
                       q_pe.stride(0) if P else 0, q_pe.stride(1) if P else 0,
                       out.stride(0), block_table.stride(0), splits, sliding_window or 0, scale, _DT[q_nope_abs.dtype], _st()),
           f"mla_decode(B={B},H={H},R={R})", 2 if splits > 1 else 1)
    return (out, lse) if return_lse else out


def _mla_tc_ok(q_nope_abs, q_pe, kv_cache) -> bool:
    R = q_nope_abs.shape[-1]
    if q_pe is None:
        shape_ok = q_nope_abs.dtype == torch.bfloat16 and R % 8 == 0 and R <= 512 and kv_cache.shape[-1] == R
    else:
        P = q_pe.shape[-1]
        widths = (R == 512 and P == 64) or (q_nope_abs.dtype == torch.bfloat16 and R % 8 == 0 and R <= 512 and P % 8 == 0 and P <= 64)
        shape_ok = (q_nope_abs.dtype in _HALF_DTYPES and widths and kv_cache.shape[-1] == R + P and q_pe.data_ptr() % 16 == 0
                    and q_pe.stride(-1) == 1 and (q_pe.stride(0) * 2) % 16 == 0 and (q_pe.stride(1) * 2) % 16 == 0)
    return (shape_ok and kv_cache.dtype == q_nope_abs.dtype and kv_cache.dim() == 3
            and kv_cache.shape[1] in (16, 32, 64, 128) and q_nope_abs.stride(-1) == 1
            and (q_nope_abs.stride(0) * 2) % 16 == 0 and (q_nope_abs.stride(1) * 2) % 16 == 0
            and q_nope_abs.data_ptr() % 16 == 0 and envs.VLLM_B200_ATTN != "simt")


_HALF_DTYPES = (torch.bfloat16, torch.float16)


def mla_simt(q_abs, q_pe, kv_cache, block_table, seq_lens, qsl, scale, sliding_window: Optional[int] = None):
    """Variable-length attention over the latent cache for any width and dtype (csrc/latent.cu); fp32 arithmetic."""
    T, H, R = q_abs.shape
    P = 0 if q_pe is None else q_pe.shape[-1]
    assert kv_cache.shape[-1] == R + P and kv_cache.dtype == q_abs.dtype and kv_cache.is_contiguous()
    q_abs = q_abs if q_abs.stride(-1) == 1 else q_abs.contiguous()
    q_pe = q_pe if q_pe is None or q_pe.stride(-1) == 1 else q_pe.contiguous()
    out = torch.empty((T, H, R), dtype=q_abs.dtype, device=q_abs.device)
    _check(_mla_simt(q_abs.data_ptr(), _p(q_pe), kv_cache.data_ptr(), out.data_ptr(), block_table.data_ptr(),
                     block_table.stride(0), seq_lens.data_ptr(), _p(qsl), seq_lens.numel(), T, H, R, P, kv_cache.shape[1],
                     q_abs.stride(0), q_abs.stride(1), q_pe.stride(0) if P else 0, q_pe.stride(1) if P else 0,
                     out.stride(0), out.stride(1), sliding_window or 0, scale, _DT[q_abs.dtype], _st()), f"mla_simt(T={T},H={H},R={R})")
    return out


def mla_prefill_ok(q, dim: int, rot: int, v_dim: int, kv_lora_rank: int) -> bool:
    return (q.dtype in _HALF_DTYPES and dim % 8 == 0 and 8 <= dim <= 128 and rot % 8 == 0 and rot <= 64 and v_dim % 8 == 0
            and 8 <= v_dim <= 128 and kv_lora_rank % 8 == 0 and q.stride(0) % 8 == 0 and q.data_ptr() % 16 == 0
            and envs.VLLM_B200_ATTN != "simt")


def mla_prefill(q, k, v, out, q_start, q_len, seq_len, kv_start, h0: int, max_q: int, scale, k_pe=None, window: int = 0) -> None:
    """Causal attention of prompt portions over expanded keys and values (csrc/mla_prefill.cu), written into ``out``.
    q [T, H, dim + rot], out [T, H, vdim]; k [KV, hl, dim], v [KV, hl, vdim] hold heads h0 .. h0 + hl - 1, k_pe [KV, rot] the rotated key
    part of all heads (None: rot = 0)."""
    T, H, DQ = q.shape
    KV, hl, D = k.shape
    VD, P = v.shape[-1], 0 if k_pe is None else k_pe.shape[-1]
    assert DQ == D + P and (k_pe is None or (k_pe.stride(1) == 1 and k_pe.data_ptr() % 16 == 0))
    assert q.stride(2) == 1 and q.stride(1) == DQ and k.stride(2) == 1 and k.stride(1) == D and v.stride(2) == 1 and v.stride(1) == VD
    assert out.shape == (T, H, VD) and out.stride(1) == VD and out.stride(2) == 1
    for t in (q, k, v, out):
        assert t.data_ptr() % 16 == 0
    _check(_mla_prefill(q.data_ptr(), k.data_ptr(), v.data_ptr(), _p(k_pe), out.data_ptr(), q_start.data_ptr(), q_len.data_ptr(),
                        seq_len.data_ptr(), kv_start.data_ptr(), kernel_error_flag(q.device).data_ptr(), q_len.numel(), T, KV, H,
                        h0, hl, D, P, VD, q.stride(0), k.stride(0), v.stride(0), 0 if k_pe is None else k_pe.stride(0), out.stride(0), max_q,
                        window, scale, _DT[q.dtype], _st()),
           f"mla_prefill(T={T},KV={KV},H={H})")


def latent_rope_cache(proj, q_off: int, heads: int, dim: int, rot: int, kv_off: int, kv_rank: int, kv_weight, eps: float, positions, cos_sin,
                      neox: bool, cache=None, slots=None) -> None:
    """On the columns of a merged projection, in place (csrc/latent.cu): see ops.latent_rope_cache."""
    assert proj.dim() == 2 and proj.stride(1) == 1 and (cos_sin is None or cos_sin.shape[-1] == rot)
    if cache is not None:
        assert cache.shape[-1] == kv_rank + rot and cache.dtype == proj.dtype and cache.is_contiguous() and slots.dtype == torch.int64
    es = proj.element_size()
    _check(_latent_rope(proj.data_ptr() + q_off * es, proj.data_ptr() + kv_off * es if kv_rank else None, proj.stride(0), heads, dim, rot,
                        kv_rank, _p(kv_weight), eps, _p(positions), _p(cos_sin), int(neox), _p(cache), kv_rank + rot,
                        _p(slots) if cache is not None else None, proj.shape[0], _DT[proj.dtype], _st()), "latent_rope_cache")


def latent_norm_cache(lat, q_rank: int, q_weight, kv_rank: int, kv_weight, eps: float, cache=None, slots=None, want_kv: bool = True):
    """(c_q, c_kv): RMSNorm of the two halves of a latent down-projection [T, q_rank + kv_rank]; c_kv also goes into its
    cache rows (csrc/latent.cu).  kv_rank = 0: queries only."""
    T = lat.shape[0]
    cq = torch.empty((T, q_rank), dtype=lat.dtype, device=lat.device)
    ckv = torch.empty((T, kv_rank), dtype=lat.dtype, device=lat.device) if kv_rank and want_kv else None
    if cache is not None:
        assert cache.shape[-1] == kv_rank and cache.dtype == lat.dtype and cache.is_contiguous() and slots.dtype == torch.int64
    _check(_latent_norm(lat.data_ptr(), lat.stride(0), q_rank, _p(q_weight), cq.data_ptr(), kv_rank, _p(kv_weight), _p(ckv),
                        _p(cache), kv_rank, _p(slots) if cache is not None else None, T, eps, _DT[lat.dtype], _st()),
           "latent_norm_cache")
    return cq, ckv


def mla_attention(q_nope_abs, q_pe, kv_cache, md, scale, kv_lora_rank, sliding_window: Optional[int] = None):
    """MLA as MQA over the latent cache (K = latent (+ rope) row, V = the latent part of the same row).

    Decode batches run on the tcgen05 MLA kernel (csrc/mla_decode.cu: the latent tile is shared by all heads of the
    CTA and by both matrix products, split-KV for long contexts; no host synchronisation, graph capturable).
    Everything it does not cover — other widths with a rope part, fp32, variable-length batches — runs on the generic
    kernel of csrc/latent.cu, which needs no host lengths either."""
    R = q_nope_abs.shape[-1]
    if md.decode_only and R == kv_lora_rank and _mla_tc_ok(q_nope_abs, q_pe, kv_cache):
        return mla_decode_tc(q_nope_abs, q_pe, kv_cache, md.block_table, md.seq_lens, scale, md.max_seq_len,
                             md.num_splits or 0, sliding_window=sliding_window)
    B = md.num_reqs
    return mla_simt(q_nope_abs, q_pe, kv_cache, md.block_table, md.seq_lens[:B],
                    None if md.decode_only else md.query_start_loc, scale, sliding_window)


# ------------------------------------------------------------------ sampling
def argmax(logits: torch.Tensor) -> torch.Tensor:
    B, V = logits.shape
    out = torch.empty(B, dtype=torch.int64, device=logits.device)
    _check(_argmax(logits.data_ptr(), logits.stride(0), B, V, out.data_ptr(), _DT[logits.dtype], _st()), "argmax")
    return out


_step_buf: dict[int, torch.Tensor] = {}


def fused_sample(logits, temperature, seeds, step, out: Optional[torch.Tensor] = None):
    """``step``: per-row int32 [B] noise counters (a python int is broadcast)."""
    B, V = logits.shape
    if out is None:
        out = torch.empty(B, dtype=torch.int64, device=logits.device)
    if not isinstance(step, torch.Tensor):
        step = torch.full((B,), int(step) & 0x7FFFFFFF, dtype=torch.int32, device=logits.device)
    _check(_fused_sample(logits.data_ptr(), logits.stride(0), B, V, temperature.data_ptr(), seeds.data_ptr(),
                         step.data_ptr(), out.data_ptr(), _DT[logits.dtype], _st()), "fused_sample")
    return out


_fused_sample_cand = _sig("vb_fused_sample_cand", _vp, _i64, _i, _i, _vp, _vp, _vp, _i, _vp, _i, _vp)
_select_cand = _sig("vb_select_candidate", _vp, _i, _vp, _i, _vp)


def fused_sample_candidates(logits_local, temperature, seeds, step, idx_off: int, v_valid: int) -> torch.Tensor:
    """Per-row best (value, global id) of this rank's vocab shard as a [B, 8] bf16-viewable 16-byte record."""
    B = logits_local.shape[0]
    cand = torch.empty((B, 4), dtype=torch.float32, device=logits_local.device)
    _check(_fused_sample_cand(logits_local.data_ptr(), logits_local.stride(0), B, max(v_valid, 0), temperature.data_ptr(),
                              seeds.data_ptr(), step.data_ptr(), idx_off, cand.data_ptr(), _DT[logits_local.dtype], _st()),
           "fused_sample_cand")
    return cand


def select_candidates(cands: torch.Tensor, W: int, out: torch.Tensor) -> torch.Tensor:
    """cands: [B, W, 4] fp32 records gathered from the W ranks → winning token id per row."""
    B = out.shape[0]
    _check(_select_cand(cands.data_ptr(), W, out.data_ptr(), B, _st()), "select_candidate")
    return out


def topk_topp_mask_(logits: torch.Tensor, top_k, top_p, min_p=None) -> torch.Tensor:
    assert logits.dtype == torch.float32 and logits.is_contiguous()
    B, V = logits.shape
    _check(_topk_topp(logits.data_ptr(), B, V, _p(top_k), _p(top_p), _p(min_p), _st()), "topk_topp")
    return logits


def row_lse(logits: torch.Tensor) -> torch.Tensor:
    B, V = logits.shape
    out = torch.empty(B, dtype=torch.float32, device=logits.device)
    _check(_row_lse(logits.data_ptr(), logits.stride(0), B, V, out.data_ptr(), _DT[logits.dtype], _st()), "row_lse")
    return out


# ------------------------------------------------------------------ fp32 residual stream (csrc/stream.cu)
_embed_stream = _sig("vb_embed_stream", _vp, _vp, _vp, _vp, _f, _vp, _vp, _i, _i, _i, _i, _i, _vp)
_post_norm = _sig("vb_post_norm_add", _vp, _i64, _vp, _vp, _i, _vp, _i, _vp, _vp, _i, _vp, _i, _i, _f, _i, _vp)


def embed_stream(ids, positions, table, pos_table, scale: float):
    """(x fp32, copy of x in the table's dtype — x itself when that is fp32)."""
    T, H = ids.numel(), table.shape[1]
    x = torch.empty((T, H), dtype=torch.float32, device=table.device)
    out = None if table.dtype == torch.float32 else torch.empty((T, H), dtype=table.dtype, device=table.device)
    assert ids.dtype == torch.int32 and positions.dtype == torch.int64 and table.is_contiguous()
    _check(_embed_stream(ids.data_ptr(), positions.data_ptr(), table.data_ptr(), _p(pos_table), float(scale), x.data_ptr(),
                         _p(out), T, H, table.shape[0], 0 if pos_table is None else pos_table.shape[0], _DT[table.dtype], _st()),
           "embed_stream")
    return x, (x if out is None else out)


def post_norm_add(x, y, weight, eps: float, gemma: bool, next_weight=None, next_gemma: bool = False, inv=None, pair_w=None):
    """In place: x += rmsnorm(y') * w, y' = y [T, H] or (``inv``, ``pair_w`` [T, k]) the weighted sum of expert rows of y.
    Returns x in y's dtype (x itself when that is fp32), or its norm with ``next_weight``."""
    T, H = x.shape
    assert x.dtype == torch.float32 and x.is_contiguous() and y.stride(-1) == 1
    k = 1 if inv is None else inv.numel() // T
    out = None
    if next_weight is not None or y.dtype != torch.float32:
        out = torch.empty((T, H), dtype=y.dtype, device=y.device)
    _check(_post_norm(y.data_ptr(), y.stride(0), _p(inv), _p(pair_w), k, weight.data_ptr(), int(gemma), x.data_ptr(),
                      _p(next_weight), int(next_gemma), _p(out), T, H, eps, _DT[y.dtype], _st()), "post_norm_add")
    return x if out is None else out


_norm_add = _sig("vb_norm_add", _vp, _i, _vp, _i64, _vp, _vp, _vp, _f, _vp, _vp, _vp, _i, _i, _vp, _i, _i, _f, _i, _vp)


def norm_add(x, y, y_bias, norm, mult: float, next_norm, eps: float, ids=None):
    """In place on the fp32 stream: x += mult * norm(y + y_bias), or (``ids``) x = y[ids] with y the embedding table.  ``norm``,
    ``next_norm``: (weight, bias) of layer norms.  Returns next_norm(x) — or x — in y's dtype."""
    T, H = x.shape
    assert x.dtype == torch.float32 and x.is_contiguous() and y.stride(-1) == 1 and (ids is None or ids.dtype == torch.int32)
    w1, b1 = norm if norm is not None else (None, None)
    w2, b2 = next_norm if next_norm is not None else (None, None)
    out = torch.empty((T, H), dtype=y.dtype, device=y.device) if w2 is not None or y.dtype != torch.float32 else None
    _check(_norm_add(_p(ids), y.shape[0], y.data_ptr(), y.stride(0), _p(y_bias), _p(w1), _p(b1), mult, x.data_ptr(), _p(w2), _p(b2),
                     0, 1, _p(out), T, H, eps, _DT[y.dtype], _st()), "norm_add")
    return x if out is None else out


_add_norm = _sig("vb_add_norm", _vp, _i64, _vp, _i64, _vp, _vp, _vp, _i, _i, _vp, _i64, _vp, _vp, _vp, _i, _i, _vp, _i, _i, _f, _i, _vp)


def add_norm(x, y, next_norm, eps: float, dtype=None, rows=None, inv=None, pair_w=None, ids=None, experts: int = 0, h=None):
    """In place on the fp32 stream: x += y + routed sum (``rows`` of the experts by ``inv``, weights ``pair_w``, and ``h`` for expert
    numbers from ``experts`` on).  ``next_norm``: (weight, bias or None) of a layer norm.  Returns next_norm(x) — or x — in ``dtype``
    (y's)."""
    T, H = x.shape
    dtype = dtype or y.dtype
    assert x.dtype == torch.float32 and x.is_contiguous()
    assert all(t is None or (t.dtype == dtype and t.stride(-1) == 1) for t in (y, rows, h)) and (ids is None or ids.dtype == torch.int32)
    w2, b2 = next_norm if next_norm is not None else (None, None)
    out = torch.empty((T, H), dtype=dtype, device=x.device) if w2 is not None or dtype != torch.float32 else None

    def st(t):
        return 0 if t is None else t.stride(0)
    _check(_add_norm(_p(y), st(y), _p(rows), st(rows), _p(inv), _p(pair_w), _p(ids), 0 if pair_w is None else pair_w.shape[1], experts,
                     _p(h), st(h), x.data_ptr(), _p(w2), _p(b2), 0, 1, _p(out), T, H, eps, _DT[dtype], _st()), "add_norm")
    return x if out is None else out


_hyper = _sig("vb_hyper_step", _vp, _i, _vp, _i64, _vp, _vp, _vp, _vp, _i, _vp, _vp, _i, _i, _f, _i, _vp)
_xielu = _sig("vb_xielu", _vp, _vp, _vp, _i64, _i, _vp)


def _hyper_call(ids, vocab, y, embed_weight, coef, into, x, weight, eps, dtype):
    T, S, H = x.shape
    assert x.dtype == torch.float32 and x.is_contiguous() and into.dtype == torch.float32 and into.numel() == S
    assert (coef is None or (coef.dtype == torch.float32 and coef.numel() == S + S * S)) and (ids is None or ids.dtype == torch.int32)
    assert weight.dtype == dtype and (y is None or (y.dtype == dtype and y.stride(-1) == 1))
    out = torch.empty((T, H), dtype=dtype, device=x.device)
    _check(_hyper(_p(ids), vocab, _p(y), 0 if y is None else y.stride(0), _p(embed_weight), _p(coef), into.data_ptr(), x.data_ptr(), S,
                  weight.data_ptr(), out.data_ptr(), T, H, eps, _DT[dtype], _st()), "hyper_step")
    return out


def hyper_entry(ids, table, streams: int, embed_weight, into, weight, eps: float):
    T = table.shape[0] if ids is None else ids.numel()
    x = torch.empty((T, streams, table.shape[1]), dtype=torch.float32, device=table.device)
    return x, _hyper_call(ids, table.shape[0], table, embed_weight, None, into, x, weight, eps, table.dtype)


def hyper_step(x, y, coef, into, weight, eps: float, dtype):
    return _hyper_call(None, 0, y, None, coef if y is not None else None, into, x, weight, eps, dtype)


def xielu(x, coef, out=None):
    x = x.contiguous()
    out = torch.empty_like(x) if out is None else out
    _check(_xielu(x.data_ptr(), out.data_ptr(), coef.data_ptr(), x.numel(), _DT[x.dtype], _st()), "xielu")
    return out


def linear_xielu(x, weight, bias, coef):
    """xielu(x W^T + b): in the epilogue of the decode GEMM, else one pass over its result in place."""
    x2 = x.reshape(-1, x.shape[-1])
    if 0 < x2.shape[0] <= 256 and _tc_ok(x2, weight) and _plan(x2.shape[0], weight.shape[0], x2.shape[1])[0]:
        return gemm_tc(x2, weight, bias, act=3, act_coef=coef).view(x.shape[:-1] + (weight.shape[0],))
    y = linear(x, weight, bias)
    return xielu(y, coef, out=y)


# ------------------------------------------------------------------ GEMM
class _GemmWorkspace:
    def __init__(self) -> None:
        self.ws: Optional[torch.Tensor] = None
        self.counters: Optional[torch.Tensor] = None


_gemm_ws: dict[int, _GemmWorkspace] = {}
_plan_cache: dict[tuple, tuple] = {}


def _plan(M: int, N: int, K: int):
    key = (M, N, K)
    p = _plan_cache.get(key)
    if p is None:
        swap, bn, splits, tiles = _i(), _i(), _i(), _i()
        wsb = _i64()
        _gemm_plan(M, N, K, num_sms(), ctypes.byref(swap), ctypes.byref(bn), ctypes.byref(splits), ctypes.byref(wsb),
                   ctypes.byref(tiles))
        p = (swap.value, bn.value, 1 if batch_invariant() else splits.value, wsb.value, tiles.value)
        _plan_cache[key] = p
    return p


def gemm_tc(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None,
            out: Optional[torch.Tensor] = None, act: int = 0, act_coef: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Y = X W^T on our tcgen05 kernel. x: [M, K] (row stride free), w: [N, K] contiguous.  ``act`` 1 (M <= 256): W's
    rows interleave (gate_i, up_i) and the epilogue emits silu(gate) * up → [M, N/2]; 3 (M <= 256): xIELU with ``act_coef``."""
    M, K = x.shape
    N = w.shape[0]
    swap, bn, splits, wsb, tiles = _plan(M, N, K)
    dev = x.device.index or 0
    g = _gemm_ws.setdefault(dev, _GemmWorkspace())
    if splits > 1:
        if g.ws is None or g.ws.numel() * 4 < wsb or g.counters.numel() < tiles:
            if torch.cuda.is_current_stream_capturing():
                raise RuntimeError("GEMM split-K workspace must be allocated before CUDA-graph capture")
            g.ws = torch.empty(max(wsb // 4, 16 << 20), dtype=torch.float32, device=x.device)
            g.counters = torch.zeros(max(tiles, 4096), dtype=torch.int32, device=x.device)
    y = out if out is not None else torch.empty((M, N // 2 if act == 1 else N), dtype=x.dtype, device=x.device)
    _check(_gemm_tc(x.data_ptr(), w.data_ptr(), _p(bias), y.data_ptr(), M, N, K, x.stride(0), swap, bn, splits,
                    _p(g.ws), _p(g.counters), int(act), _p(act_coef), _DT[x.dtype], _st()), f"gemm_tc(M={M},N={N},K={K})")
    return y


_gemm_sk_plan = _sig("vb_gemm_sk_plan", _i, _i, _i, _i, ctypes.POINTER(_i), ctypes.POINTER(_i), ctypes.POINTER(_i),
                     ctypes.POINTER(_i64), ctypes.POINTER(_i))
_gemm_sk = _sig("vb_gemm_sk", _vp, _vp, _vp, _vp, _i, _i, _i, _i64, _i, _i, _i, _vp, _vp, _i, _i, _vp)
_sk_plan_cache: dict[tuple, tuple] = {}
_sk_ws: dict[int, tuple] = {}


def _sk_workspace(dev: torch.device) -> tuple:
    """Stream-K partial-tile workspace + tile counters, sized once for the largest plan (SMs x 2 slots x 256 x 128 fp32)."""
    key = dev.index or 0
    ws = _sk_ws.get(key)
    if ws is None:
        if torch.cuda.is_current_stream_capturing():
            raise RuntimeError("stream-K GEMM workspace must be allocated before CUDA-graph capture")
        ws = _sk_ws[key] = (torch.empty(num_sms() * 2 * 256 * 128, dtype=torch.float32, device=dev),
                            torch.zeros(16384, dtype=torch.int32, device=dev))
    return ws


def gemm_sk(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None,
            act: bool = False) -> torch.Tensor:
    """Y = X W^T on the persistent stream-K tcgen05 kernel (csrc/gemm_sk.cu), M <= 256.  ``act``: W's rows are
    interleaved (gate_i, up_i) pairs and the epilogue emits silu(gate) * up ([M, N/2])."""
    M, K = x.shape
    N = w.shape[0]
    key = (M, N, K)
    plan = _sk_plan_cache.get(key)
    if plan is None:
        bn, grid, per, tiles = _i(), _i(), _i(), _i()
        wsb = _i64()
        rc = _gemm_sk_plan(M, N, K, num_sms(), ctypes.byref(bn), ctypes.byref(grid), ctypes.byref(per), ctypes.byref(wsb),
                           ctypes.byref(tiles))
        assert rc == 0 and tiles.value <= 16384
        plan = _sk_plan_cache[key] = (bn.value, grid.value, per.value)
    bn, grid, per = plan
    ws, counters = _sk_workspace(x.device)
    y = out if out is not None else torch.empty((M, N // 2 if act else N), dtype=x.dtype, device=x.device)
    _check(_gemm_sk(x.data_ptr(), w.data_ptr(), _p(bias), y.data_ptr(), M, N, K, x.stride(0), bn, grid, per, ws.data_ptr(),
                    counters.data_ptr(), int(act), _DT[x.dtype], _st()), f"gemm_sk(M={M},N={N},K={K})")
    return y


def _tc_ok(x2: torch.Tensor, w: torch.Tensor, force: bool = False) -> bool:
    mode = envs.VLLM_B200_GEMM
    if mode == "cublas" and not force:
        return False
    K = x2.shape[1]
    ok = (x2.dtype in (torch.bfloat16, torch.float16) and w.dtype == x2.dtype and K % 64 == 0
          and x2.stride(1) == 1 and (x2.stride(0) * 2) % 16 == 0 and x2.data_ptr() % 16 == 0 and w.is_contiguous())
    if mode == "tcgen05" or force:
        return ok
    # auto: our kernel for the weight-streaming decode shapes, cuBLASLt for the rest
    return ok and x2.shape[0] <= 256


def linear(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    K = x.shape[-1]
    x2 = x.reshape(-1, K)
    if x2.shape[0] > 0 and _tc_ok(x2, weight):
        # decode shapes: persistent stream-K kernel (every SM streams weights all the time); VLLM_B200_GEMM_SK=0 selects
        # the tile-per-CTA / cluster split-K kernel for A/B measurements
        if x2.shape[0] <= 256 and envs.VLLM_B200_GEMM_SK and weight.shape[0] * (K // 64) >= 64:
            y = gemm_sk(x2, weight, bias)
        else:
            y = gemm_tc(x2, weight, bias)
        return y.view(x.shape[:-1] + (weight.shape[0],))
    return torch.nn.functional.linear(x, weight, bias)


# ------------------------------------------------------------------ symmetric-heap collectives
_comm_ar_rows = _sig("vb_comm_allreduce_rows", _vp, _vp, _vp, _vp, _i, _i, _vp, _i64, _i64, _vp, _vp, _f, _i, _i, _i,
                     _i, _i, _vp)
_comm_ag = _sig("vb_comm_all_gather", _vp, _vp, _vp, _vp, _i, _i, _vp, _i64, _i, _i, _i, _i, _vp)
_comm_bar = _sig("vb_comm_barrier", _vp, _vp, _vp, _vp, _i, _i, _vp)


def comm_allreduce_rows(c, x, in_off, out_off, residual, norm_w, eps, T, H, gemma, dtype) -> None:
    _check(_comm_ar_rows(c.local_ptr, c.peer_arr, c._mc(), c.state.data_ptr(), c.rank, c.world, _p(x), in_off,
                         out_off, _p(residual), _p(norm_w), eps, T, H, int(gemma), num_sms(), _DT[dtype], _st()),
           "comm_allreduce_rows")


_comm_ar_oneshot = _sig("vb_comm_allreduce_oneshot", _vp, _vp, _vp, _vp, _i, _i, _vp, _i64, _vp, _i, _i, _i, _i, _vp)


def comm_allreduce_oneshot(c, x, in_off, dst, T, H) -> None:
    """Sum over ranks of [T,H] (``x`` or what already sits in the staging region) straight into the private ``dst``."""
    _check(_comm_ar_oneshot(c.local_ptr, c.peer_arr, c._mc(), c.state.data_ptr(), c.rank, c.world, _p(x), in_off,
                            dst.data_ptr(), T, H, num_sms(), _DT[dst.dtype], _st()), "comm_allreduce_oneshot")


def comm_all_gather(c, x, out_off, rows, cols) -> None:
    _check(_comm_ag(c.local_ptr, c.peer_arr, c._mc(), c.state.data_ptr(), c.rank, c.world, x.data_ptr(), out_off,
                    rows, cols, num_sms(), _DT[x.dtype], _st()), "comm_all_gather")


_gemm_ar_plan = _sig("vb_gemm_ar_plan", _i, _i, _i, _i, ctypes.POINTER(_i), ctypes.POINTER(_i), ctypes.POINTER(_i64),
                     ctypes.POINTER(_i))
_gemm_ar = _sig("vb_gemm_ar", _vp, _vp, _vp, _vp, _i, _i, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i64, _i, _i, _vp, _vp,
                _i64, _i64, _i, _i, _i64, _i64, _f, _i, _i, _vp)
_ar_plan_cache: dict[tuple, Optional[tuple]] = {}


def gemm_ar(c, x, w, residual, norm_w, out, eps, gemma, mode=0, oring_off=0, oring_stride=0) -> bool:
    """Fused RowParallel GEMM + all-reduce + residual + RMSNorm (csrc/gemm_ar.cu). False = shape not covered."""
    from vllm_b200.parallel.symm import LAM_T_CAP
    M, K = x.shape
    N = w.shape[0]
    key = (M, N, K)
    plan = _ar_plan_cache.get(key, 0)
    if plan == 0:
        bn, splits, tiles = _i(), _i(), _i()
        wsb = _i64()
        rc = _gemm_ar_plan(M, N, K, num_sms(), ctypes.byref(bn), ctypes.byref(splits), ctypes.byref(wsb),
                           ctypes.byref(tiles))
        plan = (bn.value, splits.value, wsb.value, tiles.value) if rc == 0 else None
        _ar_plan_cache[key] = plan
    if plan is None:
        return False
    bn, splits, wsb, tiles = plan
    dev = x.device.index or 0
    g = _gemm_ws.setdefault(dev, _GemmWorkspace())
    if g.ws is None or g.ws.numel() * 4 < wsb or g.counters.numel() < tiles:
        if torch.cuda.is_current_stream_capturing():
            raise RuntimeError("GEMM split-K workspace must be allocated before CUDA-graph capture")
        g.ws = torch.empty(max(wsb // 4, 16 << 20), dtype=torch.float32, device=x.device)
        g.counters = torch.zeros(max(tiles, 4096), dtype=torch.int32, device=x.device)
    _check(_gemm_ar(c.local_ptr, c.peer_arr, c._mc(), c.state.data_ptr(), c.rank, c.world, x.data_ptr(), w.data_ptr(),
                    residual.data_ptr(), norm_w.data_ptr(), out.data_ptr() if out is not None else None, M, N, K,
                    x.stride(0), bn, splits, g.ws.data_ptr(), g.counters.data_ptr(), c.off_lam, c.lam_stride, LAM_T_CAP, mode, oring_off, oring_stride, eps,
                    int(gemma),
                    _DT[x.dtype], _st()), f"gemm_ar(M={M},N={N},K={K})")
    return True


def gemm_ar_set_trace(t: Optional[torch.Tensor]) -> None:
    """Point the fused kernel's phase stamps ([n_ctas, 8] int64 globaltimer values) at ``t`` (None = off)."""
    fn = _library_for("vb_gemm_ar_set_trace").vb_gemm_ar_set_trace
    fn.argtypes, fn.restype = [_vp], None
    fn(t.data_ptr() if t is not None else None)


def comm_barrier(c) -> None:
    _check(_comm_bar(c.local_ptr, c.peer_arr, c._mc(), c.state.data_ptr(), c.rank, c.world, _st()), "comm_barrier")


# ------------------------------------------------------------------ MoE (csrc/moe.cu + grouped mode of gemm_tc.cu)
_moe_topk = _sig("vb_moe_topk_softmax", _vp, _vp, _vp, _i, _i, _i, _i, _f, _i, _vp)
_moe_align = _sig("vb_moe_align2", _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _vp, _vp)
_moe_finish = _sig("vb_moe_finish", _vp, _vp, _vp, _vp, _i, _i, _f, _i, _i, _vp)
_gemm_grouped_red = _sig("vb_gemm_tc_grouped_red", _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _vp, _vp, _i64, _i, _i, _vp, _vp, _i, _i,
                         _i, _vp)
_comm_ar_rows2 = _sig("vb_comm_allreduce_rows2", _vp, _vp, _vp, _vp, _i, _i, _vp, _i64, _i64, _vp, _vp, _f, _i, _i, _i, _i, _i64,
                      _i, _vp)
_moe_combine = _sig("vb_moe_combine", _vp, _vp, _vp, _vp, _i, _i, _i, _i, _vp)
_moe_gather = _sig("vb_moe_gather", _vp, _vp, _vp, _i, _i, _i, _vp)
_gemm_grouped = _sig("vb_gemm_tc_grouped2", _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i, _i, _vp)
_grouped_simt = _sig("vb_moe_grouped_simt", _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _vp)
_grouped_topk = _sig("vb_moe_grouped_topk", _vp, _vp, _i, _vp, _i, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i, _i, _f, _i, _vp)
_GROUPED_ACT = {None: 0, "none": 0, "relu2": 2}


def topk_softmax(gating, k, renormalize, scale: float = 1.0):
    T, E = gating.shape
    if E > 512 or k > 32 or gating.dtype not in _DT or not gating.is_contiguous():
        from vllm_b200.ops import ref
        w, ids = ref.topk_softmax(gating, k, renormalize)
        return w * scale, ids
    w = torch.empty((T, k), dtype=torch.float32, device=gating.device)
    ids = torch.empty((T, k), dtype=torch.int32, device=gating.device)
    _check(_moe_topk(gating.data_ptr(), w.data_ptr(), ids.data_ptr(), T, E, k, int(renormalize), float(scale),
                     _DT[gating.dtype], _st()), "moe_topk_softmax")
    return w, ids


def moe_align(topk_ids: torch.Tensor, num_local_experts: int, expert_map: Optional[torch.Tensor] = None,
              with_pairs: bool = False):
    """(sorted_tok [R], inv [R], offs [E+1]) for R = T*k (token, slot) pairs — all on the device.  ``with_pairs`` also
    returns sorted_pair [R]: the pair index (token * k + slot) of every sorted row."""
    T, k = topk_ids.shape
    R = T * k
    dev = topk_ids.device
    sorted_tok = torch.empty(R, dtype=torch.int32, device=dev)
    inv = torch.empty(R, dtype=torch.int32, device=dev)
    offs = torch.empty(num_local_experts + 1, dtype=torch.int32, device=dev)
    pairs = torch.empty(R, dtype=torch.int32, device=dev) if with_pairs else None
    _check(_moe_align(topk_ids.data_ptr(), _p(expert_map), sorted_tok.data_ptr(), inv.data_ptr(), offs.data_ptr(), R, k,
                      num_local_experts, _p(pairs), _st()), "moe_align")
    return (sorted_tok, inv, offs, pairs) if with_pairs else (sorted_tok, inv, offs)


def gemm_tc_grouped_combine(xs, w, offs, bn, sorted_pair, pair_w, k: int, H: int, *, acc_ptr: int = 0, comm=None,
                            acc_off: int = 0, per: int = 1) -> None:
    """Grouped GEMM whose epilogue adds w(row) * y[row] into the fp32 accumulator row of its token: a local buffer
    (``acc_ptr``) on one GPU; with ``comm`` the buffer at ``acc_off`` of the symmetric heap OF THE RANK THAT OWNS THE
    TOKEN (token // per), reached with red.add over NVLink → top-k combine + reduce-scatter inside the GEMM."""
    R, K = xs.shape
    E, N, _ = w.shape
    if comm is not None:
        rc = _gemm_grouped_red(xs.data_ptr(), w.data_ptr(), None, offs.data_ptr(), R, N, K, E, bn, comm.local_ptr + acc_off,
                               comm.peer_arr, acc_off, comm.world, per, sorted_pair.data_ptr(), pair_w.data_ptr(), k, H,
                               _DT[xs.dtype], _st())
    else:
        rc = _gemm_grouped_red(xs.data_ptr(), w.data_ptr(), None, offs.data_ptr(), R, N, K, E, bn, acc_ptr, None, 0, 1, 1,
                               sorted_pair.data_ptr(), pair_w.data_ptr(), k, H, _DT[xs.dtype], _st())
    _check(rc, f"gemm_tc_grouped_combine(R={R},N={N},K={K},E={E})")


def comm_finish_rows_acc32(c, acc_off: int, out_off: int, residual, norm_w, eps, T, H, gemma, dtype) -> None:
    """Second half of the fused MoE tail under TP/EP: barrier → every rank reads (and re-zeroes) the fp32 sums of the
    rows it owns, adds its residual rows, normalises and multicasts the rows → barrier (csrc/comm.cu ar_rows_kernel)."""
    _check(_comm_ar_rows2(c.local_ptr, c.peer_arr, c._mc(), c.state.data_ptr(), c.rank, c.world, None, c.off_in, out_off,
                          _p(residual), _p(norm_w), eps, T, H, int(gemma), num_sms(), acc_off, _DT[dtype], _st()),
           "comm_finish_rows_acc32")


def moe_finish(acc_ptr: int, residual, norm_w, out, T: int, H: int, eps: float, gemma: bool = False) -> None:
    _check(_moe_finish(acc_ptr, _p(residual), _p(norm_w), out.data_ptr(), T, H, eps, int(gemma), _DT[out.dtype], _st()),
           "moe_finish")


def moe_gather(x: torch.Tensor, sorted_tok: torch.Tensor) -> torch.Tensor:
    R, H = sorted_tok.numel(), x.shape[1]
    xs = torch.empty((R, H), dtype=x.dtype, device=x.device)
    _check(_moe_gather(x.data_ptr(), sorted_tok.data_ptr(), xs.data_ptr(), R, H, _DT[x.dtype], _st()), "moe_gather")
    return xs


def moe_combine(y: torch.Tensor, inv: torch.Tensor, w: torch.Tensor, T: int) -> torch.Tensor:
    H = y.shape[1]
    k = inv.numel() // T
    out = torch.empty((T, H), dtype=y.dtype, device=y.device)
    if y.dtype in _HALF_DTYPES and H % 8 == 0:
        _check(_moe_combine(y.data_ptr(), inv.data_ptr(), w.data_ptr(), out.data_ptr(), T, H, k, _DT[y.dtype], _st()),
               "moe_combine")
    else:
        _check(_post_norm(y.data_ptr(), y.stride(0), inv.data_ptr(), w.data_ptr(), k, None, 0, None, None, 0, out.data_ptr(), T, H,
                          0.0, _DT[y.dtype], _st()), "moe_combine")
    return out


def gemm_tc_grouped(xs: torch.Tensor, w: torch.Tensor, offs: torch.Tensor, bn: int, act: Optional[str] = None,
                    flat: bool = False) -> torch.Tensor:
    """Y[r] = act(xs[r] · w[e(r)]^T), rows sorted by expert (``offs``). w: [E, N, K].  ``flat``: the grid follows the row
    count (large batches) instead of every chunk an expert could have."""
    R, K = xs.shape
    E, N, _ = w.shape
    y = torch.empty((R, N), dtype=xs.dtype, device=xs.device)
    _check(_gemm_grouped(xs.data_ptr(), w.data_ptr(), y.data_ptr(), offs.data_ptr(), R, N, K, E, bn, _GROUPED_ACT[act], int(flat),
                         _DT[xs.dtype], _st()), f"gemm_tc_grouped(R={R},N={N},K={K},E={E})")
    return y


def grouped_simt(x: torch.Tensor, w: torch.Tensor, offs: torch.Tensor, R: int, row_tok: Optional[torch.Tensor] = None,
                 act: Optional[str] = None) -> torch.Tensor:
    """The grouped product on the CUDA cores (any dtype and row width); ``row_tok`` gathers rows of x on the way in."""
    E, N, K = w.shape
    assert x.is_contiguous() and w.is_contiguous() and x.dtype == w.dtype
    y = torch.empty((R, N), dtype=x.dtype, device=x.device)
    _check(_grouped_simt(x.data_ptr(), w.data_ptr(), y.data_ptr(), offs.data_ptr(), _p(row_tok), R, N, K, E, _GROUPED_ACT[act],
                         _DT[x.dtype], _st()), f"grouped_simt(R={R},N={N},K={K},E={E})")
    return y


def grouped_topk(scores, k, n_group, topk_group, renormalize, scoring="sigmoid", bias=None, routed_scaling_factor=1.0, group_score=None):
    T, E = scores.shape
    lg = scores.float().contiguous()
    w = torch.empty((T, k), dtype=torch.float32, device=scores.device)
    ids = torch.empty((T, k), dtype=torch.int32, device=scores.device)
    b = None if bias is None else bias.float().contiguous()
    _check(_grouped_topk(lg.data_ptr(), None, 0, None, 0, _p(b), w.data_ptr(), ids.data_ptr(), T, E, k, n_group,
                         topk_group if n_group > 1 else 1, _group_top2(group_score, bias), int(scoring != "sigmoid"), int(renormalize),
                         float(routed_scaling_factor), 2, _st()), f"grouped_topk(E={E},k={k})")
    return w, ids


def _group_top2(group_score: Optional[str], bias) -> int:
    return int(bias is not None if group_score is None else group_score == "top2")


ROUTER_FUSED_TOKENS = 256       # above this the logits come from one tensor-core product with fp32 output


def router_topk(x, gate, k, n_group, topk_group, renormalize, scoring="sigmoid", bias=None, routed_scaling_factor=1.0, x_half=None,
                group_score=None):
    """Routing of x [T, H] (fp32 stream or model dtype) with gate [E, H]: 32-bit logits, scores, choice and weights.
    ``x_half``: the 16-bit copy of x for the large-batch product."""
    T, H = x.shape
    E = gate.shape[0]
    if T > ROUTER_FUSED_TOKENS or H > 8192:
        xh = x if x.dtype == gate.dtype else x_half
        if gate.dtype == torch.float32 or xh is None:
            lg = x.float() @ gate.float().t()
        else:
            lg = torch.mm(xh, gate.t(), out_dtype=torch.float32)
        return grouped_topk(lg, k, n_group, topk_group, renormalize, scoring, bias, routed_scaling_factor, group_score)
    w = torch.empty((T, k), dtype=torch.float32, device=x.device)
    ids = torch.empty((T, k), dtype=torch.int32, device=x.device)
    assert x.is_contiguous() and gate.is_contiguous() and (x.dtype == torch.float32 or x.dtype == gate.dtype)
    assert bias is None or bias.dtype == torch.float32
    _check(_grouped_topk(None, x.data_ptr(), int(x.dtype == torch.float32), gate.data_ptr(), H, _p(bias), w.data_ptr(),
                         ids.data_ptr(), T, E, k, n_group, topk_group if n_group > 1 else 1, _group_top2(group_score, bias),
                         int(scoring != "sigmoid"), int(renormalize), float(routed_scaling_factor), _DT[gate.dtype], _st()), f"router_topk(E={E},k={k},H={H})")
    return w, ids


def fused_moe(x, w13, w2, topk_w, topk_ids, act="silu", expert_map=None, gated: bool = True, on_device: bool = False):
    from vllm_b200.ops import moe
    if not gated or on_device:
        return moe.fused_moe_rows(x, w13, w2, topk_w, topk_ids, act, expert_map, gated)
    return moe.fused_moe_cuda(x, w13, w2, topk_w, topk_ids, act, expert_map)


_gemm_fp8_plan = _sig("vb_gemm_fp8_plan", _i, _i, _i, ctypes.POINTER(_i), ctypes.POINTER(_i), ctypes.POINTER(_i))
_gemm_fp8 = _sig("vb_gemm_fp8", _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i64, _i64, _i, _i, _i, _i, _i, _i, _i, _vp)
_gemm_fp8_grouped = _sig("vb_gemm_fp8_grouped", _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i64, _i, _i, _vp)
_fp8_plan_cache: dict[tuple, tuple] = {}


def _fp8_plan(M: int, N: int, K: int) -> tuple:
    key = (M, N, K)
    p = _fp8_plan_cache.get(key)
    if p is None:
        swap, bn, splits = _i(), _i(), _i()
        _gemm_fp8_plan(M, N, K, ctypes.byref(swap), ctypes.byref(bn), ctypes.byref(splits))
        p = _fp8_plan_cache[key] = (swap.value, bn.value, 1 if batch_invariant() else splits.value)
    return p


def gemm_fp8_block(xq, xs, wq, ws, out_dtype=torch.bfloat16, bias=None, out=None):
    """Block-scaled fp8 GEMM (tcgen05 kind::f8f6f4, csrc/gemm_fp8.cu).  xq [M, K] e4m3; xs [M, K/128] fp32 with
    stride(0) == 1 (the column-major output of ``per_token_group_quant_fp8(col_major=True)``); wq [N, K] e4m3;
    ws [ceil(N/128), K/128] fp32."""
    M, K = xq.shape
    N = wq.shape[0]
    assert xs.stride(0) == 1 and ws.is_contiguous() and wq.is_contiguous() and xq.stride(1) == 1
    swap, bn, splits = _fp8_plan(M, N, K)
    y = out if out is not None else torch.empty((M, N), dtype=out_dtype, device=xq.device)
    _check(_gemm_fp8(xq.data_ptr(), wq.data_ptr(), xs.data_ptr(), ws.data_ptr(), _p(bias), y.data_ptr(), M, N, K,
                     xq.stride(0), xs.stride(1), 0, 1, 1, swap, bn, splits, _DT[y.dtype], _st()),
           f"gemm_fp8_block(M={M},N={N},K={K})")
    return y


def gemm_fp8_scaled(xq, wq, scale_a, scale_b, out_dtype=torch.bfloat16, bias=None):
    """W8A8 fp8 GEMM with per-token / per-tensor activation scales and per-channel / per-tensor weight scales
    (the reference's ``cutlass_scaled_mm`` contract): y = (xq · wq^T) * scale_a[:, None] * scale_b[None, :]."""
    M, K = xq.shape
    N = wq.shape[0]
    swap, bn, splits = _fp8_plan(M, N, K)
    y = torch.empty((M, N), dtype=out_dtype, device=xq.device)
    sa, sb = scale_a.reshape(-1).float().contiguous(), scale_b.reshape(-1).float().contiguous()
    _check(_gemm_fp8(xq.data_ptr(), wq.data_ptr(), sa.data_ptr(), sb.data_ptr(), _p(bias), y.data_ptr(), M, N, K,
                     xq.stride(0), 0, 1, int(sa.numel() > 1), int(sb.numel() > 1), swap, bn, splits, _DT[y.dtype], _st()),
           f"gemm_fp8_scaled(M={M},N={N},K={K})")
    return y


def gemm_fp8_grouped(xq, xs, wq, ws, offs, bn: int, out_dtype=torch.bfloat16):
    """Grouped (MoE) block-scaled fp8 GEMM: rows of xq sorted by expert (``offs``), wq [E, N, K], ws [E, N/128, K/128]."""
    R, K = xq.shape
    E, N, _ = wq.shape
    y = torch.empty((R, N), dtype=out_dtype, device=xq.device)
    _check(_gemm_fp8_grouped(xq.data_ptr(), wq.data_ptr(), xs.data_ptr(), ws.data_ptr(), y.data_ptr(), offs.data_ptr(), R, N,
                             K, E, xs.stride(1), bn, _DT[y.dtype], _st()), f"gemm_fp8_grouped(R={R},N={N},K={K},E={E})")
    return y


def block_fp8_linear(x, wq, w_scale, block=128, bias=None):
    """Activations quantised per (token, 128-group) on the fly, weights per 128x128 block: fused quantiser kernel +
    tcgen05 block-scaled GEMM.  Shapes the kernel does not cover take the fp32 reference."""
    K = x.shape[-1]
    x2 = x.reshape(-1, K)
    if (block == 128 and K % 128 == 0 and x2.dtype in (torch.bfloat16, torch.float16) and x2.shape[0] > 0
            and wq.dtype == torch.float8_e4m3fn and wq.is_contiguous() and w_scale.dtype == torch.float32):
        xq, xs = per_token_group_quant_fp8(x2, 128, col_major=True)
        y = gemm_fp8_block(xq, xs, wq, w_scale.contiguous(), x.dtype, bias)
        return y.view(x.shape[:-1] + (wq.shape[0],))
    from vllm_b200.ops import ref
    return ref.block_fp8_linear(x, wq, w_scale, block, bias)


def scaled_mm(a, b, scale_a, scale_b, out_dtype, bias=None):
    if (a.dtype == torch.float8_e4m3fn and b.dtype == torch.float8_e4m3fn and a.shape[1] % 16 == 0 and a.stride(1) == 1
            and b.is_contiguous() and out_dtype in (torch.bfloat16, torch.float16) and (a.stride(0) % 16) == 0):
        return gemm_fp8_scaled(a, b, scale_a, scale_b, out_dtype, bias)
    from vllm_b200.ops import ref
    return ref.scaled_mm(a, b, scale_a, scale_b, out_dtype, bias)


# ------------------------------------------------------------------ LoRA (csrc/lora.cu)
_lora_shrink = _sig("vb_lora_shrink", _vp, _i64, _vp, _vp, _vp, _i, _i, _i, _i, _i, _vp)
_lora_expand = _sig("vb_lora_expand", _vp, _i64, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i, _i, _vp)


def lora_bgmv(x, y, A, B, token_slots, offs) -> None:
    """y[t] += B[slot(t)] (A[slot(t)] x[t]) for every token with slot >= 0, in place.  A [S, n_sub, r, K],
    B [S, N, r] (scaling folded in), ``offs`` = (n_sub, o1, o2, o3) sub-projection boundaries of the N outputs."""
    T, K = x.shape
    N, r = B.shape[1], B.shape[2]
    n_sub, o1, o2, o3 = offs
    v = torch.empty((T, n_sub, r), dtype=torch.float32, device=x.device)
    _check(_lora_shrink(x.data_ptr(), x.stride(0), A.data_ptr(), token_slots.data_ptr(), v.data_ptr(), T, K, r, n_sub,
                        _DT[x.dtype], _st()), "lora_shrink")
    _check(_lora_expand(y.data_ptr(), y.stride(0), B.data_ptr(), token_slots.data_ptr(), v.data_ptr(), T, N, r, n_sub,
                        o1, o2, o3, _DT[y.dtype], _st()), "lora_expand")


# ------------------------------------------------------------------ activation quantisation (csrc/quant.cu)
_quant_rows = _sig("vb_quant_rows", _vp, _i64, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i, _i, _i, _i, _f, _f, _i,
                   _vp)
_absmax_scale = _sig("vb_absmax_scale", _vp, _i64, _i64, _i64, _vp, _vp, _f, _i, _i, _vp)
_fp4_quant = _sig("vb_fp4_quant", _vp, _i64, _vp, _vp, _vp, _i, _i, _i, _i, _i, _vp)
_Q_FP8_STATIC, _Q_FP8_TOKEN, _Q_FP8_GROUP, _Q_INT8_TOKEN, _Q_INT8_STATIC = range(5)
_PRE_NONE, _PRE_RMS, _PRE_ACT = range(3)
_amax_scratch: dict[int, torch.Tensor] = {}


def _quant_call(x2, H, pre, qm, out_dtype, *, residual=None, weight=None, scale_in=None, group=128, col_major=False,
                ue8m0=False, gemma=False, act=0, eps=0.0, scale_ub=0.0):
    T = x2.shape[0]
    dev = x2.device
    q = torch.empty((T, H), dtype=out_dtype, device=dev)
    scale = None
    stride = 0
    if qm in (_Q_FP8_TOKEN, _Q_INT8_TOKEN):
        scale = torch.empty((T, 1), dtype=torch.float32, device=dev)
    elif qm == _Q_FP8_GROUP:
        G = H // group
        if col_major:
            stride = (T + 3) // 4 * 4            # TMA-friendly leading dimension
            scale = torch.empty((G, stride), dtype=torch.float32, device=dev)
        else:
            scale = torch.empty((T, G), dtype=torch.float32, device=dev)
    _check(_quant_rows(x2.data_ptr(), x2.stride(0), _p(residual), _p(weight), q.data_ptr(), _p(scale), _p(scale_in), T, H,
                       pre, qm, group, int(col_major), stride, int(ue8m0), int(gemma), act, eps, scale_ub, _DT[x2.dtype],
                       _st()), "quant_rows")
    if qm == _Q_FP8_GROUP and col_major:
        scale = scale[:, :T].t()                 # logical [T, G] view over the column-major storage
    return q, scale


def _rows(x):
    x2 = x.reshape(-1, x.shape[-1])
    if x2.stride(-1) != 1:
        x2 = x2.contiguous()
    return x2


def dynamic_scale(x: torch.Tensor, qmax: float = 448.0) -> torch.Tensor:
    """scale[0] = max|x| / qmax on the device (pass 1 of dynamic per-tensor quantisation)."""
    x2 = _rows(x)
    dev = x2.device.index or 0
    scr = _amax_scratch.get(dev)
    if scr is None:
        if torch.cuda.is_current_stream_capturing():
            raise RuntimeError("dynamic per-tensor quantisation scratch must exist before CUDA-graph capture")
        scr = _amax_scratch[dev] = torch.zeros(1, dtype=torch.int32, device=x2.device)
    scale = torch.empty(1, dtype=torch.float32, device=x2.device)
    _check(_absmax_scale(x2.data_ptr(), x2.shape[0], x2.shape[1], x2.stride(0), scr.data_ptr(), scale.data_ptr(), qmax,
                         num_sms(), _DT[x2.dtype], _st()), "absmax_scale", 2)
    return scale


def scaled_fp8_quant(x, scale=None, per_token: bool = False, scale_ub: float = 0.0):
    x2 = _rows(x)
    H = x2.shape[1]
    if per_token:
        q, s = _quant_call(x2, H, _PRE_NONE, _Q_FP8_TOKEN, torch.float8_e4m3fn, scale_ub=scale_ub)
        return q.view(x.shape), s.view(x.shape[:-1] + (1,))
    if scale is None:
        scale = dynamic_scale(x2)
    q, _ = _quant_call(x2, H, _PRE_NONE, _Q_FP8_STATIC, torch.float8_e4m3fn, scale_in=scale.reshape(-1))
    return q.view(x.shape), scale


def scaled_int8_quant(x, scale=None):
    x2 = _rows(x)
    H = x2.shape[1]
    if scale is None:
        q, s = _quant_call(x2, H, _PRE_NONE, _Q_INT8_TOKEN, torch.int8)
        return q.view(x.shape), s.view(x.shape[:-1] + (1,))
    q, _ = _quant_call(x2, H, _PRE_NONE, _Q_INT8_STATIC, torch.int8, scale_in=scale.reshape(-1))
    return q.view(x.shape), scale


def per_token_group_quant_fp8(x, group: int = 128, col_major: bool = False, ue8m0: bool = False):
    x2 = _rows(x)
    H = x2.shape[1]
    if H % group or group not in (32, 64, 128) or H % 8 or x2.dtype not in (torch.bfloat16, torch.float16):
        from vllm_b200.ops import ref
        return ref.per_token_group_quant_fp8(x2, group)
    return _quant_call(x2, H, _PRE_NONE, _Q_FP8_GROUP, torch.float8_e4m3fn, group=group, col_major=col_major, ue8m0=ue8m0)


def rms_norm_quant(x, weight, eps, *, residual=None, scale=None, mode: str = "static", group: int = 128,
                   gemma: bool = False, col_major: bool = False, ue8m0: bool = False):
    """Fused (residual add +) RMSNorm + fp8 quantisation.  mode: static | token | group.  ``residual`` is updated in
    place (residual += x) like fused_add_rms_norm.  Returns (q, scale)."""
    x2 = _rows(x)
    H = x2.shape[1]
    qm = {"static": _Q_FP8_STATIC, "token": _Q_FP8_TOKEN, "group": _Q_FP8_GROUP}[mode]
    if residual is not None:
        assert residual.is_contiguous()
    q, s = _quant_call(x2, H, _PRE_RMS, qm, torch.float8_e4m3fn, residual=residual, weight=weight, eps=eps, gemma=gemma,
                       scale_in=None if scale is None else scale.reshape(-1), group=group, col_major=col_major,
                       ue8m0=ue8m0)
    return q.view(x.shape), (scale if mode == "static" else s)


def act_mul_quant(x, act: str = "silu", *, scale=None, mode: str = "static", group: int = 128, col_major: bool = False,
                  ue8m0: bool = False):  # noqa: D401
    """Fused act(gate) * up + fp8 quantisation over x[..., 2H] → (q[..., H], scale)."""
    x2 = _rows(x)
    H = x2.shape[1] // 2
    qm = {"static": _Q_FP8_STATIC, "token": _Q_FP8_TOKEN, "group": _Q_FP8_GROUP}[mode]
    a = {"silu": 0, "gelu": 1, "gelu_tanh": 2, "gelu_pytorch_tanh": 2}[act]
    q, s = _quant_call(x2, H, _PRE_ACT, qm, torch.float8_e4m3fn, act=a, scale_in=None if scale is None else scale.reshape(-1),
                       group=group, col_major=col_major, ue8m0=ue8m0)
    return q.view(x.shape[:-1] + (H,)), (scale if mode == "static" else s)


def scaled_fp4_quant(x, global_scale=None, mx: bool = False, swizzled: bool = False):
    """NVFP4 (block 16, e4m3 block scales x fp32 ``global_scale``) or MXFP4 (block 32, e8m0 scales).
    Returns (packed uint8 [T, H/2], block scales uint8 [T, H/16 or H/32] — or the 128x4-tiled buffer if swizzled)."""
    x2 = _rows(x)
    T, H = x2.shape
    blk = 32 if mx else 16
    q = torch.empty((T, H // 2), dtype=torch.uint8, device=x2.device)
    G = H // blk
    if swizzled:
        sf = torch.zeros(((T + 127) // 128) * ((G + 3) // 4) * 512, dtype=torch.uint8, device=x2.device)
    else:
        sf = torch.empty((T, G), dtype=torch.uint8, device=x2.device)
    if global_scale is None and not mx:
        global_scale = torch.ones(1, dtype=torch.float32, device=x2.device)
    _check(_fp4_quant(x2.data_ptr(), x2.stride(0), q.data_ptr(), sf.data_ptr(), _p(global_scale), T, H, int(mx),
                      int(swizzled), _DT[x2.dtype], _st()), "fp4_quant")
    return q, sf


# ------------------------------------------------------------------ q/k norm + RoPE + cache (csrc/qknorm_rope.cu)
_qknorm_rope = _sig("vb_qknorm_rope_cache", _vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i64, _i64, _i64, _vp,
                    _vp, _i, _i, _i, _i, _f, _f, _f, _i, _vp)


def qknorm_rope_ok(head_dim: int, rot: int, is_neox: bool) -> bool:
    E = head_dim // 32
    if head_dim % 32 or E not in (2, 4, 8, 16):
        return False
    if rot:
        if is_neox:
            half = rot // 2
            if half % E:
                return False
            span = half // E
            return span & (span - 1) == 0
        return E % 2 == 0
    return True


_qknorm_rope_any = _sig("vb_qknorm_rope_any", _vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i, _i64, _i64, _i64, _vp,
                        _vp, _i, _i, _i, _i, _f, _i, _vp)


_qknorm_rope_row = _sig("vb_qknorm_rope_row", _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i, _i64, _i64, _i64, _vp,
                        _vp, _i, _i, _i, _i, _f, _i, _vp)


def fused_qk_norm_rope(positions, q, k, q_weight, k_weight, cos_sin_cache, head_dim, eps, is_neox=True, *, v=None,
                       kv_cache=None, slot_mapping=None, gemma: bool = False, k_scale: float = 1.0, v_scale: float = 1.0,
                       vt: bool = False, v_head_dim: Optional[int] = None, keep32: bool = False, whole: bool = False, v_cos_sin=None):
    """In place: per-head RMSNorm(q), RMSNorm(k) → RoPE → (optionally) K/V insert into the paged cache; one launch.
    ``keep32``: no rounding to the model dtype between the norm and the rotation.  ``whole``: one norm over all heads (weights as
    long); ``k`` may be None.  Weights None: no norms.  ``v_cos_sin``: values are rotated on their way into the cache."""
    T = q.shape[0]
    assert v_cos_sin is None or (not whole and v_cos_sin.shape[-1] == (v_head_dim or head_dim))
    Hq, Hkv = q.shape[-1] // head_dim, 0 if k is None else k.shape[-1] // head_dim
    rot = cos_sin_cache.shape[-1] if cos_sin_cache is not None else 0
    assert q.stride(-1) == 1 and (k is None or k.stride(-1) == 1)
    if whole:
        dv = v_head_dim or head_dim
        BS, dc = (kv_cache.shape[3], kv_cache.shape[4]) if kv_cache is not None else (1, max(head_dim, dv))
        assert kv_cache is None or kv_cache.dtype == q.dtype, "whole-projection norms write caches of the model dtype"
        _check(_qknorm_rope_row(_p(positions), q.data_ptr(), _p(k), _p(v), _p(q_weight), _p(k_weight), _p(cos_sin_cache), rot, T, Hq, Hkv,
                                head_dim, dv, dc, q.stride(0), 0 if k is None else k.stride(0), 0 if v is None else v.stride(0),
                                _p(kv_cache), _p(slot_mapping), BS, int(is_neox), int(gemma), int(vt), eps, _DT[q.dtype], _st()),
               "qknorm_rope_row")
        return q, k
    if (q_weight is None and k_weight is None and kv_cache is not None and v is not None and (v_head_dim or head_dim) == head_dim == kv_cache.shape[4]
            and q.dtype in _HALF_DTYPES and head_dim % 16 == 0 and rot % 16 == 0 and kv_cache.dtype == q.dtype
            and all(t.data_ptr() % 16 == 0 and t.stride(0) % 8 == 0 for t in (q, k, v))):
        # nothing to norm: the row kernel
        return rope_and_cache(positions, q, k, v, cos_sin_cache, head_dim, is_neox, kv_cache, slot_mapping, vt=vt, v_cos_sin=v_cos_sin)
    flags = 4 if keep32 else 0
    BS = 1
    dv = v_head_dim or head_dim
    dc = max(head_dim, dv)
    if kv_cache is not None:
        flags |= _kv_fp8(kv_cache) | (2 if vt else 0)
        BS, dc = kv_cache.shape[3], kv_cache.shape[4]
    step = min(head_dim // 32, 16 // q.element_size())          # elements of one vector access of the register kernel
    vec = all(t is None or (t.stride(0) % step == 0 and t.data_ptr() % (step * t.element_size()) == 0) for t in (q, k, v)) if step else False
    if not (q.dtype in _HALF_DTYPES and dv == dc == head_dim and vec and qknorm_rope_ok(head_dim, rot, is_neox)
            and (v_cos_sin is None or qknorm_rope_ok(head_dim, head_dim, is_neox))):
        assert not flags & 1, "this head shape needs a cache of the model dtype"
        _check(_qknorm_rope_any(_p(positions), q.data_ptr(), k.data_ptr(), _p(v), _p(q_weight), _p(k_weight), _p(cos_sin_cache),
                                _p(v_cos_sin), rot, T, Hq, Hkv, head_dim, dv, dc, q.stride(0), k.stride(0), v.stride(0) if v is not None else 0,
                                _p(kv_cache), _p(slot_mapping), BS, int(is_neox), int(gemma), int(vt), eps, _DT[q.dtype], _st()),
               "qknorm_rope_any")
        return q, k
    _check(_qknorm_rope(_p(positions), q.data_ptr(), k.data_ptr(), _p(v), _p(q_weight), _p(k_weight), _p(cos_sin_cache),
                        _p(v_cos_sin), rot, T, Hq, Hkv, head_dim, q.stride(0), k.stride(0), v.stride(0) if v is not None else 0,
                        _p(kv_cache), _p(slot_mapping), BS, int(is_neox), int(gemma), flags, eps, k_scale, v_scale,
                        _DT[q.dtype], _st()), "qknorm_rope_cache")
    return q, k


# ------------------------------------------------------------------ cache maintenance (csrc/cache_ops.cu)
_copy_blocks = _sig("vb_copy_blocks", _vp, _vp, _vp, _i, _i64, _vp)
_gather_cache = _sig("vb_gather_cache", _vp, _vp, _vp, _i64, _vp, _vp, _i, _i, _i, _i, _i64, _i64, _f, _i, _i, _vp)
_convert_fp8 = _sig("vb_convert_fp8", _vp, _vp, _i64, _f, _i, _i, _i, _vp)


def swap_blocks(src: torch.Tensor, dst: torch.Tensor, mapping) -> None:
    """dst[j] = src[i] for (i, j) in mapping; whole blocks (dim 0).  Either side may be pinned host memory."""
    if isinstance(mapping, torch.Tensor):
        m = mapping.to(torch.int64)
    else:
        if not mapping:
            return
        m = torch.tensor(mapping, dtype=torch.int64)
    dev = src.device if src.is_cuda else dst.device
    m = m.to(dev, non_blocking=True).contiguous()
    block_bytes = src[0].numel() * src.element_size()
    assert dst[0].numel() * dst.element_size() == block_bytes and src.is_contiguous() and dst.is_contiguous()
    assert block_bytes % 16 == 0
    for t in (src, dst):
        assert t.is_cuda or t.is_pinned(), "host side of swap_blocks must be pinned (mapped) memory"
    _check(_copy_blocks(src.data_ptr(), dst.data_ptr(), m.data_ptr(), m.shape[0], block_bytes, _st()), "copy_blocks")


def copy_blocks(cache: torch.Tensor, mapping) -> None:
    swap_blocks(cache, cache, mapping)


def gather_cache(cache, block_table, cu_seq_lens, out, max_tokens: int, seq_starts=None, scale: float = 1.0):
    """Dense [total_tokens, row] copy of the cached rows of a batch (cache [blocks, BS, row], fp8 → out.dtype with
    ``scale`` when the cache is 8-bit)."""
    B = cu_seq_lens.numel() - 1
    BS, row = cache.shape[1], cache.shape[2]
    src8 = cache.element_size() == 1
    _check(_gather_cache(cache.data_ptr(), out.data_ptr(), block_table.data_ptr(), block_table.stride(0),
                         cu_seq_lens.data_ptr(), _p(seq_starts), B, max_tokens, BS, row, cache.stride(0), out.stride(0),
                         scale, int(src8), _DT[out.dtype], _st()), "gather_cache")
    return out


def convert_fp8(x: torch.Tensor, scale: float = 1.0, to_fp8: bool = True, out_dtype=torch.bfloat16):
    xc = x.contiguous()
    n = xc.numel()
    if n % 8:
        from vllm_b200.ops import ref
        return ref.convert_fp8(x, scale, to_fp8)
    if to_fp8:
        out = torch.empty(xc.shape, dtype=torch.float8_e4m3fn, device=xc.device)
        _check(_convert_fp8(xc.data_ptr(), out.data_ptr(), n, scale, 1, num_sms(), _DT[xc.dtype], _st()), "convert_fp8")
    else:
        out = torch.empty(xc.shape, dtype=out_dtype, device=xc.device)
        _check(_convert_fp8(xc.data_ptr(), out.data_ptr(), n, scale, 0, num_sms(), _DT[out_dtype], _st()), "convert_fp8")
    return out


# ------------------------------------------------------------------ SSM / linear attention (csrc/ssm.cu, linear_attn.cu)
_conv1d = _sig("vb_causal_conv1d", _vp, _i64, _vp, _i64, _vp, _vp, _vp, _i64, _vp, _vp, _vp, _i64, _i, _i, _i, _i, _i, _i, _vp)
_sel_scan = _sig("vb_selective_scan", _vp, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i64, _i64, _vp, _vp, _vp, _i64, _i, _i, _i,
                 _vp)
_ssd_scan = _sig("vb_ssd_scan", _vp, _i64, _vp, _i64, _vp, _vp, _vp, _vp, _vp, _i64, _i64, _vp, _vp, _vp, _i64, _i, _i, _i, _i,
                 _i, _i, _f, _f, _i, _vp)
_gla_scan = _sig("vb_gla_scan", _vp, _vp, _vp, _i64, _i64, _i64, _f, _vp, _vp, _i64, _vp, _vp, _i, _f, _vp, _vp, _i64, _i64, _vp, _vp,
                 _vp, _i64, _i, _i, _i, _i, _i, _i, _vp)
_gla_decay = _sig("vb_gla_decay", _vp, _i64, _vp, _vp, _vp, _i, _i, _i, _f, _i, _vp)
_gated_norm = _sig("vb_gated_norm", _vp, _vp, _vp, _i64, _vp, _i, _vp, _i64, _i, _i, _i, _i, _f, _f, _i, _vp)
_memory_scan = _sig("vb_memory_scan", _vp, _vp, _vp, _i64, _i64, _i64, _f, _vp, _vp, _vp, _i64, _i64, _vp, _vp, _vp, _i64, _i, _i, _i, _i,
                    _i, _i, _vp)
_memory_gates = _sig("vb_memory_gates", _vp, _i64, _vp, _i, _vp, _vp, _f, _vp, _vp, _i64, _i64, _vp, _vp, _vp, _i64, _i, _i, _i, _i, _vp)
_gdn_scan = _sig("vb_gdn_scan", _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i64, _i64, _vp, _vp, _vp, _i64, _i, _i, _i, _i, _vp)


def _state_view(cache: torch.Tensor) -> torch.Tensor:
    """The recurrent-state pool as [rows, floats] fp32 (one row per request)."""
    c = cache.view(cache.shape[0], -1)
    return c if c.dtype == torch.float32 else c.view(torch.float32)


def causal_conv1d(x, weight, bias, cache, md, act: bool = True) -> torch.Tensor:
    """Depthwise causal conv over each request's tokens with the (k-1)-window kept at the head of its state row.
    x [T, C] (any dtype and row stride) → fp32 [T, C]; the window in the cache is advanced in place."""
    T, C = x.shape
    st = _state_view(cache)
    out = torch.empty((T, C), dtype=torch.float32, device=x.device)
    bt = md.block_table
    assert x.stride(1) == 1 and weight.is_contiguous() and weight.dtype == x.dtype
    _check(_conv1d(x.data_ptr(), x.stride(0), out.data_ptr(), out.stride(0), weight.data_ptr(), _p(bias), st.data_ptr(),
                   st.stride(0), md.query_start_loc.data_ptr(), md.seq_lens.data_ptr(), bt.data_ptr(), bt.stride(0),
                   md.num_reqs, T, C, weight.shape[-1], int(act), _DT[x.dtype], _st()), "causal_conv1d")
    return out


def selective_scan(x, dt, B, C, A, D, cache, state_off: int, md) -> torch.Tensor:
    """Mamba-1: fp32 x/dt [T, di], B/C [T, N], A [di, N], D [di] → y [T, di]; state rows updated in place."""
    T, di = x.shape
    N = B.shape[-1]
    st = _state_view(cache)
    y = torch.zeros((T, di), dtype=torch.float32, device=x.device)
    bt = md.block_table
    args = [t.contiguous() for t in (x, dt, B, C, A, D)]
    _check(_sel_scan(*[t.data_ptr() for t in args], y.data_ptr(), st.data_ptr(), st.stride(0), state_off,
                     md.query_start_loc.data_ptr(), md.seq_lens.data_ptr(), bt.data_ptr(), bt.stride(0), md.num_reqs, di, N,
                     _st()), "selective_scan")
    return y


def _scan_out(T: int, n: int, md, device) -> torch.Tensor:
    """Output rows of a scan; rows of no request (bucket padding) must be finite."""
    return (torch.zeros if md.flat else torch.empty)((T, n), dtype=torch.float32, device=device)


def ssd_scan(xbc, dt_raw, dt_bias, A_log, D, cache, state_off: int, md, nh: int, hd: int, G: int, N: int,
             dt_min: float = 0.0, dt_max: float = float("inf")) -> torch.Tensor:
    """Mamba-2: conv output xbc fp32 [T, nh*hd + 2*G*N], raw dt [T, nh] (any dtype and row stride) → y [T, nh*hd] fp32 (D skip
    included); the states at ``state_off`` of the request's slot (``ops.scan_state_elems``) advance in place."""
    T = xbc.shape[0]
    st = _state_view(cache)
    y = _scan_out(T, nh * hd, md, xbc.device)
    bt = md.block_table
    dt_max = min(dt_max, 3.0e38)
    assert xbc.dtype == torch.float32 and xbc.stride(1) == 1 and dt_raw.stride(1) == 1
    _check(_ssd_scan(xbc.data_ptr(), xbc.stride(0), dt_raw.data_ptr(), dt_raw.stride(0), dt_bias.data_ptr(),
                     A_log.data_ptr(), D.data_ptr(), y.data_ptr(), st.data_ptr(), st.stride(0), state_off,
                     md.query_start_loc.data_ptr(), md.seq_lens.data_ptr(), bt.data_ptr(), bt.stride(0), md.num_reqs,
                     md.max_query_len, nh, hd, G, N, dt_min, dt_max, _DT[dt_raw.dtype], _st()), "ssd_scan")
    return y


def gla_scan(q, k, v, a1, a2, a2_bias, tau: float, q_scale: float, cache, md, H: int, R: int, C: int, state_off: int = 0):
    """Gated linear attention: q, k [T, H*R], v [T, H*C] (row strides free), decay sigmoid(a1 @ a2.T + a2_bias)^(1/tau) per key
    channel → o [T, H*C] fp32; the slot's states advance in place."""
    T = q.shape[0]
    st = _state_view(cache)
    o = _scan_out(T, H * C, md, q.device)
    bt = md.block_table
    rank = a1.shape[1]
    assert all(t.stride(1) == 1 and t.dtype == q.dtype for t in (q, k, v, a1)) and a2.is_contiguous() and a2.dtype == q.dtype
    alpha = None
    if not md.decode_only:          # whole prompts: once per token and channel; decode steps evaluate it in the scan
        alpha = torch.empty((T, H * R), dtype=torch.float32, device=q.device)
        _check(_gla_decay(a1.data_ptr(), a1.stride(0), a2.data_ptr(), a2_bias.data_ptr(), alpha.data_ptr(), T, H * R, rank,
                          1.0 / tau, _DT[q.dtype], _st()), "gla_decay")
    _check(_gla_scan(q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0), k.stride(0), v.stride(0), q_scale, _p(alpha),
                     a1.data_ptr(), a1.stride(0), a2.data_ptr(), a2_bias.data_ptr(), rank, 1.0 / tau, o.data_ptr(), st.data_ptr(),
                     st.stride(0), state_off, md.query_start_loc.data_ptr(), md.seq_lens.data_ptr(), bt.data_ptr(), bt.stride(0),
                     md.num_reqs, md.max_query_len, H, R, C, _DT[q.dtype], _st()), "gla_scan")
    return o


def memory_gates(h, w, bias, cap: float, cache, m_off: int, md):
    """Gates of a matrix memory: h [T, W] (row stride free), w [2 heads, W] (input gates, forget gates), bias fp32 → [T, heads, 4] fp32
    (decay, input factor, exp(-m), -); the slots' running maxima at ``m_off`` advance in place.  32-bit throughout."""
    T, H = h.shape[0], w.shape[0] // 2
    st = _state_view(cache)
    bt = md.block_table
    assert h.stride(1) == 1 and w.is_contiguous() and w.dtype == h.dtype and bias.dtype == torch.float32
    gates = _scan_out(T, H * 4, md, h.device)
    logits = None
    if not md.decode_only:
        logits = torch.mm(h, w.t(), out_dtype=torch.float32) if h.dtype != torch.float32 else h @ w.t()
    _check(_memory_gates(h.data_ptr(), h.stride(0), w.data_ptr(), h.shape[1], _p(logits), bias.data_ptr(), cap, gates.data_ptr(),
                         st.data_ptr(), st.stride(0), m_off, md.query_start_loc.data_ptr(), md.seq_lens.data_ptr(), bt.data_ptr(),
                         bt.stride(0), md.num_reqs, md.max_query_len, H, _DT[h.dtype], _st()), "memory_gates")
    return gates.view(T, H, 4)


def memory_scan(q, k, v, gates, q_scale: float, cache, md, H: int, R: int, C: int, state_off: int = 0):
    """Matrix memory: q, k [T, H*R], v [T, H*C] (row strides free) → [T, H, C rounded up to four + 4] fp32, n . q in the last quad's
    first column; the slots' states advance in place."""
    T = q.shape[0]
    st = _state_view(cache)
    cols = -(-C // 4) * 4 + 4
    o = _scan_out(T, H * cols, md, q.device)
    bt = md.block_table
    assert all(t.stride(1) == 1 and t.dtype == q.dtype for t in (q, k, v)) and gates.is_contiguous()
    _check(_memory_scan(q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0), k.stride(0), v.stride(0), q_scale, gates.data_ptr(),
                        o.data_ptr(), st.data_ptr(), st.stride(0), state_off, md.query_start_loc.data_ptr(), md.seq_lens.data_ptr(),
                        bt.data_ptr(), bt.stride(0), md.num_reqs, md.max_query_len, H, R, C, _DT[q.dtype], _st()), "memory_scan")
    return o.view(T, H, cols)


def gated_norm(y, z, weight, groups: int, eps: float, gate_first: bool, out=None, scale: float = 1.0, gate: str = "silu", gates=None):
    """y fp32 [T, n]: RMS norm over ``groups`` equal parts, silu(z) (``gate`` "sigmoid": sigmoid(z)) before (``gate_first``) or behind it,
    times the weight (repeated along the parts where it is shorter) and ``scale``; in z's dtype.  ``gates``: y is the result of
    ``memory_scan`` with these gates, divided by its normaliser first."""
    T, n = z.shape
    if out is None:
        out = torch.empty((T, n), dtype=z.dtype, device=z.device)
    W = n // groups
    wl = weight.numel()
    assert y.is_contiguous() and z.stride(1) == 1 and out.stride(1) == 1 and weight.dtype == z.dtype and n % groups == 0 and n % wl == 0
    assert y.numel() == T * groups * (W if gates is None else -(-W // 4) * 4 + 4)
    _check(_gated_norm(y.data_ptr(), _p(gates), z.data_ptr(), z.stride(0), weight.data_ptr(), wl, out.data_ptr(), out.stride(0), T, groups,
                       W, int(gate_first) | 2 * int(gate == "sigmoid"), eps, scale, _DT[z.dtype], _st()), "gated_norm")
    return out


def gdn_scan(q, k, v, g, beta, cache, state_off: int, md) -> torch.Tensor:
    """Gated delta rule: fp32 q/k [T, nv, dk], v [T, nv, dv], g/beta [T, nv] → o [T, nv, dv]; state [nv, dk, dv]."""
    T, nv, dk = q.shape
    dv = v.shape[-1]
    st = _state_view(cache)
    o = torch.zeros((T, nv, dv), dtype=torch.float32, device=q.device)
    bt = md.block_table
    a = [t.contiguous() for t in (q, k, v, g, beta)]
    _check(_gdn_scan(*[t.data_ptr() for t in a], o.data_ptr(), st.data_ptr(), st.stride(0), state_off,
                     md.query_start_loc.data_ptr(), md.seq_lens.data_ptr(), bt.data_ptr(), bt.stride(0), md.num_reqs, nv, dk,
                     dv, _st()), "gdn_scan")
    return o


# ------------------------------------------------------------------ GPU-side input preparation (csrc/input_prep.cu)
_prep_step = _sig("vb_prep_step3", _vp, _vp, _vp, _i, _i, _i, _vp, _i64, _vp, _i64, _vp, _vp, _vp, _vp, _vp, _vp, _i64, _i, _i, _vp,
                  _i, _vp)
_bt_diff = _sig("vb_block_table_diff", _vp, _i64, _vp, _vp, _vp, _vp, _vp, _i, _vp)
_append_sampled = _sig("vb_append_sampled", _vp, _i64, _vp, _vp, _vp, _i, _vp)


def prep_step(rows, num_computed, num_sched, token_table, block_rows, input_ids, positions, qsl, seq_lens, slot_mapping,
              block_table, nblk: int, block_size: int, pos_delta=None, pad_b: int = 0, write_tokens: bool = True,
              pad_t: int = 0) -> None:
    """Expand per-request (row, computed, scheduled) triples into the per-token step inputs on the device.  Entries
    [nb, pad_b) are CUDA-graph bucket padding: one-token requests on the null block (decode buckets, ``pad_t`` = 0) or
    empty requests plus padding tokens up to ``pad_t`` (mixed-batch buckets)."""
    nb = rows.numel()
    _check(_prep_step(rows.data_ptr(), num_computed.data_ptr(), num_sched.data_ptr(), nb, max(pad_b, nb), pad_t,
                      token_table.data_ptr(), token_table.stride(0), block_rows.data_ptr(), block_rows.stride(0),
                      input_ids.data_ptr(), positions.data_ptr(), qsl.data_ptr(), seq_lens.data_ptr(),
                      slot_mapping.data_ptr(), block_table.data_ptr(), block_table.stride(0), nblk, block_size,
                      _p(pos_delta), int(write_tokens), _st()), "prep_step")


def block_table_apply_diffs(block_rows, d_row, d_start, d_cnt, d_off, ids_flat) -> None:
    _check(_bt_diff(block_rows.data_ptr(), block_rows.stride(0), d_row.data_ptr(), d_start.data_ptr(), d_cnt.data_ptr(),
                    d_off.data_ptr(), ids_flat.data_ptr(), d_row.numel(), _st()), "block_table_diff")


def append_sampled(token_table, rows, pos, sampled) -> None:
    _check(_append_sampled(token_table.data_ptr(), token_table.stride(0), rows.data_ptr(), pos.data_ptr(),
                           sampled.data_ptr(), rows.numel(), _st()), "append_sampled")


# ------------------------------------------------------------------ weight-only FP4 decode GEMM (csrc/gemm_w4.cu)
_gemm_w4 = _sig("vb_gemm_w4", _vp, _vp, _vp, _vp, _i, _i, _i, _i64, _f, _i, _i, _vp)
W4_MAX_TOKENS = 128


def pack_w4_tiles(codes: torch.Tensor, scales: torch.Tensor, fmt: str) -> torch.Tensor:
    """Tile-major operand layout of the W4A16 kernel.  ``codes``: uint8 [N, K/2] (two e2m1 codes per byte, low nibble
    first); ``scales``: one byte per 16 (``nvfp4``: e4m3) or 32 (``mxfp4``: e8m0) columns, [N, K/16] or [N, K/32].
    Returns uint8 [ceil(N/128), K/64, 4096 + 128 * {4, 2}]: every (128-row tile, 64-column block) is one contiguous
    record = the codes of its 128 rows followed by their scales."""
    N, K2 = codes.shape
    K = K2 * 2
    assert K % 64 == 0, "W4 kernel: K must be a multiple of 64"
    spb = 4 if fmt == "nvfp4" else 2                 # scale bytes per row per 64-column block
    sc = scales.view(torch.uint8) if scales.dtype != torch.uint8 else scales
    assert sc.shape == (N, K // 64 * spb), (sc.shape, N, K)
    Np = (N + 127) // 128 * 128
    if Np != N:
        codes = torch.nn.functional.pad(codes, (0, 0, 0, Np - N))
        sc = torch.nn.functional.pad(sc, (0, 0, 0, Np - N))
    c = codes.view(Np // 128, 128, K // 64, 32).permute(0, 2, 1, 3).reshape(Np // 128, K // 64, 4096)
    s = sc.reshape(Np // 128, 128, K // 64, spb).permute(0, 2, 1, 3).reshape(Np // 128, K // 64, 128 * spb)
    return torch.cat([c, s], dim=-1).contiguous()


def gemm_w4(x: torch.Tensor, tiled: torch.Tensor, N: int, gscale: float, fmt: str, bias: Optional[torch.Tensor] = None
            ) -> torch.Tensor:
    """Y = X · dequant(W)^T for FP4 weights in the tile-major layout of ``pack_w4_tiles`` (M <= 128 tokens)."""
    M, K = x.shape
    y = torch.empty((M, N), dtype=x.dtype, device=x.device)
    _check(_gemm_w4(x.data_ptr(), tiled.data_ptr(), _p(bias), y.data_ptr(), M, N, K, x.stride(0), float(gscale),
                    0 if fmt == "nvfp4" else 1, _DT[x.dtype], _st()), f"gemm_w4(M={M},N={N},K={K},{fmt})")
    return y


def gemm_w4_ok(x: torch.Tensor, K: int) -> bool:
    return (x.is_cuda and x.dtype in (torch.bfloat16, torch.float16) and x.dim() == 2 and 0 < x.shape[0] <= W4_MAX_TOKENS
            and K % 64 == 0 and x.stride(1) == 1 and (x.stride(0) * 2) % 16 == 0)


# ------------------------------------------------------------------ L2 weight prefetch on a side stream
_l2_prefetch = _sig("vb_l2_prefetch", _vp, _i64, _vp)
_side_streams: dict[int, torch.cuda.Stream] = {}
_side_dirty: dict[int, bool] = {}


def l2_prefetch_async(t: torch.Tensor) -> None:
    """Start pulling ``t`` into L2 on a forked stream, ordered after everything enqueued so far on the current stream
    (so it runs concurrently with the NEXT kernel launched here).  A hint only: nothing ever waits for it except
    ``l2_prefetch_join`` at the end of the forward pass (required to close a CUDA-graph capture)."""
    dev = t.device.index or 0
    side = _side_streams.get(dev)
    if side is None:
        if torch.cuda.is_current_stream_capturing():
            return
        side = _side_streams[dev] = torch.cuda.Stream(t.device)
    cur = torch.cuda.current_stream()
    side.wait_stream(cur)
    with torch.cuda.stream(side):
        _check(_l2_prefetch(t.data_ptr(), t.numel() * t.element_size(), side.cuda_stream), "l2_prefetch", 0)
    _side_dirty[dev] = True


def l2_prefetch_join() -> None:
    dev = torch.cuda.current_device()
    if _side_dirty.get(dev):
        torch.cuda.current_stream().wait_stream(_side_streams[dev])
        _side_dirty[dev] = False
