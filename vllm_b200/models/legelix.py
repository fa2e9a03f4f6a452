"""Legelix: chunk-local attention beside a state-space mixer, and gated linear attention, in sandwich-norm residual blocks.

    x_{n+1} = x_n + m N'(F_n(N(x_n)))     F_n: mixer and feed-forward in turn; layer norms N in front of it and N' behind it
    logits = W_head N(x_last)

* The stream x stays in fp32; one kernel per boundary (``ops.norm_add``) does N', the residual sum and the next N.
* ``gla`` layers: ``layers/gla.py``.
* ``parallel`` layers: ``a * attention(h) + b * mamba2(h)``.  Both read the same h, so their input projections are one GEMM,
  and so are their output projections: the factors a and b go into the mixers' outputs, which lie side by side.

Sizes and constants come from the configuration layer by layer: layers may differ in everything, and a layer may have no
feed-forward.  Under tensor parallelism the mixers are replicated (as the framework's other state-space mixers are); the
feed-forward and the head are sharded.
"""
from __future__ import annotations

from typing import Iterable, Optional

import torch
import torch.nn as nn

from vllm_b200 import ops
from vllm_b200.config import VllmConfig
from vllm_b200.layers.attention import Attention
from vllm_b200.layers.common import LayerNorm, RMSNorm, VocabParallelEmbedding
from vllm_b200.layers.gla import GatedLinearAttention
from vllm_b200.layers.linear import MergedReplicatedLinear, SummedReplicatedLinear
from vllm_b200.layers.mamba import Mamba2Mixer
from vllm_b200.layers.rotary import get_rope
from vllm_b200.models.llama import LlamaForCausalLM, LlamaMLP
from vllm_b200.parallel.state import get_pp_group
from vllm_b200.parallel.utils import get_pp_indices


class AttentionBesideMamba(nn.Module):
    def __init__(self, hidden: int, m: dict, eps: float, max_position: int, dtype, prefix: str) -> None:
        super().__init__()
        a, s = m["left"], m["right"]
        H, G, d, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
        inner, bc = s["heads"] * s["vdim"], 2 * s["groups"] * s["state"]
        # q | k | v (biased) and z | x B C | dt
        self.in_proj = MergedReplicatedLinear(hidden, [H * d, G * d, G * dv, inner, inner + bc, s["heads"]], True, dtype, None,
                                              f"{prefix}.in_proj", align=8)
        self.q_norm, self.k_norm = RMSNorm(d, eps, dtype), RMSNorm(d, eps, dtype)
        self.sinks = nn.Parameter(torch.zeros(H, dtype=torch.float32), requires_grad=False)
        rot, sc = a["rot"], a["rot"].get("scaling")
        rope = get_rope(d, rot["dims"], max_position, float(rot["base"]), False, sc and dict(
            rope_type="llama3", factor=sc["factor"], low_freq_factor=sc["low"], high_freq_factor=sc["high"],
            original_max_position_embeddings=sc["original"]))
        self.attn = Attention(H, d, a["scale"], G, prefix=f"{prefix}.attn", rope=rope, sinks=self.sinks,
                              chunk_size=a["mask"]["size"], v_head_size=dv, fused_prologue=True, out_scale=m["left_scale"])
        self.mamba = Mamba2Mixer(hidden, s["heads"], s["vdim"], s["state"], s["conv"], s["groups"], False, True, 128, eps, dtype,
                                 f"{prefix}.mamba", norm_groups=s["norm_groups"], own_projections=False)
        self.left_scale, self.right_scale = float(m["left_scale"]), float(m["right_scale"])
        self.out_proj = SummedReplicatedLinear([H * dv, inner], hidden, dtype, f"{prefix}.out_proj")
        self.out_bias = nn.Parameter(torch.zeros(hidden, dtype=torch.float32), requires_grad=False)     # times left_scale

    def forward(self, positions: torch.Tensor, h: torch.Tensor) -> torch.Tensor:
        """Without ``out_bias``."""
        q, k, v, z, xbc, dt = self.in_proj.parts(self.in_proj(h))
        x, (left, right) = self.out_proj.buffer(h)
        self.attn(q, k, v, positions, qk_norm=(self.q_norm, self.k_norm), out=left)
        self.mamba.mix(z, xbc, dt, out=right, scale=self.right_scale)
        return self.out_proj(x)


class LegelixLayer(nn.Module):
    def __init__(self, cfg: dict, max_position: int, dtype, quant_config, prefix: str, idx: int) -> None:
        super().__init__()
        spec = cfg["layers"][idx]
        H, eps = cfg["hidden_size"], cfg["norm"]["eps"]
        self.kind, self.mult = spec["type"], float(cfg["residual_mult"])
        m = spec["mixer"]
        if self.kind == "gla":
            self.mixer = GatedLinearAttention(H, m["heads"], m["dim"], m["vdim"], m["rank"], m["tau"], eps, dtype, f"{prefix}.mixer")
        elif self.kind == "parallel":
            self.mixer = AttentionBesideMamba(H, m, eps, max_position, dtype, f"{prefix}.mixer")
        else:
            raise ValueError(f"{prefix}: unknown mixer {self.kind!r}")
        self.norm1, self.norm1b = LayerNorm(H, eps, dtype=dtype), LayerNorm(H, eps, dtype=dtype)
        self.mlp = None
        if spec.get("mlp") is not None:
            if spec["mlp"].get("kind") != "dense":
                raise ValueError(f"{prefix}: unknown feed-forward kind {spec['mlp'].get('kind')!r}")
            self.mlp = LlamaMLP(H, spec["mlp"]["ff"], "silu", False, dtype, quant_config, f"{prefix}.mlp")
            self.norm2, self.norm2b = LayerNorm(H, eps, dtype=dtype), LayerNorm(H, eps, dtype=dtype)

    def forward(self, positions: torch.Tensor, stream: torch.Tensor, h: torch.Tensor, next_norm: Optional[LayerNorm]) -> torch.Tensor:
        """``h``: norm1 of the stream (fp32, updated in place).  Returns ``next_norm`` of it, or its copy in the model dtype."""
        bias = None
        if self.kind == "gla":
            y = self.mixer(h)
        else:
            y, bias = self.mixer(positions, h), self.mixer.out_bias
        h = _step(stream, y, bias, self.norm1b, self.mult, next_norm if self.mlp is None else self.norm2)
        if self.mlp is None:
            return h
        return _step(stream, self.mlp(h), None, self.norm2b, self.mult, next_norm)


def _step(stream, y, y_bias, norm: LayerNorm, mult: float, next_norm: Optional[LayerNorm]) -> torch.Tensor:
    return ops.norm_add(stream, y, y_bias, (norm.weight, norm.bias), mult,
                        None if next_norm is None else (next_norm.weight, next_norm.bias), norm.eps)


class LegelixModel(nn.Module):
    def __init__(self, vllm_config: VllmConfig, prefix: str = "model", quant_config=None) -> None:
        super().__init__()
        mc = vllm_config.model_config
        self.cfg = cfg = mc.hf_config
        dtype = mc.torch_dtype
        pp = get_pp_group()
        self.pp_rank, self.pp_size = max(pp.rank_in_group, 0), pp.world_size
        self.start, self.end = get_pp_indices(cfg["num_hidden_layers"], self.pp_rank, self.pp_size)
        H, eps = cfg["hidden_size"], cfg["norm"]["eps"]
        self.embed_tokens = None
        if self.pp_rank == 0:
            self.embed_tokens = VocabParallelEmbedding(cfg["vocab_size"], H, dtype, prefix=f"{prefix}.embed_tokens", replicate=True)
        self.layers = nn.ModuleList([LegelixLayer(cfg, mc.max_model_len, dtype, quant_config, f"{prefix}.layers.{i}", i)
                                     for i in range(self.start, self.end)])
        self.norm = LayerNorm(H, eps, dtype=dtype) if self.pp_rank == self.pp_size - 1 else None

    def embed_input_ids(self, input_ids: torch.Tensor) -> torch.Tensor:
        return self.embed_tokens(input_ids)

    def forward(self, input_ids, positions, intermediate_tensors=None, inputs_embeds=None):
        norms = [layer.norm1 for layer in self.layers] + [self.norm]
        first = norms[0]
        if self.pp_rank > 0:
            stream, h = intermediate_tensors["residual"].contiguous(), ops.layer_norm(
                intermediate_tensors["residual"], first.weight.float(), first.bias.float(), first.eps).to(first.weight.dtype)
        elif inputs_embeds is not None:
            stream = inputs_embeds.float()
            h = ops.layer_norm(stream, first.weight.float(), first.bias.float(), first.eps).to(inputs_embeds.dtype)
        else:
            stream, h = ops.embed_norm(input_ids, self.embed_tokens.weight, (first.weight, first.bias), first.eps)
        for layer, nxt in zip(self.layers, norms[1:]):
            h = layer(positions, stream, h, nxt)
        if self.norm is None:
            return {"hidden_states": h, "residual": stream}
        return h


class LegelixForCausalLM(LlamaForCausalLM):
    model_cls = LegelixModel

    @staticmethod
    def kernel_sources(cfg: dict, dtype: torch.dtype) -> list[str]:
        """CUDA sources of this model's steps (ops/cuda.py ``prebuild``)."""
        out = {"stream", "linear_attn", "norm_act", "input_prep"}
        half = dtype != torch.float32
        if half:
            out.add("gemm_tc")
        for spec in cfg["layers"]:
            if spec["type"] != "parallel":
                continue
            a = spec["mixer"]["left"]
            out |= {"ssm", "qknorm_rope"}
            cu, d, dv, group = ops.cuda_ops(), a["dim"], a["vdim"], a["heads"] // a["kv_heads"]
            if half and cu.tc_attention_ok(d, dv, group):
                out |= {"attention_tc", "attention_tc_decode"}
            elif spec["mixer"]["left_scale"] == 1.0 and cu._simt_attention_ok(d, dv, 64, group, dtype):
                out.add("attention_simt")
            else:
                out.add("attention_any")
        return sorted(out)

    # checkpoint tensor (behind "l<i>.") → (parameter, shard)
    _layer_tensors = {
        **{n + s: (n + p, None) for n in ("norm1", "norm1b", "norm2", "norm2b") for s, p in (("", ".weight"), (".b", ".bias"))},
        "mlp.gate": ("mlp.gate_up_proj.weight", 0), "mlp.up": ("mlp.gate_up_proj.weight", 1), "mlp.down": ("mlp.down_proj.weight", None)}
    _gla_tensors = {"mix.q": ("mixer.in_proj.weight", 0), "mix.k": ("mixer.in_proj.weight", 1), "mix.v": ("mixer.in_proj.weight", 2),
                    "mix.g": ("mixer.in_proj.weight", 3), "mix.a1": ("mixer.in_proj.weight", 4), "mix.a2": ("mixer.a2", None),
                    "mix.a2.b": ("mixer.a2_bias", None), "mix.norm": ("mixer.norm_weight", None), "mix.o": ("mixer.out_proj.weight", None)}
    _parallel_tensors = {
        **{f"mix.left.{n}{s}": (f"mixer.in_proj.{p}", i) for i, n in enumerate("qkv") for s, p in (("", "weight"), (".b", "bias"))},
        "mix.left.q.norm": ("mixer.q_norm.weight", None), "mix.left.k.norm": ("mixer.k_norm.weight", None),
        "mix.left.sink": ("mixer.sinks", None), "mix.left.o": ("mixer.out_proj.weight", 0), "mix.left.o.b": ("mixer.out_bias", None),
        "mix.right.conv": ("mixer.mamba.conv_weight", None), "mix.right.conv.b": ("mixer.mamba.conv_bias", None),
        "mix.right.dt_bias": ("mixer.mamba.dt_bias", None), "mix.right.A_log": ("mixer.mamba.A_log", None),
        "mix.right.D": ("mixer.mamba.D", None), "mix.right.norm": ("mixer.mamba.norm_weight", None),
        "mix.right.o": ("mixer.out_proj.weight", 1)}
    _model_tensors = {"embed": "model.embed_tokens.weight", "final.norm": "model.norm.weight", "final.norm.b": "model.norm.bias",
                      "head": "lm_head.weight"}

    def _place(self, name: str, w: torch.Tensor) -> list[tuple[str, Optional[int], torch.Tensor]]:
        """(parameter, shard, values) of a checkpoint tensor; empty: it belongs to another pipeline stage."""
        if name in self._model_tensors:
            target = self._model_tensors[name]
            here = self.model.embed_tokens is not None if name == "embed" else self.is_last
            return [(target, None, w)] if here else []
        idx, _, rest = name[1:].partition(".")
        if name[:1] == "l" and idx.isdigit() and int(idx) < len(self.cfg["layers"]):
            i = int(idx)
            if not self.model.start <= i < self.model.end:
                return []
            head = f"model.layers.{i - self.model.start}."
            layer = self.model.layers[i - self.model.start]
            if layer.kind == "parallel" and rest == "mix.right.in":          # z | x B C | dt
                sizes = layer.mixer.in_proj.output_sizes[3:]
                return [(head + "mixer.in_proj.weight", 3 + j, part) for j, part in enumerate(w.split(sizes, dim=0))]
            place = (self._gla_tensors if layer.kind == "gla" else self._parallel_tensors).get(rest) or self._layer_tensors.get(rest)
            if place is not None:
                if rest == "mix.left.o.b":
                    w = w.float() * layer.mixer.left_scale
                return [(head + place[0], place[1], w)]
        raise ValueError(f"unexpected tensor {name!r} in a Legelix checkpoint")

    def load_weights(self, weights: Iterable[tuple[str, torch.Tensor]]) -> set[str]:
        params, modules = dict(self.named_parameters()), dict(self.named_modules())
        loaded: set[str] = set()
        for name, w in weights:
            for target, shard, values in self._place(name, w):
                if target not in params:
                    raise ValueError(f"tensor {name!r} has no place in this configuration")
                p, mod = params[target], modules[target.rsplit(".", 1)[0]]
                loader = getattr(mod, "weight_loader", None)
                if loader is not None:
                    loader(p, values, shard)
                else:
                    assert p.shape == values.shape, (name, p.shape, values.shape)
                    p.data.copy_(values)
                loaded.add(target)
        return loaded
