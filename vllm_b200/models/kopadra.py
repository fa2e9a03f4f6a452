"""Kopadra: gated full attention beside xLSTM matrix memories, with dense and mixture-of-experts feed-forwards, in pre-norm blocks.

    x_{n+1} = x_n + F_n(N(x_n))           F_n: mixer and feed-forward in turn; N a layer norm without a bias
    logits = c tanh(E N(x_last) / c)      E the embedding table

* The stream x stays in fp32; one kernel per boundary (``ops.add_norm``) adds F_n's output, or combines the experts', and takes the
  next N.
* ``attention`` layers: RMS norms over the whole q and k projections, rotation of a part of each head with YaRN frequencies, an
  output gate; a layer with ``kv_from`` reads the keys and values of that earlier layer.
* ``mlstm`` layers: ``layers/mlstm.py``.
* Experts: a softmax router with a selection bias and group-limited choice, in 32-bit (``GroupedRouter``); some of the router's
  outputs are identity experts; a shared expert runs for every token.

Sizes and constants come from the configuration layer by layer: layers may differ in everything, and a layer may have no
feed-forward.  Under tensor parallelism the mixers are replicated (norms over whole projections need whole rows, and the
framework's other recurrent mixers are replicated too); feed-forwards and the head are sharded.
"""
from __future__ import annotations

import math
from typing import Iterable, Optional

import torch
import torch.nn as nn

from vllm_b200 import ops
from vllm_b200.config import VllmConfig
from vllm_b200.layers.attention import Attention
from vllm_b200.layers.common import LayerNorm, RMSNorm, VocabParallelEmbedding
from vllm_b200.layers.linear import MergedReplicatedLinear, ReplicatedLinear
from vllm_b200.layers.mlstm import MatrixMemory
from vllm_b200.layers.moe import FusedMoE, GroupedRouter
from vllm_b200.layers.rotary import get_rope
from vllm_b200.models.llama import LlamaForCausalLM, LlamaMLP
from vllm_b200.parallel.state import get_pp_group
from vllm_b200.parallel.utils import get_pp_indices


class GatedAttention(nn.Module):
    def __init__(self, hidden: int, m: dict, eps: float, max_position: int, dtype, prefix: str, kv_from: Optional[str]) -> None:
        super().__init__()
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        self.shares = kv_from is not None
        # q | k | v (biased) and the gate; a layer with another's keys has q and the gate
        sizes = [H * d, H * dv] if self.shares else [H * d, G * d, G * dv, H * dv]
        self.in_proj = MergedReplicatedLinear(hidden, sizes, True, dtype, None, f"{prefix}.in_proj", align=8)
        self.q_norm = RMSNorm(H * d, eps, dtype)
        self.k_norm = None if self.shares else RMSNorm(G * d, eps, dtype)
        rot = m.get("rot") or dict(base=10000.0, dims=0)
        sc = rot.get("scaling")
        rope = get_rope(d, rot["dims"], max_position, float(rot["base"]), True, dict(
            exact=True, **({} if not sc else dict(
                rope_type="yarn", factor=sc["factor"], original_max_position_embeddings=sc["original"], beta_fast=sc["fast"],
                beta_slow=sc["slow"], attn_factor=min(0.0, 0.1 * math.log(sc["factor"])) + 1, ordered_ramp=True, fixed_length=True))))
        self.attn = Attention(H, d, m["scale"], G, prefix=f"{prefix}.attn", rope=rope, v_head_size=dv, fused_prologue=True,
                              whole_qk_norm=True, kv_sharing_target=kv_from)
        self.out_proj = ReplicatedLinear(H * dv, hidden, False, dtype, None, f"{prefix}.out_proj")

    def forward(self, positions: torch.Tensor, h: torch.Tensor) -> torch.Tensor:
        parts = self.in_proj.parts(self.in_proj(h))
        q, k, v, g = (parts[0], None, None, parts[1]) if self.shares else parts
        return self.out_proj(self.attn(q, k, v, positions, qk_norm=(self.q_norm, self.k_norm), gate=g))


class KopadraExperts(nn.Module):
    def __init__(self, spec: dict, hidden: int, dtype, quant_config, prefix: str, enable_ep: bool) -> None:
        super().__init__()
        r, groups = spec["router"], spec["router"].get("groups") or {"count": 1, "keep": 1}
        identity = int(r.get("identity") or 0)
        self.router = GroupedRouter(hidden, r["experts"] + identity, r["top"], dtype, groups["count"], groups["keep"],
                                    scoring_func="softmax", renormalize=True, routed_scaling_factor=float(r["scale"]), group_score="max")
        self.experts = FusedMoE(r["experts"], r["top"], hidden, spec["expert"]["ff"], dtype, act="silu", enable_ep=enable_ep,
                                prefix=f"{prefix}.experts", quant_config=quant_config, identity_experts=identity)
        self.shared = None
        if spec.get("shared"):
            self.shared = LlamaMLP(hidden, spec["shared"]["ff"], "silu", False, dtype, quant_config, f"{prefix}.shared")

    def forward_add_norm(self, h: torch.Tensor, stream: torch.Tensor, next_norm: Optional[LayerNorm]) -> torch.Tensor:
        return self.experts.forward_add_norm(h, self.router(h), stream, None if self.shared is None else self.shared(h), next_norm)


class KopadraLayer(nn.Module):
    def __init__(self, cfg: dict, max_position: int, dtype, quant_config, layers_prefix: str, idx: int, enable_ep: bool) -> None:
        super().__init__()
        spec, prefix = cfg["layers"][idx], f"{layers_prefix}.{idx}"
        H, eps = cfg["hidden_size"], cfg["norm"]["eps"]
        self.kind, m = spec["type"], spec["mixer"]
        if self.kind == "mlstm":
            self.mixer = MatrixMemory(H, m["heads"], m["dim"], m["vdim"], m["gate_cap"], eps, dtype, f"{prefix}.mixer")
        elif self.kind == "attention":
            j = m.get("kv_from")
            self.mixer = GatedAttention(H, m, eps, max_position, dtype, f"{prefix}.mixer",
                                        None if j is None else f"{layers_prefix}.{j}.mixer.attn")
        else:
            raise ValueError(f"{prefix}: unknown mixer {self.kind!r}")
        self.norm1 = LayerNorm(H, eps, False, dtype)
        self.mlp, self.mlp_kind = None, None
        if spec.get("mlp") is not None:
            self.mlp_kind = spec["mlp"]["kind"]
            if self.mlp_kind == "dense":
                self.mlp = LlamaMLP(H, spec["mlp"]["ff"], "gelu_pytorch_tanh", False, dtype, quant_config, f"{prefix}.mlp")
            elif self.mlp_kind == "moe":
                self.mlp = KopadraExperts(spec["mlp"], H, dtype, quant_config, f"{prefix}.mlp", enable_ep)
            else:
                raise ValueError(f"{prefix}: unknown feed-forward kind {self.mlp_kind!r}")
            self.norm2 = LayerNorm(H, eps, False, dtype)

    def forward(self, positions: torch.Tensor, stream: torch.Tensor, h: torch.Tensor, next_norm: Optional[LayerNorm]) -> torch.Tensor:
        """``h``: norm1 of the stream (fp32, updated in place).  Returns ``next_norm`` of it, or its copy in the model dtype."""
        y = self.mixer(h) if self.kind == "mlstm" else self.mixer(positions, h)
        h = _step(stream, y, next_norm if self.mlp is None else self.norm2)
        if self.mlp is None:
            return h
        if self.mlp_kind == "dense":
            return _step(stream, self.mlp(h), next_norm)
        return self.mlp.forward_add_norm(h, stream, next_norm)


def _step(stream: torch.Tensor, y: torch.Tensor, norm: Optional[LayerNorm]) -> torch.Tensor:
    return ops.add_norm(stream, y, None, 0.0) if norm is None else ops.add_norm(stream, y, (norm.weight, norm.bias), norm.eps)


class KopadraModel(nn.Module):
    def __init__(self, vllm_config: VllmConfig, prefix: str = "model", quant_config=None) -> None:
        super().__init__()
        mc = vllm_config.model_config
        self.cfg = cfg = mc.hf_config
        dtype = mc.torch_dtype
        pp = get_pp_group()
        self.pp_rank, self.pp_size = max(pp.rank_in_group, 0), pp.world_size
        self.start, self.end = get_pp_indices(cfg["num_hidden_layers"], self.pp_rank, self.pp_size)
        H, eps = cfg["hidden_size"], cfg["norm"]["eps"]
        ep = bool(vllm_config.parallel_config.enable_expert_parallel)
        self.embed_tokens = None
        if self.pp_rank == 0:
            self.embed_tokens = VocabParallelEmbedding(cfg["vocab_size"], H, dtype, prefix=f"{prefix}.embed_tokens", replicate=True)
        self.layers = nn.ModuleList([KopadraLayer(cfg, mc.max_model_len, dtype, quant_config, f"{prefix}.layers", i, ep)
                                     for i in range(self.start, self.end)])
        self.norm = LayerNorm(H, eps, False, dtype) if self.pp_rank == self.pp_size - 1 else None

    def embed_input_ids(self, input_ids: torch.Tensor) -> torch.Tensor:
        return self.embed_tokens(input_ids)

    def forward(self, input_ids, positions, intermediate_tensors=None, inputs_embeds=None):
        norms = [layer.norm1 for layer in self.layers] + [self.norm]
        first = norms[0]
        if self.pp_rank > 0:
            stream, h = intermediate_tensors["residual"].contiguous(), intermediate_tensors["hidden_states"]
            h = ops.layer_norm(stream, first.weight.float(), None, first.eps).to(h.dtype)
        elif inputs_embeds is not None:
            stream = inputs_embeds.float()
            h = ops.layer_norm(stream, first.weight.float(), None, first.eps).to(inputs_embeds.dtype)
        else:
            stream, h = ops.embed_norm(input_ids, self.embed_tokens.weight, (first.weight, None), first.eps)
        for layer, nxt in zip(self.layers, norms[1:]):
            h = layer(positions, stream, h, nxt)
        if self.norm is None:
            return {"hidden_states": h, "residual": stream}
        return h


class KopadraForCausalLM(LlamaForCausalLM):
    model_cls = KopadraModel

    def __init__(self, vllm_config: VllmConfig, prefix: str = "") -> None:
        if vllm_config.cache_config.cache_dtype.startswith("fp8"):
            raise ValueError("norms over whole projections write caches of the model dtype (kv_cache_dtype fp8 is not supported)")
        super().__init__(vllm_config, prefix)
        # the head is the embedding table: one tensor where a rank holds all of both
        self.tied = self.is_last and self.model.embed_tokens is not None and self.lm_head.tp_size == 1
        if self.tied:
            self.lm_head.tie_weights(self.model.embed_tokens)

    @staticmethod
    def kernel_sources(cfg: dict, dtype: torch.dtype) -> list[str]:
        """CUDA sources of this model's steps (ops/cuda.py ``prebuild``)."""
        out = {"stream", "norm_act", "input_prep"}
        half = dtype != torch.float32
        cu = ops.cuda_ops()
        attn = [l["mixer"] for l in cfg["layers"] if l["type"] == "attention"]
        # one cache layout for all attention layers: the tensor-core kernels run where they take every layer's head shape
        tensor_cores = half and all(cu.tc_attention_ok(a["dim"], a["vdim"], a["heads"] // a["kv_heads"]) for a in attn)
        for a in attn:
            out.add("qknorm_rope")
            if tensor_cores:
                out |= {"attention_tc", "attention_tc_decode"}
            elif half and cu._simt_attention_ok(a["dim"], a["vdim"], 64, a["heads"] // a["kv_heads"], dtype):
                out.add("attention_simt")
            else:
                out.add("attention_any")
        if any(l["type"] == "mlstm" for l in cfg["layers"]):
            out.add("linear_attn")
        if any(l.get("mlp") and l["mlp"]["kind"] == "moe" for l in cfg["layers"]):
            out.add("moe")
        if half:
            out.add("gemm_tc")
        return sorted(out)

    # checkpoint tensor (behind "l<i>.") → (parameter, shard)
    _layer_tensors = {"norm1": ("norm1.weight", None), "norm2": ("norm2.weight", None)}
    _dense_tensors = {"mlp.gate": ("mlp.gate_up_proj.weight", 0), "mlp.up": ("mlp.gate_up_proj.weight", 1),
                      "mlp.down": ("mlp.down_proj.weight", None)}
    _moe_tensors = {"mlp.router": ("mlp.router.weight", None), "mlp.correction": ("mlp.router.bias", None),
                    "mlp.shared.gate": ("mlp.shared.gate_up_proj.weight", 0), "mlp.shared.up": ("mlp.shared.gate_up_proj.weight", 1),
                    "mlp.shared.down": ("mlp.shared.down_proj.weight", None)}
    _expert_shards = {"gate": ("w13_weight", "w1"), "up": ("w13_weight", "w3"), "down": ("w2_weight", "w2")}
    _mlstm_tensors = {**{f"mix.{n}": ("mixer.in_proj.weight", i) for i, n in enumerate("qkvg")},
                      "mix.i": ("mixer.gate_proj.weight", 0), "mix.f": ("mixer.gate_proj.weight", 1), "mix.i.b": ("mixer.gate_bias", 0),
                      "mix.f.b": ("mixer.gate_bias", 1), "mix.norm": ("mixer.norm_weight", None), "mix.o": ("mixer.out_proj.weight", None)}
    _attention_tensors = {"mix.q.norm": ("mixer.q_norm.weight", None), "mix.k.norm": ("mixer.k_norm.weight", None),
                          "mix.o": ("mixer.out_proj.weight", None)}

    def _place(self, name: str) -> Optional[tuple[str, object, Optional[int]]]:
        """(parameter, shard, expert) of a checkpoint tensor; None: it belongs to another pipeline stage."""
        if name == "final.norm":
            return ("model.norm.weight", None, None) if self.is_last else None
        idx, _, rest = name[1:].partition(".")
        if name[:1] == "l" and idx.isdigit() and int(idx) < len(self.cfg["layers"]):
            i = int(idx)
            if not self.model.start <= i < self.model.end:
                return None
            head, layer = f"model.layers.{i - self.model.start}.", self.model.layers[i - self.model.start]
            part = rest.split(".")
            if layer.mlp_kind == "moe" and len(part) == 3 and part[0] == "mlp" and part[1][:1] == "e" and part[1][1:].isdigit() \
                    and part[2] in self._expert_shards and int(part[1][1:]) < layer.mlp.experts.num_experts:
                p, shard = self._expert_shards[part[2]]
                return f"{head}mlp.experts.{p}", shard, int(part[1][1:])
            places = [self._layer_tensors, {"dense": self._dense_tensors, "moe": self._moe_tensors}.get(layer.mlp_kind, {})]
            if layer.kind == "mlstm":
                places.append(self._mlstm_tensors)
            else:
                names = "qg" if layer.mixer.shares else "qkvg"
                places.append({**self._attention_tensors, **{f"mix.{n}": ("mixer.in_proj.weight", j) for j, n in enumerate(names)},
                               **{f"mix.{n}.b": ("mixer.in_proj.bias", j) for j, n in enumerate(names) if n != "g"}})
            for table in places:
                if rest in table:
                    return head + table[rest][0], table[rest][1], None
        raise ValueError(f"unexpected tensor {name!r} in a Kopadra checkpoint")

    def load_weights(self, weights: Iterable[tuple[str, torch.Tensor]]) -> set[str]:
        params, modules = dict(self.named_parameters(remove_duplicate=False)), dict(self.named_modules())
        loaded: set[str] = set()
        for name, w in weights:
            if name == "embed":
                places = [("model.embed_tokens.weight", None, None)] if self.model.embed_tokens is not None else []
                if self.is_last and not self.tied:
                    places.append(("lm_head.weight", None, None))
            else:
                got = self._place(name)
                places = [] if got is None else [got]
            for target, shard, expert in places:
                if target not in params:
                    raise ValueError(f"tensor {name!r} has no place in this configuration")
                p, mod = params[target], modules[target.rsplit(".", 1)[0]]
                loader = getattr(mod, "weight_loader", None)
                if expert is not None:
                    mod.weight_loader(p, w, shard, expert)
                elif loader is not None:
                    loader(p, w, shard)
                else:
                    dst = p.data if shard is None else p.data.chunk(2)[shard]
                    assert dst.shape == w.shape, (name, dst.shape, w.shape)
                    dst.copy_(w)
                loaded.add(target)
        return loaded
