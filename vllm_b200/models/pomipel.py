"""Pomipel: position-free latent attention and group-limited experts in post-norm residual blocks.

    x_0 = s_e E[t] + P[i]                 token t at index i: scaled embedding plus a learned position
    x_{n+1} = x_n + N(F_n(x_n))           F_n: attention and experts in turn; the norm N is behind F_n, nothing in front of it
    logits = s_l W_head N(x_last)

* The stream x stays in fp32 (csrc/stream.cu); each step leaves the 16-bit copy the next GEMM reads.
* Mixer: ``layers/latent.py``; a layer with ``kv_from`` reads the latent cache of that earlier layer.
* Feed-forward: ungated squared-ReLU experts (``FusedMoE(gated=False)``) behind a sigmoid router with a selection bias and
  group-limited choice, in 32-bit (``GroupedRouter``); a chosen expert is mixed in with its plain sigmoid score.

Sizes and constants come from the configuration layer by layer: layers may differ in heads, widths and experts, and a
layer may have no feed-forward.
"""
from __future__ import annotations

from typing import Iterable, Optional

import torch
import torch.nn as nn

from vllm_b200 import ops
from vllm_b200.config import VllmConfig
from vllm_b200.layers.common import LogitsProcessor, ParallelLMHead, RMSNorm, VocabParallelEmbedding
from vllm_b200.layers.latent import LatentAttention
from vllm_b200.layers.moe import FusedMoE, GroupedRouter
from vllm_b200.models.llama import LlamaForCausalLM
from vllm_b200.parallel.state import get_pp_group
from vllm_b200.parallel.utils import get_pp_indices


class PomipelExperts(nn.Module):
    def __init__(self, spec: dict, hidden_size: int, dtype, quant_config, prefix: str, enable_ep: bool) -> None:
        super().__init__()
        if spec.get("kind") != "moe":
            raise ValueError(f"{prefix}: unknown feed-forward kind {spec.get('kind')!r}")
        r = spec["router"]
        groups = r.get("groups") or {"count": 1, "keep": 1}
        self.router = GroupedRouter(hidden_size, r["experts"], r["top"], dtype, groups["count"], groups["keep"])
        self.experts = FusedMoE(r["experts"], r["top"], hidden_size, spec["expert"]["ff"], dtype, act="relu2", gated=False,
                                enable_ep=enable_ep, prefix=f"{prefix}.experts", quant_config=quant_config)

    def forward_post_norm(self, h, stream, norm, next_norm):
        return self.experts.forward_post_norm(h, self.router(stream, h), stream, norm, next_norm)


class PomipelLayer(nn.Module):
    def __init__(self, cfg: dict, dtype, quant_config, layers_prefix: str, idx: int, enable_ep: bool) -> None:
        super().__init__()
        spec = cfg["layers"][idx]
        H, eps = cfg["hidden_size"], cfg["norm"]["eps"]
        prefix = f"{layers_prefix}.{idx}"
        if spec["type"] != "latent_attention":
            raise ValueError(f"{prefix}: unknown mixer {spec['type']!r}")
        m = spec["mixer"]
        src = m.get("kv_from")
        self.mixer = LatentAttention(H, m["heads"], m["dim"], m["vdim"], m["q_rank"], m["kv_rank"], m["scale"], eps, dtype,
                                     quant_config, f"{prefix}.mixer",
                                     None if src is None else f"{layers_prefix}.{src}.mixer.attn")
        self.norm1 = RMSNorm(H, eps, dtype, gemma=True)
        self.mlp = self.norm2 = None
        if spec.get("mlp") is not None:
            self.mlp = PomipelExperts(spec["mlp"], H, dtype, quant_config, f"{prefix}.mlp", enable_ep)
            self.norm2 = RMSNorm(H, eps, dtype, gemma=True)

    def forward(self, stream: torch.Tensor, h: torch.Tensor, next_norm: Optional[RMSNorm]) -> torch.Tensor:
        """``stream`` (fp32) is updated in place; ``h`` is its copy in the model dtype.  Returns the next copy, or
        ``next_norm`` of the stream."""
        last = next_norm if self.mlp is None else None
        n1 = self.norm1
        h = ops.post_norm_add(stream, self.mixer(h), n1.weight, n1.eps, True, None if last is None else last.weight, True)
        if self.mlp is None:
            return h
        return self.mlp.forward_post_norm(h, stream, self.norm2, next_norm)


class PomipelModel(nn.Module):
    def __init__(self, vllm_config: VllmConfig, prefix: str = "model", quant_config=None) -> None:
        super().__init__()
        mc = vllm_config.model_config
        self.cfg = cfg = mc.hf_config
        dtype = mc.torch_dtype
        pp = get_pp_group()
        self.pp_rank, self.pp_size = max(pp.rank_in_group, 0), pp.world_size
        self.start, self.end = get_pp_indices(cfg["num_hidden_layers"], self.pp_rank, self.pp_size)
        H = cfg["hidden_size"]
        self.embed_scale = float(cfg["embedding"]["scale"])
        self.embed_tokens = self.pos_embed = None
        if self.pp_rank == 0:
            self.embed_tokens = VocabParallelEmbedding(cfg["vocab_size"], H, dtype, prefix=f"{prefix}.embed_tokens", replicate=True)
            self.pos_embed = nn.Embedding(cfg["max_positions"], H, dtype=dtype)
            self.pos_embed.weight.requires_grad_(False)
        ep = bool(vllm_config.parallel_config.enable_expert_parallel)
        self.layers = nn.ModuleList([PomipelLayer(cfg, dtype, quant_config, f"{prefix}.layers", i, ep)
                                     for i in range(self.start, self.end)])
        self.norm = RMSNorm(H, cfg["norm"]["eps"], dtype, gemma=True) if self.pp_rank == self.pp_size - 1 else None

    def embed_input_ids(self, input_ids: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError("input embeddings cannot replace token ids here: the learned position vector of each token "
                                  "is added in the same step")

    def forward(self, input_ids, positions, intermediate_tensors=None, inputs_embeds=None):
        if inputs_embeds is not None:
            raise NotImplementedError("Pomipel takes token ids")
        if self.pp_rank == 0:
            stream, h = ops.embed_stream(input_ids, positions, self.embed_tokens.weight, self.pos_embed.weight, self.embed_scale)
        else:
            stream, h = intermediate_tensors["residual"].contiguous(), intermediate_tensors["hidden_states"]
        for i, layer in enumerate(self.layers):
            h = layer(stream, h, self.norm if i + 1 == len(self.layers) else None)
        if self.norm is None:
            return {"hidden_states": h, "residual": stream}
        return h


class PomipelForCausalLM(LlamaForCausalLM):
    model_cls = PomipelModel
    # CUDA sources of this model's steps (ops/cuda.py ``prebuild``)
    kernel_sources = ("stream", "latent", "mla_decode", "mla_prefill", "moe", "gemm_tc", "cache_ops", "input_prep")

    def __init__(self, vllm_config: VllmConfig, prefix: str = "") -> None:
        mc = vllm_config.model_config
        if mc.max_model_len > mc.hf_config["max_positions"]:
            raise ValueError(f"max_model_len {mc.max_model_len} exceeds the model's {mc.hf_config['max_positions']} learned positions")
        if vllm_config.cache_config.cache_dtype.startswith("fp8"):
            raise ValueError("latent caches hold the model dtype (kv_cache_dtype fp8 is not supported)")
        super().__init__(vllm_config, prefix)
        if self.is_last:
            self.logits_processor = LogitsProcessor(mc.vocab_size, scale=float(mc.hf_config["logit_scale"]))

    # checkpoint tensor (behind "l<i>.") → (parameter, shard)
    _layer_tensors = {"norm1": ("norm1.weight", None), "norm2": ("norm2.weight", None), "mix.dq": ("mixer.down.weight", 0),
                      "mix.dq.norm": ("mixer.q_norm.weight", None), "mix.uq": ("mixer.uq.weight", None),
                      "mix.dkv": ("mixer.down.weight", 1), "mix.dkv.norm": ("mixer.kv_norm.weight", None),
                      "mix.uk": ("mixer.ukv.weight", 0), "mix.uv": ("mixer.ukv.weight", 1), "mix.o": ("mixer.o.weight", None),
                      "mlp.router": ("mlp.router.weight", None), "mlp.correction": ("mlp.router.bias", None)}
    _model_tensors = {"embed": "model.embed_tokens.weight", "pos": "model.pos_embed.weight", "final.norm": "model.norm.weight",
                      "head": "lm_head.weight"}

    def load_weights(self, weights: Iterable[tuple[str, torch.Tensor]]) -> set[str]:
        params, modules = dict(self.named_parameters()), dict(self.named_modules())
        loaded: set[str] = set()
        for name, w in weights:
            shard: object = None
            expert = None
            if name in self._model_tensors:
                target = self._model_tensors[name]
            elif name[:1] == "l" and name[1:].split(".", 1)[0].isdigit():
                idx, rest = name[1:].split(".", 1)
                if not self.model.start <= int(idx) < self.model.end:
                    continue                                        # another pipeline stage
                head = f"model.layers.{int(idx) - self.model.start}."
                part = rest.split(".")
                if part[0] == "mlp" and len(part) == 3 and part[1][:1] == "e" and part[1][1:].isdigit():
                    expert = int(part[1][1:])
                    suffix, shard = {"up": ("w13_weight", "w1"), "down": ("w2_weight", "w2")}[part[2]]
                    target = f"{head}mlp.experts.{suffix}"
                elif rest in self._layer_tensors:
                    suffix, shard = self._layer_tensors[rest]
                    target = head + suffix
                else:
                    raise ValueError(f"unexpected tensor {name!r} in a Pomipel checkpoint")
            else:
                raise ValueError(f"unexpected tensor {name!r} in a Pomipel checkpoint")
            if target not in params:
                if target in self._model_tensors.values():
                    continue                                        # another pipeline stage
                raise ValueError(f"tensor {name!r} has no place in this configuration")
            p, mod = params[target], modules[target.rsplit(".", 1)[0]]
            loader = getattr(mod, "weight_loader", None)
            if expert is not None:
                mod.weight_loader(p, w, shard, expert)
            elif loader is not None:
                loader(p, w, shard)
            else:
                assert p.shape == w.shape, (name, p.shape, w.shape)
                p.data.copy_(w)
            loaded.add(target)
        return loaded
