"""Gizilorn: windowed attention whose heads talk to one another, beside windowed latent attention, in pre-norm blocks joined by
hyper-connections.

    x_s = N(E[t])                                        S equal streams
    u = sum_s in[s] x_s;  y = F_n(N(u));  x_t <- sum_s mix[s, t] x_s + out[t] y         F_n: mixer and feed-forward in turn
    logits = W N(sum_s x_s)

* The streams stay in fp32; one kernel per boundary (``layers/hyper.py``) writes F_n's output to them and takes the next N.
* ``attention`` layers: capped scores, a sink of score zero in the softmax, weights mixed across heads behind it (``Attention(talk=)``), and
  values that are cached rotated by their position and turned back in the output (``Attention(v_rope=)``).
* ``latent_attention`` layers: ``layers/latent.py`` with direct queries, a rotated part and an output gate; a layer with ``kv_from`` reads
  the latents of that earlier layer.
* Feed-forward: two biased projections around xIELU, whose two numbers are learned per layer.

Every layer has a window.  Pages stay for the longest of them, so that all layers share pages and one block table.  Sizes and
constants come from the configuration layer by layer: layers may differ in everything, and a layer may have no feed-forward.  Under
tensor parallelism the attention layers are replicated (each head needs the weights of all); latent layers, feed-forwards and the
head are sharded.
"""
from __future__ import annotations

from typing import Iterable, Optional

import torch
import torch.nn as nn

from vllm_b200 import ops
from vllm_b200.config import VllmConfig
from vllm_b200.layers import hyper
from vllm_b200.layers.attention import Attention
from vllm_b200.layers.common import XIELU, RMSNorm, VocabParallelEmbedding
from vllm_b200.layers.latent import LatentAttention
from vllm_b200.layers.linear import ColumnParallelLinear, LinearMethod, MergedReplicatedLinear, ReplicatedLinear, RowParallelLinear
from vllm_b200.layers.rotary import get_rope
from vllm_b200.models.llama import LlamaForCausalLM
from vllm_b200.parallel.state import get_pp_group
from vllm_b200.parallel.utils import get_pp_indices


class TalkingAttention(nn.Module):
    def __init__(self, hidden: int, m: dict, max_position: int, cache_window: int, dtype, prefix: str) -> None:
        super().__init__()
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        base = float(m["rot"]["base"])
        self.in_proj = MergedReplicatedLinear(hidden, [H * d, G * d, G * dv], True, dtype, None, f"{prefix}.in_proj", align=8)
        self.talk = nn.Parameter(torch.eye(H, dtype=torch.float32), requires_grad=False)
        self.attn = Attention(H, d, m["scale"], G, sliding_window=m["mask"]["size"], logits_soft_cap=float(m["softcap"]),
                              prefix=f"{prefix}.attn", rope=get_rope(d, m["rot"]["dims"], max_position, base, True, dict(exact=True)),
                              sinks=torch.zeros(H), v_head_size=dv, fused_prologue=True, talk=self.talk,
                              v_rope=get_rope(dv, dv, max_position, base, True, dict(exact=True)), cache_window=cache_window)
        self.out_proj = ReplicatedLinear(H * dv, hidden, False, dtype, None, f"{prefix}.out_proj")

    def forward(self, positions: torch.Tensor, h: torch.Tensor) -> torch.Tensor:
        return self.out_proj(self.attn(*self.in_proj.parts(self.in_proj(h)), positions))


class GizilornMLP(nn.Module):
    def __init__(self, hidden: int, ff: int, dtype, quant_config, prefix: str) -> None:
        super().__init__()
        self.up_proj = ColumnParallelLinear(hidden, ff, True, dtype=dtype, quant_config=quant_config, prefix=f"{prefix}.up_proj")
        self.act = XIELU()
        self.down_proj = RowParallelLinear(ff, hidden, True, dtype=dtype, quant_config=quant_config, prefix=f"{prefix}.down_proj")

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        up = self.up_proj
        if type(up.quant_method) is LinearMethod and not up.lora_table:
            return self.down_proj(ops.linear_xielu(h, up.weight, up.bias, self.act.coef))
        return self.down_proj(self.act(up(h)))


class GizilornLayer(nn.Module):
    def __init__(self, cfg: dict, max_position: int, dtype, quant_config, layers_prefix: str, idx: int) -> None:
        super().__init__()
        spec, prefix = cfg["layers"][idx], f"{layers_prefix}.{idx}"
        H, eps = cfg["hidden_size"], cfg["norm"]["eps"]
        keep = max(l["mixer"]["mask"]["size"] for l in cfg["layers"])
        self.kind, m = spec["type"], spec["mixer"]
        if self.kind == "attention":
            self.mixer = TalkingAttention(H, m, max_position, keep, dtype, f"{prefix}.mixer")
        elif self.kind == "latent_attention":
            j = m.get("kv_from")
            rope = get_rope(m["rot_dim"], m["rot_dim"], max_position, float(m["rot"]["base"]), False, dict(exact=True)) if m["rot_dim"] else None
            self.mixer = LatentAttention(H, m["heads"], m["dim"], m["vdim"], 0, m["kv_rank"], m["scale"], eps, dtype, quant_config,
                                         f"{prefix}.mixer", None if j is None else f"{layers_prefix}.{j}.mixer.attn", rope,
                                         m["mask"]["size"], keep, True)
        else:
            raise ValueError(f"{prefix}: unknown mixer {self.kind!r}")
        self.norm1, self.hc1 = RMSNorm(H, eps, dtype), hyper.HyperConnection(cfg["streams"])
        self.mlp = None
        if spec.get("mlp") is not None:
            if spec["mlp"]["kind"] != "dense":
                raise ValueError(f"{prefix}: unknown feed-forward kind {spec['mlp']['kind']!r}")
            self.mlp = GizilornMLP(H, spec["mlp"]["ff"], dtype, quant_config, f"{prefix}.mlp")
            self.norm2, self.hc2 = RMSNorm(H, eps, dtype), hyper.HyperConnection(cfg["streams"])

    def mix(self, positions: torch.Tensor, h: torch.Tensor) -> torch.Tensor:
        return self.mixer(positions, h) if self.kind == "attention" else self.mixer(h, positions)


class GizilornModel(nn.Module):
    def __init__(self, vllm_config: VllmConfig, prefix: str = "model", quant_config=None) -> None:
        super().__init__()
        mc = vllm_config.model_config
        self.cfg = cfg = mc.hf_config
        dtype = mc.torch_dtype
        pp = get_pp_group()
        self.pp_rank, self.pp_size = max(pp.rank_in_group, 0), pp.world_size
        self.start, self.end = get_pp_indices(cfg["num_hidden_layers"], self.pp_rank, self.pp_size)
        H, eps = cfg["hidden_size"], cfg["norm"]["eps"]
        self.embed_tokens = self.embed_norm = None
        if self.pp_rank == 0:
            self.embed_tokens = VocabParallelEmbedding(cfg["vocab_size"], H, dtype, prefix=f"{prefix}.embed_tokens", replicate=True)
            self.embed_norm = RMSNorm(H, eps, dtype)
        self.layers = nn.ModuleList([GizilornLayer(cfg, mc.max_model_len, dtype, quant_config, f"{prefix}.layers", i)
                                     for i in range(self.start, self.end)])
        self.norm = RMSNorm(H, eps, dtype) if self.pp_rank == self.pp_size - 1 else None
        self.register_buffer("ones", torch.ones(cfg["streams"], dtype=torch.float32), persistent=False)

    def embed_input_ids(self, input_ids: torch.Tensor) -> torch.Tensor:
        return self.embed_norm(self.embed_tokens(input_ids))

    def forward(self, input_ids, positions, intermediate_tensors=None, inputs_embeds=None):
        steps = []                                  # (sublayer, its connection, its norm)
        for layer in self.layers:
            steps.append((lambda h, layer=layer: layer.mix(positions, h), layer.hc1, layer.norm1))
            if layer.mlp is not None:
                steps.append((layer.mlp, layer.hc2, layer.norm2))
        _, hc, norm = steps[0]
        if self.pp_rank > 0:
            x, h = intermediate_tensors["residual"].contiguous(), intermediate_tensors["hidden_states"]
            h = ops.hyper_step(x, None, None, hc.into, norm.weight, norm.eps, h.dtype)
        elif inputs_embeds is not None:
            x, h = hyper.enter(None, inputs_embeds, None, hc, norm)
        else:
            x, h = hyper.enter(input_ids, self.embed_tokens.weight, self.embed_norm, hc, norm)
        for i, (sublayer, hc, norm) in enumerate(steps):
            # the last sublayer's successor reads the plain sum of the streams (on a stage that is not the last, nothing reads h)
            into, nxt = (steps[i + 1][1].into, steps[i + 1][2]) if i + 1 < len(steps) else (self.ones, self.norm or norm)
            h = hc.step(x, sublayer(h), into, nxt)
        if self.norm is None:
            return {"hidden_states": h, "residual": x}
        return h


class GizilornForCausalLM(LlamaForCausalLM):
    model_cls = GizilornModel

    def __init__(self, vllm_config: VllmConfig, prefix: str = "") -> None:
        if vllm_config.cache_config.cache_dtype.startswith("fp8"):
            raise ValueError("latents and rotated values are cached in the model dtype (kv_cache_dtype fp8 is not supported)")
        super().__init__(vllm_config, prefix)

    @staticmethod
    def kernel_sources(cfg: dict, dtype: torch.dtype) -> list[str]:
        """CUDA sources of this model's steps (ops/cuda.py ``prebuild``)."""
        out = {"stream", "norm_act", "input_prep"}
        half = dtype != torch.float32
        cu = ops.cuda_ops()
        attn = [l["mixer"] for l in cfg["layers"] if l["type"] == "attention"]
        latent = [l["mixer"] for l in cfg["layers"] if l["type"] == "latent_attention"]
        if attn:
            out |= {"qknorm_rope", "rope_cache", "attention_talk"} if half else {"qknorm_rope", "attention_talk"}
            # one cache layout for all attention layers: the tensor-core kernels run where they take every layer's head shape
            if half and all(cu.tc_attention_ok(a["dim"], a["vdim"], a["heads"] // a["kv_heads"]) for a in attn):
                out |= {"attention_tc", "attention_talk_decode"}
            else:
                out.add("attention_any")
        if latent:
            out.add("latent")
        if half and latent:
            out |= {"mla_decode", "mla_prefill", "cache_ops"}
        if half:
            out.add("gemm_tc")
        return sorted(out)

    # checkpoint tensor (behind "l<i>.") → (parameter, shard)
    _layer_tensors = {"norm1": ("norm1.weight", None), **{f"hc1.{n}": ("hc1.coef" if n != "in" else "hc1.into", n) for n in ("in", "out", "mix")}}
    _mlp_tensors = {"norm2": ("norm2.weight", None), **{f"hc2.{n}": ("hc2.coef" if n != "in" else "hc2.into", n) for n in ("in", "out", "mix")},
                    "mlp.up": ("mlp.up_proj.weight", None), "mlp.up.b": ("mlp.up_proj.bias", None), "mlp.act": ("mlp.act.coef", None),
                    "mlp.down": ("mlp.down_proj.weight", None), "mlp.down.b": ("mlp.down_proj.bias", None)}
    _attention_tensors = {**{f"mix.{n}": ("mixer.in_proj.weight", i) for i, n in enumerate("qkv")},
                          **{f"mix.{n}.b": ("mixer.in_proj.bias", i) for i, n in enumerate("qkv")},
                          "mix.talk": ("mixer.talk", None), "mix.o": ("mixer.out_proj.weight", None)}
    _latent_tensors = {"mix.uk": ("mixer.ukv.weight", 0), "mix.uv": ("mixer.ukv.weight", 1), "mix.o": ("mixer.o.weight", None)}
    _model_tensors = {"embed": "model.embed_tokens.weight", "embed.norm": "model.embed_norm.weight", "final.norm": "model.norm.weight",
                      "head": "lm_head.weight"}

    def _place(self, name: str) -> Optional[tuple[str, object]]:
        """(parameter, shard) of a checkpoint tensor; None: it belongs to another pipeline stage."""
        if name in self._model_tensors:
            here = self.model.embed_tokens is not None if name.startswith("embed") else self.is_last
            return (self._model_tensors[name], None) if here else None
        idx, _, rest = name[1:].partition(".")
        if name[:1] == "l" and idx.isdigit() and int(idx) < len(self.cfg["layers"]):
            i = int(idx)
            if not self.model.start <= i < self.model.end:
                return None
            layer = self.model.layers[i - self.model.start]
            places = dict(self._layer_tensors)
            if layer.mlp is not None:
                places.update(self._mlp_tensors)
            if layer.kind == "attention":
                places.update(self._attention_tensors)
            else:
                part = layer.mixer.part
                places.update(self._latent_tensors)
                places.update({"mix.q": ("mixer.in_proj.weight", part["q"]), "mix.g": ("mixer.in_proj.weight", part["g"])})
                if "kv" in part:
                    places.update({"mix.dkv": ("mixer.in_proj.weight", part["kv"]), "mix.dkv.norm": ("mixer.kv_norm.weight", None)})
            if rest in places:
                return f"model.layers.{i - self.model.start}.{places[rest][0]}", places[rest][1]
        raise ValueError(f"unexpected tensor {name!r} in a Gizilorn checkpoint")

    def load_weights(self, weights: Iterable[tuple[str, torch.Tensor]]) -> set[str]:
        params, modules = dict(self.named_parameters()), dict(self.named_modules())
        loaded: set[str] = set()
        for name, w in weights:
            got = self._place(name)
            if got is None:
                continue
            target, shard = got
            p, mod = params[target], modules[target.rsplit(".", 1)[0]]
            loader = getattr(mod, "weight_loader", None)
            if target.endswith("_proj.bias") and isinstance(mod, ColumnParallelLinear):
                n = p.shape[0]
                p.data.copy_(w.narrow(0, mod.tp_rank * n, n))
            elif loader is not None:
                loader(p, w, shard)
            else:
                assert p.shape == w.shape, (name, p.shape, w.shape)
                p.data.copy_(w)
            loaded.add(target)
        return loaded
