"""Helpers of the tests that run small models through the engine and compare logits with a plain implementation."""
from __future__ import annotations

import json
import os

import pytest
import torch

# largest row error over the spread of the logits
TOL = {"float32": 2e-4, "bfloat16": 0.12}
PLACES = [pytest.param(("cpu", "float32"), id="cpu-float32"),
          pytest.param(("cuda", "bfloat16"), id="cuda-bfloat16", marks=pytest.mark.gpu),
          pytest.param(("cuda", "float32"), id="cuda-float32", marks=pytest.mark.gpu)]


class Engine:
    """A replay of one model; ``feed`` runs steps and collects logits per request and position."""

    def __init__(self, path, place, max_tokens=1024, **kw):
        from vllm_b200.engine.replay import StepReplay
        self.replay = StepReplay(path, place[1], max_tokens, device=place[0], **kw)
        self.at, self.rows = {}, {}

    def feed(self, *steps):
        """A step is a list of (request, tokens, finished?)."""
        for step in steps:
            got = self.replay.step([dict(id=r, tokens=t, want=list(range(len(t)))) for r, t, *_ in step],
                                   [r for r, _, *e in step if e and e[0]])
            n = 0
            for r, t, *_ in step:
                self.rows.setdefault(r, []).append(torch.from_numpy(got[n:n + len(t)]))
                n += len(t)
        return self

    def logits(self, r):
        return torch.cat(self.rows.pop(r))

    def __enter__(self):
        return self

    def __exit__(self, *_):
        self.replay.shutdown()


def portions(toks, sizes):
    out, i, k = [], 0, 0
    while i < len(toks):
        out.append(toks[i:i + sizes[k % len(sizes)]])
        i, k = i + sizes[k % len(sizes)], k + 1
    return out


def save_model(cfg, w, path):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in w.items()}, os.path.join(path, "model.safetensors"))
    return str(path)


def tokens(cfg, n, seed=0, avoid=()):
    g = torch.Generator().manual_seed(1000 + seed)
    ok = torch.tensor([t for t in range(cfg["vocab"]) if t not in avoid])
    return ok[torch.randint(0, len(ok), (n,), generator=g)].tolist()


def row_error(got, want):
    """Largest error of a row of logits, mean taken off, over the spread of the expected logits."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    spread = (want.double() - want.double().mean(-1, keepdim=True)).pow(2).mean().sqrt()
    return float((d.pow(2).mean(-1).sqrt() / spread).max()) if len(d) else 0.0


def make_llm(path, place, **kw):
    from vllm_b200 import LLM
    d = dict(device=place[0], dtype=place[1], max_model_len=320, max_num_seqs=8, max_num_batched_tokens=64, skip_tokenizer_init=True,
             kv_cache_memory_bytes=16 << 20)
    return LLM(path, **{**d, **kw})


def generate(llm, prompts, n):
    from vllm_b200 import SamplingParams
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts],
                        SamplingParams(max_tokens=n, temperature=0.0, ignore_eos=True, detokenize=False))
    return [list(o.outputs[0].token_ids) for o in outs]


def check_greedy(forward, prompts, got, slack):
    """Every generated token is the best by the equations (``forward``: tokens → logits), within ``slack`` of their spread."""
    for p, out in zip(prompts, got):
        lg = forward(p + out[:-1])[len(p) - 1:]
        spread = lg.std()
        for row, t in zip(lg, out):
            assert float(row.max() - row[t]) <= slack * float(spread)
