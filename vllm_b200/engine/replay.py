"""Replay of a trace of steps: given token ids go through the engine step by step and chosen logits come out.

Steps arrive on standard input, one JSON object a line::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}

``entries`` bring each request's next tokens — whole prompts, portions of prompts and single tokens side by side, run as
ONE batch — and ``want`` the places among them whose logits are asked for; ``end`` lists requests that are finished after
the step.  The logits of a step go to ``<out>/<step>.f32`` (little-endian 32-bit floats, [wanted, vocab], in the order of
the entries), and ``done <step>`` is printed when it is complete.

Nothing here computes: the steps run through the engine core's scheduler (slots of its cache manager, given back at
``end``), executor and model runner, with the kernels that generation uses.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import IO, Any, Optional

import numpy as np

from vllm_b200.core.request import RequestStatus
from vllm_b200.engine.arg_utils import EngineArgs
from vllm_b200.engine.core import EngineCore
from vllm_b200.sampling_params import SamplingParams
from vllm_b200.utils import cdiv

MAX_LIVE_REQUESTS = 4


class StepReplay:
    """An engine core for prescribed steps.  ``max_tokens``: the most tokens live requests hold at any time, each
    request's count rounded up to whole pages — the cache pool has exactly that many slots."""

    def __init__(self, model: str, dtype: str = "bfloat16", max_tokens: int = 2048, max_requests: int = MAX_LIVE_REQUESTS,
                 **engine_args: Any) -> None:
        kw = dict(dtype=dtype, skip_tokenizer_init=True, enforce_eager=True, enable_prefix_caching=False, max_num_seqs=max_requests,
                  max_num_batched_tokens=max_tokens, gpu_memory_utilization=0.5, kv_cache_memory_bytes=16 << 30,
                  distributed_executor_backend="uni")
        args = EngineArgs(model=model, **{**kw, **engine_args})
        cfg = args.create_engine_config()
        page = cfg.cache_config.block_size
        longest = min(cfg.scheduler_config.max_model_len, cdiv(max_tokens, page) * page)
        cfg.scheduler_config.max_model_len = cfg.model_config.max_model_len = longest
        cfg.cache_config.num_gpu_blocks_override = cdiv(max_tokens, page) + 1     # + the null page
        self.core = EngineCore(cfg)
        self.device = self.core.model_executor.worker.device
        self.sampling = SamplingParams(temperature=0.0, max_tokens=1, ignore_eos=True)

    def step(self, entries: list[dict], end: Optional[list[str]] = None) -> np.ndarray:
        """Runs one step; returns the wanted logits [wanted, vocab]."""
        rows: list[np.ndarray] = []
        if entries:
            got = self.core.run_given([(e["id"], e["tokens"]) for e in entries], {e["id"]: e.get("want") or [] for e in entries},
                                      self.sampling)
            rows = [got[e["id"]].numpy() for e in entries if e.get("want")]
            if self.device.type == "cuda":
                from vllm_b200.ops import cuda_ops
                cuda_ops().check_kernel_error(self.device)
        if end:
            self.core.scheduler.finish_requests(list(end), RequestStatus.FINISHED_ABORTED)
        vocab = self.core.vllm_config.model_config.vocab_size
        return np.concatenate(rows) if rows else np.zeros((0, vocab), dtype=np.float32)

    def run(self, lines: IO[str], out_dir: str, report: IO[str]) -> None:
        for line in lines:
            if not line.strip():
                continue
            s = json.loads(line)
            logits = self.step(s.get("entries") or [], s.get("end"))
            if len(logits):
                logits.astype("<f4").tofile(os.path.join(out_dir, f"{s['step']}.f32"))
            print(f"done {s['step']}", file=report, flush=True)

    def shutdown(self) -> None:
        self.core.shutdown()


def main(argv: Optional[list[str]] = None) -> None:
    ap = argparse.ArgumentParser("trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="folder with config.json and the weights")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True,
                    help="the most tokens live requests hold at any time, each request's count rounded up to whole pages")
    ap.add_argument("--device", default="auto", help="auto, cuda or cpu")
    a = ap.parse_args(argv)
    os.makedirs(a.out, exist_ok=True)
    replay = StepReplay(a.model, a.dtype, a.max_tokens, device=a.device)
    replay.run(sys.stdin, a.out, sys.stdout)
    replay.shutdown()


if __name__ == "__main__":
    main()
