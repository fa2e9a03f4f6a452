"""Hyper-connections: several copies of the residual stream, read and written by every sublayer with weights of its own.

    u = sum_s in[s] x_s;   y = sublayer(norm(u));   x_t <- sum_s mix[s, t] x_s + out[t] y

The streams x [T, S, H] and the three weights are fp32.  The write of one sublayer, the read of the next and its norm are one step
(``ops.hyper_step``, csrc/stream.cu): a stream is read and written once per sublayer and u never exists in memory.
"""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn as nn

from vllm_b200 import ops
from vllm_b200.layers.common import RMSNorm


class HyperConnection(nn.Module):
    """The weights of one sublayer."""

    def __init__(self, streams: int) -> None:
        super().__init__()
        self.streams = streams
        self.into = nn.Parameter(torch.full((streams,), 1.0 / streams, dtype=torch.float32), requires_grad=False)
        coef = torch.cat([torch.ones(streams), torch.eye(streams).flatten()])
        self.coef = nn.Parameter(coef.to(self.into), requires_grad=False)            # out [S], then mix [S (from), S (to)]

    def weight_loader(self, param: nn.Parameter, w: torch.Tensor, shard_id=None) -> None:
        S = self.streams
        dst = {"in": self.into.data, "out": self.coef.data[:S], "mix": self.coef.data[S:].view(S, S)}[shard_id]
        assert dst.shape == w.shape, (shard_id, dst.shape, w.shape)
        dst.copy_(w)

    def step(self, x: torch.Tensor, y: torch.Tensor, into: torch.Tensor, norm: RMSNorm) -> torch.Tensor:
        """Writes y to the streams; returns what the next sublayer reads (``into``), normed."""
        return ops.hyper_step(x, y, self.coef, into, norm.weight, norm.eps)


def enter(ids: Optional[torch.Tensor], table: torch.Tensor, embed_norm: Optional[RMSNorm], first: HyperConnection, norm: RMSNorm
          ) -> tuple[torch.Tensor, torch.Tensor]:
    """(equal streams of the normed embeddings, what the first sublayer reads, normed).  ``ids`` None: ``table`` holds a row per token."""
    return ops.hyper_entry(ids, table, first.streams, None if embed_norm is None else embed_norm.weight, first.into, norm.weight, norm.eps)
