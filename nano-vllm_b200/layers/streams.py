"""Hyper-connections: the residual is kept as several fp32 copies ("streams").

A sublayer reads one combination of the copies and its output goes back to all
of them after they have been mixed.  What lies between two sublayers - mix,
add, the next combination and its RMSNorm - is one launch (ops.stream_step).
"""
from __future__ import annotations

import torch
from torch import nn

from .. import ops


class StreamConnection(nn.Module):
    """The coefficients of one sublayer: w_in [S], w_out [S], mix [from, to]."""

    def __init__(self, streams: int) -> None:
        super().__init__()
        self.w_in = nn.Parameter(torch.zeros(streams, dtype=torch.float32), requires_grad=False)
        self.w_out = nn.Parameter(torch.zeros(streams, dtype=torch.float32), requires_grad=False)
        self.mix = nn.Parameter(torch.zeros(streams, streams, dtype=torch.float32), requires_grad=False)


class StreamNorm(nn.Module):
    """RMSNorm of a stream combination; the weight is kept in fp32 and padded with zeros to the stored width."""

    def __init__(self, dim: int, padded: int, eps: float) -> None:
        super().__init__()
        self.dim, self.eps = dim, eps
        self.weight = nn.Parameter(torch.zeros(padded, dtype=torch.float32), requires_grad=False)
        self.weight.weight_loader = self.weight_loader

    def weight_loader(self, param: nn.Parameter, loaded_weight: torch.Tensor):
        param.data[:self.dim].copy_(loaded_weight)

    def start(self, ids: torch.Tensor, table: torch.Tensor, scale: float, streams: int, conn: StreamConnection):
        """Streams of the embedding output and the first sublayer's input."""
        x = torch.empty(ids.numel(), streams, table.shape[1], dtype=torch.float32, device=table.device)
        normed = ops.stream_step(x, None, None, None, 0.0, conn.w_in, self.weight, self.eps, self.dim, embed=(ids, table, scale))
        return x, normed

    def step(self, x: torch.Tensor, y: torch.Tensor, conn: StreamConnection, mult: float, w_in: torch.Tensor | None, store: bool) -> torch.Tensor:
        """Adds sublayer output y through `conn`, then this norm of the combination w_in (None: the plain sum)."""
        return ops.stream_step(x, y, conn.mix, conn.w_out, mult, w_in, self.weight, self.eps, self.dim, store=store)
