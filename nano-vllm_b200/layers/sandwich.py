"""Sublayers between two norms: x <- x + norm_out(sublayer(conv(norm_in(x)))), x one fp32 residual.

What lies between two sublayers - the norm of the output, the residual sum, the next norm and its causal convolution - is one
launch (ops.sandwich_step).
"""
from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..utils.context import get_context
from .linear import pad8
from .state import SlotState


class GainNorm(nn.Module):
    """RMSNorm with fp32 weights: one gain for all channels, or (per_channel) one per channel, padded with zeros."""

    def __init__(self, dim: int, eps: float, per_channel: bool = False) -> None:
        super().__init__()
        self.dim, self.eps = dim, eps
        self.weight = nn.Parameter(torch.zeros(pad8(dim) if per_channel else 1, dtype=torch.float32), requires_grad=False)
        self.weight.weight_loader = self.weight_loader

    def weight_loader(self, param: nn.Parameter, loaded_weight: torch.Tensor):
        w = loaded_weight.reshape(-1)
        param.data[:w.numel()].copy_(w)


class CausalConv(nn.Module):
    """h_t + sum_j w[:, j] h_(t - taps + 1 + j) per channel; the weight is stored [taps, padded channels]."""

    def __init__(self, dim: int, taps: int) -> None:
        super().__init__()
        self.dim, self.taps = dim, taps
        self.weight = nn.Parameter(torch.zeros(taps, pad8(dim)), requires_grad=False)
        self.weight.weight_loader = self.weight_loader

    def weight_loader(self, param: nn.Parameter, loaded_weight: torch.Tensor):
        param.data[:, :self.dim].copy_(loaded_weight.T)

    def new_state(self) -> SlotState:
        """The last taps - 1 inputs of every sequence, in the model's dtype."""
        return SlotState((self.taps - 1, pad8(self.dim)))


def _batch():
    ctx = get_context()
    return (ctx.cu_seqlens_q if ctx.is_prefill else None, ctx.context_lens, ctx.state_slots, ctx.max_seqlen_q if ctx.is_prefill else 1)


def first_input(ids: torch.Tensor, table: torch.Tensor, norm: GainNorm, conv: CausalConv | None, state: SlotState | None):
    """The residual x = table[ids] and the first sublayer's input."""
    return ops.sandwich_step(None, None, None, norm.weight, norm.eps, norm.dim, _batch(), conv.weight if conv is not None else None,
                             state.state if state is not None else None, embed=(ids, table))


def next_input(x: torch.Tensor, y: torch.Tensor, post: GainNorm, norm: GainNorm, conv: CausalConv | None, state: SlotState | None, store: bool = True):
    """x + post(y), and the next sublayer's input norm(x) with its convolution (None: the plain norm)."""
    return ops.sandwich_step(x, y, post.weight, norm.weight, norm.eps, norm.dim, _batch(), conv.weight if conv is not None else None,
                             state.state if state is not None else None, store=store)
