"""Linear attention with a constant decay per head ("lightning attention") and its gated output norm."""
from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..utils.context import get_context
from .linear import HeadsLinear, MergeHeadsLinear, pad8
from .state import SlotState

DECAY_POWERS = 65  # decay^0 .. decay^64: one chunk of the prefill kernel


class RecurrentState(SlotState):
    """One layer run's state [slots, heads, qk_pad, v_pad] in fp32."""

    def __init__(self, heads: int, qk_pad: int, v_pad: int):
        super().__init__((heads, qk_pad, v_pad), torch.float32)


class DecayedLinearAttention(nn.Module):
    """S <- decay S + k v^T, o = S^T q with q, k, v = silu(projection); the concatenated heads are RMS-normed, gated by
    sigmoid(W_g x) and projected."""

    def __init__(self, hidden_size: int, heads: int, dim: int, vdim: int, decay: list[float], eps: float) -> None:
        super().__init__()
        if len(decay) != heads:
            raise ValueError(f"{len(decay)} decay values for {heads} heads")
        self.heads, self.dim, self.vdim, self.eps = heads, dim, vdim, eps
        self.qk_pad, self.v_pad = pad8(dim), pad8(vdim)
        self.in_proj = HeadsLinear(hidden_size, [(heads, dim), (heads, dim), (heads, vdim), (heads, vdim)], silu_sections=3)
        self.o_proj = MergeHeadsLinear(heads, vdim, hidden_size)
        self.norm_weight = nn.Parameter(torch.zeros(heads * self.v_pad, dtype=torch.float32), requires_grad=False)
        self.norm_weight.weight_loader = self._load_norm
        d = torch.tensor(decay, dtype=torch.float64, device="cpu")
        powers = d.unsqueeze(1) ** torch.arange(DECAY_POWERS, dtype=torch.float64, device="cpu")
        self.register_buffer("decay", d.float().to(self.norm_weight.device), persistent=False)
        self.register_buffer("decay_powers", powers.float().contiguous().to(self.norm_weight.device), persistent=False)

    def _load_norm(self, param: nn.Parameter, loaded_weight: torch.Tensor):
        param.data.view(self.heads, self.v_pad)[:, :self.vdim].copy_(loaded_weight.view(self.heads, self.vdim))

    def forward(self, x: torch.Tensor, cache: RecurrentState) -> torch.Tensor:
        ctx = get_context()
        p = self.in_proj(x)
        o = ops.linear_attn(p, self.heads, self.qk_pad, self.v_pad, cache.state, ctx.state_slots, ctx.cu_seqlens_q if ctx.is_prefill else None,
                            ctx.context_lens, ctx.max_seqlen_q if ctx.is_prefill else 1, self.decay, self.decay_powers)
        return self.o_proj(ops.gated_norm(o, p[:, -self.heads * self.v_pad:], self.norm_weight, self.eps, self.heads * self.vdim))
