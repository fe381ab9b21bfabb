"""SiLU(gate) * up as one CUDA kernel (nanovllm/layers/activation.py:6-11), and PolyNorm."""
import torch
from torch import nn

from .. import ops


class SiluAndMul(nn.Module):

    def forward(self, x):
        return ops.silu_and_mul(x)


class PolyNorm(nn.Module):
    """a N(z) + b N(z^2) + c N(z^3) + e with learned a, b, c, e; N divides a row of `dim` values by its root mean square."""

    def __init__(self, dim: int, eps: float) -> None:
        super().__init__()
        self.dim, self.eps = dim, eps
        self.coef = nn.Parameter(torch.zeros(4, dtype=torch.float32), requires_grad=False)

    def forward(self, z: torch.Tensor) -> torch.Tensor:
        return ops.poly_norm(z, self.coef, self.eps, self.dim)
