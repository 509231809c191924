"""SiluAndMul on the F3 kernel (reference: layers/activation.py:6-13), and the dense feed-forward with a clamped
gated unit and the one with act(gate) * up that several of the listed-layer decoders share."""
import torch
from torch import nn

from .. import ops
from .linear import MergedColumnParallelLinear, PaddedMergedLinear, RowParallelLinear


class SiluAndMul(nn.Module):

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        return ops.silu_and_mul(x)


class ClampedGatedFeedForward(nn.Module):
    """W_down(g sigmoid(alpha g) (u + 1)), g = min(W_gate h, limit), u = clamp(W_up h, -limit, limit)."""

    def __init__(self, width: int, ff: int, limit: float, alpha: float = 1.702):
        super().__init__()
        self.limit, self.alpha = float(limit), float(alpha)
        self.gate_up_proj = MergedColumnParallelLinear(width, [ff, ff])
        self.down_proj = RowParallelLinear(ff, width)

    def forward(self, h):
        return self.down_proj(ops.glu_clamped(self.gate_up_proj(h), self.alpha, self.limit))


class GatedFeedForward(nn.Module):
    """W_down(act(W_gate h) * W_up h) on the kernels that take any size and 16- or 32-bit elements; act: silu, relu or
    gelu_tanh. ``extra`` columns (with a bias) that read the same input are computed in the same product: ``forward``
    then returns them too."""

    def __init__(self, width: int, ff: int, act: str = "silu", extra: int = 0):
        super().__init__()
        self.act, self.extra = act, int(extra)
        self.gate_up_proj = (PaddedMergedLinear(width, [[ff, ff], extra], bias=True) if extra else
                             MergedColumnParallelLinear(width, [ff, ff]))
        self.down_proj = RowParallelLinear(ff, width)

    def forward(self, h):
        p = self.gate_up_proj(h)
        if not self.extra:
            return self.down_proj(ops.act_and_mul(p, self.act))
        return self.down_proj(ops.act_and_mul(self.gate_up_proj.part(p, 0), self.act)), self.gate_up_proj.part(p, 1)
