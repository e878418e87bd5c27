"""The projection in front of a pass of looped layers: x <- W [x; x0] + step, with x the 32-bit residual stream, x0 the token's
embedding and ``step`` a vector of the pass.

In bfloat16 the stream enters as two bfloat16 numbers (hi + lo = x to 16 mantissa bits) against the same columns of W, and the
product leaves as floats, so the pass does not round the stream to 8 bits; x0 is a row of the bfloat16 table, exact as it is.
The operand comes from the residual launch in front of the pass (``nat.tanh_residual`` with ``want_cat``), the vector of the pass
is the GEMM's bias."""
import torch
from torch import nn

from .linear import linear_float


class PassInput(nn.Module):
    def __init__(self, width: int, times: int):
        super().__init__()
        self.width = width
        # columns of W for [hi | lo | x0] in bfloat16, [x | x0] in float32: filled by `load`
        parts = 3 if torch.get_default_dtype() == torch.bfloat16 else 2
        self.weight = nn.Parameter(torch.empty(width, parts * width), requires_grad=False)
        self.step = nn.Parameter(torch.zeros(times, width), requires_grad=False)

    def expand(self, w: torch.Tensor) -> torch.Tensor:
        """A checkpoint's [width, 2 width] tensor -> the weight's columns."""
        if tuple(w.shape) != (self.width, 2 * self.width):
            raise ValueError(f"pass input projection of shape {tuple(w.shape)}, expected {(self.width, 2 * self.width)}")
        return torch.cat([w[:, :self.width], w], 1) if self.weight.shape[1] == 3 * self.width else w

    def forward(self, x: torch.Tensor, cat: torch.Tensor, t: int) -> torch.Tensor:
        """x [n, width] float, overwritten by the pass's start; cat [n, 3 width | 2 width] its operand."""
        return linear_float(cat, self.weight, self.step[t], out=x)
