"""Dense feed-forwards: gated, with one stacked product for gate and up, or ungated with an activation of learned shape; the
activation in one launch, the down product."""
import torch
import torch.nn as nn
import torch.nn.functional as F

from .. import _cabi
from .group_norm import gate_mul
from .linear import StackedLinear


class GatedMLP(nn.Module):
    def __init__(self, spec, width, load, act):
        super().__init__()
        ff = spec["ff"]
        self.act = act
        self.stacked = StackedLinear({"gate": load("gate", (ff, width)), "up": load("up", (ff, width))})
        self.down_w = nn.Parameter(load("down", (width, ff)), requires_grad=False)

    def forward(self, h):
        p = self.stacked(h)
        return F.linear(gate_mul(p["up"], p["gate"], self.act), self.down_w)


def xielu(z, a, b):
    """a z^2 + z / 2 for z > 0, else b (e^z - 1 - z) + z / 2; z (rows, cols), any row stride."""
    _cabi.require_cuda(z)
    out = torch.empty(z.shape, dtype=z.dtype, device=z.device)
    _cabi.check(_cabi.lib().mv_xielu(out.data_ptr(), z.data_ptr(), z.stride(0), a, b, z.shape[0], z.shape[1],
                                     _cabi.layer_dtype_code(z.dtype), _cabi.stream_ptr()))
    return out


class XieluMLP(nn.Module):
    """down(xielu(up h)); the activation's two numbers are softplus(p) and 1/2 + softplus(q) of the tensor 'act'."""

    def __init__(self, spec, width, load):
        super().__init__()
        ff = spec["ff"]
        self.up_w = nn.Parameter(load("up", (ff, width)), requires_grad=False)
        self.down_w = nn.Parameter(load("down", (width, ff)), requires_grad=False)
        p, q = F.softplus(load("act", (2,)).float()).tolist()
        self.a, self.b = p, 0.5 + q

    def forward(self, h):
        return F.linear(xielu(F.linear(h, self.up_w), self.a, self.b), self.down_w)
