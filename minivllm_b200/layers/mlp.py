"""Dense gated feed-forward: one stacked product for gate and up, the activation in one launch, the down product."""
import torch.nn as nn
import torch.nn.functional as F

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
