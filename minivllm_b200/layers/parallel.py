"""Two mixers side by side on the same input.  ParallelMixers: one stacked product for both; each result has a norm of its own,
which the residual step applies when it adds half their sum (pair_residual_norm).  ScaledMixers: their sum with constant
factors, one output product for both.
"""
import torch
import torch.nn as nn
import torch.nn.functional as F

from .linear import StackedLinear


class ParallelMixers(nn.Module):
    def __init__(self, m, width, eps, load, left, right):
        """left, right: mixer classes with `parts`, perhaps `biases`, and `mix`."""
        super().__init__()
        self.left = left(m["left"], width, eps, load.scoped("left."), stack=False)
        self.right = right(m["right"], width, eps, load.scoped("right."), stack=False)
        parts, biases = {}, {}
        for side, mixer in (("left.", self.left), ("right.", self.right)):
            parts.update({side + n: w for n, w in mixer.parts.items()})
            biases.update({side + n: b for n, b in (getattr(mixer, "biases", None) or {}).items()})
            mixer.parts = mixer.biases = None
        self.stacked = StackedLinear(parts, biases)
        param = lambda t: nn.Parameter(t, requires_grad=False)
        self.left_out, self.right_out = param(load("left.out", (width,))), param(load("right.out", (width,)))

    def forward(self, h):
        """h (tokens, width) -> the two results, (tokens, width) each, before their norms."""
        p = self.stacked(h)
        side = lambda name: {n[len(name):]: t for n, t in p.items() if n.startswith(name)}
        return self.left.mix(side("left.")), self.right.mix(side("right."))


class ScaledMixers(nn.Module):
    """left, right: mixer classes with `columns`, `o_w`, `shift` and `results`.  The factors are applied to the heads' results in
    32-bit, before these are rounded for the output product, which sums over both mixers' columns."""

    def __init__(self, m, width, eps, load, left, right):
        super().__init__()
        self.scales = float(m["left_scale"]), float(m["right_scale"])
        self.left = left(m["left"], width, eps, load.scoped("left."))
        self.right = right(m["right"], width, eps, load.scoped("right."))
        self.at = self.left.columns
        self.shift = self.left.shift or self.right.shift        # of the entry in front
        self.o_w = nn.Parameter(torch.cat([self.left.o_w, self.right.o_w], dim=1), requires_grad=False)
        self.left.o_w = self.right.o_w = None

    def forward(self, inputs):
        """inputs: what the entry in front gives -> (tokens, width)."""
        h = inputs[0] if isinstance(inputs, tuple) else inputs
        o = torch.empty((h.shape[0], self.o_w.shape[1]), dtype=h.dtype, device=h.device)
        self.left.results(inputs, o[:, :self.at], self.scales[0])
        self.right.results(inputs, o[:, self.at:], self.scales[1])
        return F.linear(o, self.o_w)
