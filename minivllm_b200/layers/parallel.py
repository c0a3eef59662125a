"""Two mixers side by side on the same input, one stacked product for both; each result has a norm of its own, which the
residual step applies when it adds half their sum (pair_residual_norm).
"""
import torch.nn as nn

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
