"""Several linear layers that read the same input as one matrix product.

The weights are stacked along their output rows; every part starts at a multiple of eight columns of the result, so
that kernels may read it in 16-byte pieces.  `router_logits` is the one product whose result is wanted in fp32.
"""
import torch
import torch.nn as nn
import torch.nn.functional as F


class StackedLinear(nn.Module):
    """parts: {name: (out, in) weight}, biases: {name: (out,)} for some of them.  Calling it with (rows, in) returns
    {name: (rows, out) view}."""

    def __init__(self, parts, biases=None):
        super().__init__()
        rows, self.spans, at = [], {}, 0
        for name, w in parts.items():
            n = w.shape[0]
            self.spans[name] = (at, at + n)
            pad = -n % 8
            rows.append(w)
            if pad:
                rows.append(w.new_zeros(pad, w.shape[1]))
            at += n + pad
        self.weight = nn.Parameter(torch.cat(rows) if len(rows) > 1 else rows[0], requires_grad=False)
        self.bias = None
        if biases:
            b = self.weight.new_zeros(at)
            for name, t in biases.items():
                b[self.spans[name][0]:self.spans[name][1]] = t
            self.bias = nn.Parameter(b, requires_grad=False)

    def forward(self, h):
        y = F.linear(h, self.weight, self.bias)
        return {name: y[:, a:b] for name, (a, b) in self.spans.items()}


def router_logits(h, weight):
    """(rows, in) x (experts, in) -> fp32 (rows, experts), products accumulated and kept in fp32."""
    if h.dtype == torch.float32:
        return F.linear(h, weight)
    return torch.mm(h, weight.t(), out_dtype=torch.float32)
