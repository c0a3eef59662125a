"""Several residual streams instead of one (hyper-connections), and the convolution over time that may stand in front of a
mixer (csrc/streams.cu, csrc/short_conv.cu).

A sublayer reads a weighted sum of the fp32 streams through a norm; its result enters all streams, which mix with one
another at the same time.  The update behind one sublayer and the sum and norm in front of the next are one launch, and for
sequences with one token so is the convolution.
"""
import torch
import torch.nn as nn

from .. import _cabi
from ..utils.context import get_context
from .short_conv import conv_add, conv_state_update


class InputConvolution(nn.Module):
    """h_t + sum_j weight[:, j] h_(t - taps + 1 + j); the last taps - 1 inputs are kept per sequence."""

    def __init__(self, weight):
        super().__init__()
        self.width, self.taps = weight.shape
        self.weight = nn.Parameter(weight, requires_grad=False)
        self.weight_t = nn.Parameter(weight.t().contiguous(), requires_grad=False)
        self.slot_state = None          # assigned by the model runner

    def slot_state_spec(self, dtype):
        """Per-sequence state: name -> (shape, dtype)."""
        return {"h": ((self.taps - 1, self.width), dtype)}


class StreamEntry(nn.Module):
    """What stands in front of a sublayer: weights of the streams (None: their sum), a norm, perhaps a convolution."""

    def __init__(self, w_in, norm_w, norm_b, eps, conv=None):
        super().__init__()
        param = lambda t: nn.Parameter(t, requires_grad=False) if t is not None else None
        self.w_in, self.norm_w, self.norm_b, self.eps, self.conv = param(w_in), param(norm_w), param(norm_b), eps, conv


def _launch(x, entry, dtype, ids=None, embed=None, y=None, mix=None, w_out=None):
    _cabi.require_cuda(x, ids, embed, y, mix, w_out, entry.norm_w)
    rows, streams, width = x.shape
    conv, ctx = entry.conv, get_context()
    nd = rows if conv is None else min(ctx.num_decode, rows)
    out = torch.empty((rows, width), dtype=dtype, device=x.device)
    raw = torch.empty((rows - nd, width), dtype=dtype, device=x.device) if nd < rows else None
    ptr = lambda t: t.data_ptr() if t is not None else None
    kept = conv.slot_state["h"] if conv is not None else None
    if y is not None and y.stride(1) != 1 and width > 1:
        raise ValueError("y must have dense rows")
    _cabi.check(_cabi.lib().mv_stream_step(
        out.data_ptr(), ptr(raw), x.data_ptr(), ptr(ids), ptr(embed), embed.shape[0] if embed is not None else 0, ptr(y),
        y.stride(0) if y is not None else 0, ptr(mix), ptr(w_out), ptr(entry.w_in), ptr(entry.norm_w), ptr(entry.norm_b),
        ptr(conv.weight_t) if conv is not None else None, conv.taps if conv is not None else 0, ptr(kept),
        ptr(ctx.state_slots) if conv is not None else None, ptr(ctx.state_starts) if conv is not None else None,
        kept.shape[0] if conv is not None else 0, nd, rows, width, streams, entry.eps, _cabi.layer_dtype_code(dtype),
        _cabi.stream_ptr()))
    if raw is not None:                  # portions: the convolution needs their neighbours
        cu, slots, starts = ctx.portion_cu_q, ctx.state_slots[nd:], ctx.state_starts[nd:]
        conv_add(raw, conv.weight, None, cu, slots, starts, kept, out=out[nd:])
        conv_state_update(kept, raw, conv.taps, cu, slots, starts)
    return out


def stream_embed(ids, embed, streams, entry):
    """Streams x (rows, streams, width) fp32, each the embedding row, and the first sublayer's input: (x, h)."""
    x = torch.empty((ids.numel(), streams, embed.shape[1]), dtype=torch.float32, device=embed.device)
    return x, _launch(x, entry, embed.dtype, ids=ids, embed=embed)


def stream_step(x, y, mix, w_out, entry):
    """A sublayer's result y enters the streams x (in place): x_t = sum_s mix[s, t] x_s + w_out[t] y.  Returns the input of
    what `entry` stands in front of."""
    return _launch(x, entry, y.dtype, y=y, mix=mix, w_out=w_out)
