"""Element-wise norm (Dynamic Tanh) between the sublayers of a decoder with an fp32 residual stream, and the mixtures of a
token's input with the one before it that some mixers read (csrc/tanh_norm.cu).

The addition of a sublayer's result and the norm in front of the next sublayer are one launch, which also makes the mixtures.
"""
import torch
import torch.nn as nn

from .. import _cabi
from ..utils.context import get_context
from .short_conv import conv_state_update


class TokenShift(nn.Module):
    """mu (mixtures, width): h + (h' - h) mu[m], h' the input of the token before; the last input is kept per sequence."""

    def __init__(self, mu):
        super().__init__()
        self.mu = nn.Parameter(mu, requires_grad=False)
        self.slot_state = None          # assigned by the model runner

    def slot_state_spec(self, dtype):
        """Per-sequence state: name -> (shape, dtype)."""
        return {"h": ((self.mu.shape[1],), dtype)}


class TanhEntry(nn.Module):
    """What stands in front of a sublayer: tanh(alpha x) w + b, perhaps with mixtures."""

    def __init__(self, alpha, w, b, shift=None):
        super().__init__()
        self.alpha, self.shift = float(alpha), shift
        self.w, self.b = nn.Parameter(w, requires_grad=False), nn.Parameter(b, requires_grad=False)


def position_frequencies(width, device, base=10000.0):
    """base^(-2i / width) in double, of the sinusoids in columns 2i and 2i + 1."""
    return torch.tensor([base ** (-2.0 * i / width) for i in range((width + 1) // 2)], dtype=torch.float64, device=device)


def _launch(entry, rows, dtype, device, x=None, y=None, experts=None, ids=None, embed=None, inv_freq=None):
    _cabi.require_cuda(x, y, ids, embed, entry.w)
    ctx, shift, width = get_context(), entry.shift, entry.w.numel()
    new = x
    if x is None or shift is not None:          # rows are read again by their neighbours
        new = torch.empty((rows, width), dtype=torch.float32, device=device)
    out = torch.empty((rows, width), dtype=dtype, device=device)
    mixed = kept = cu = slots = starts = None
    if shift is not None:
        mixed = torch.empty((shift.mu.shape[0], rows, width), dtype=dtype, device=device)
        kept, cu, slots, starts = shift.slot_state["h"], ctx.cu_seqlens_q, ctx.state_slots, ctx.state_starts
    pos = weights = None
    if experts is not None:
        y, pos, weights = experts
    if y is not None and y.stride(1) != 1 and width > 1:
        raise ValueError("y must have dense rows")
    ptr = lambda t: t.data_ptr() if t is not None else None
    _cabi.check(_cabi.lib().mv_tanh_step(
        out.data_ptr(), new.data_ptr(), ptr(x), ptr(ids), ptr(embed), embed.shape[0] if embed is not None else 0,
        ptr(ctx.positions), ptr(inv_freq), ptr(y), y.stride(0) if y is not None else 0, ptr(pos), ptr(weights),
        weights.shape[1] if weights is not None else 0, entry.alpha, entry.w.data_ptr(), entry.b.data_ptr(), ptr(mixed),
        ptr(shift.mu) if shift is not None else None, mixed.shape[0] if mixed is not None else 0, ptr(kept), ptr(slots),
        ptr(starts), kept.shape[0] if kept is not None else 0, ptr(cu), slots.numel() if slots is not None else 0, rows, width,
        _cabi.layer_dtype_code(dtype), _cabi.stream_ptr()))
    if shift is not None:
        nd = min(ctx.num_decode, rows)
        if nd < rows:
            conv_state_update(kept, out[nd:], 2, ctx.portion_cu_q, slots[nd:], starts[nd:])
        return new, (out, mixed)
    return new, out


def tanh_embed(ids, embed, entry, inv_freq=None):
    """Residual stream x (rows, width) fp32 from the embedding rows, with the sinusoids of the positions when `inv_freq` is
    given, and the first sublayer's input: (x, h), or (x, (h, mixtures)) with a shift."""
    return _launch(entry, ids.numel(), embed.dtype, embed.device, ids=ids, embed=embed, inv_freq=inv_freq)


def tanh_step(x, y, entry):
    """Adds y, a sublayer's result (rows, width) or (expert rows, pos, weights), to x.  Returns the new stream (x itself
    without a shift) and the input of what `entry` stands in front of."""
    experts = y if isinstance(y, tuple) else None
    return _launch(entry, x.shape[0], entry.w.dtype, x.device, x=x, y=None if experts else y, experts=experts)
