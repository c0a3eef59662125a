"""State-space mixer (Mamba-2 / SSD): stacked input projection, causal depthwise convolution with silu, the
selective recurrence, gated group norm and output projection (csrc/mamba2.cu, csrc/short_conv.cu).

The per-sequence state (last convolution inputs, fp32 recurrent state) lives in slots assigned by the engine; the
model runner allocates what `slot_state_spec` describes and fills `slot_state`.
"""
import torch
import torch.nn as nn
import torch.nn.functional as F

from .. import _cabi
from ..utils.context import get_context
from .group_norm import gated_group_norm
from .linear import StackedLinear
from .short_conv import conv_silu, conv_state_update


def ssm_scan(xbc, dt, dt_bias, A_log, D, cu, slots, starts, state, heads, vdim, state_dim, groups, out=None,
             chunked=None):
    """xbc (tokens, heads*vdim + 2*groups*state_dim) contiguous, dt (tokens, heads); returns y (tokens, heads*vdim)
    and advances `state` (slots, heads, state_dim, vdim) fp32.  bf16 takes the chunked tensor-core kernel when it has
    the sizes."""
    _cabi.require_cuda(xbc, dt, state)
    L = _cabi.lib()
    y = torch.empty((xbc.shape[0], heads * vdim), dtype=xbc.dtype, device=xbc.device) if out is None else out
    if chunked is None:
        chunked = xbc.dtype == torch.bfloat16 and cu is not None and bool(L.mv_ssm_chunk_takes(vdim, state_dim))
    if chunked:
        _cabi.check(L.mv_ssm_chunk_scan(
            y.data_ptr(), y.stride(0), xbc.data_ptr(), xbc.stride(0), dt.data_ptr(), dt.stride(0), dt_bias.data_ptr(),
            A_log.data_ptr(), D.data_ptr(), cu.data_ptr(), slots.numel(), slots.data_ptr(), starts.data_ptr(),
            state.data_ptr(), state.shape[0], heads, vdim, state_dim, groups, _cabi.stream_ptr()))
        return y
    _cabi.check(L.mv_ssm_scan(
        y.data_ptr(), xbc.data_ptr(), dt.data_ptr(), dt.stride(0), dt_bias.data_ptr(), A_log.data_ptr(), D.data_ptr(),
        cu.data_ptr() if cu is not None else None, slots.numel(), slots.data_ptr(), starts.data_ptr(),
        state.data_ptr(), state.shape[0], heads, vdim, state_dim, groups, _cabi.layer_dtype_code(xbc.dtype),
        _cabi.stream_ptr()))
    return y


def ssm_step(u, conv_w, conv_b, conv_state, dt, dt_bias, A_log, D, slots, starts, state, heads, vdim, state_dim,
             groups, out=None):
    """One token per sequence: convolution (conv_state is only read) and one step of the recurrence."""
    _cabi.require_cuda(u, dt, state)
    y = torch.empty((u.shape[0], heads * vdim), dtype=u.dtype, device=u.device) if out is None else out
    _cabi.check(_cabi.lib().mv_ssm_step(
        y.data_ptr(), u.data_ptr(), u.stride(0), conv_w.data_ptr(), conv_b.data_ptr(), conv_w.shape[1],
        conv_state.data_ptr(), dt.data_ptr(), dt.stride(0), dt_bias.data_ptr(), A_log.data_ptr(), D.data_ptr(),
        slots.numel(), slots.data_ptr(), starts.data_ptr(), state.data_ptr(), state.shape[0], heads, vdim, state_dim,
        groups, _cabi.layer_dtype_code(u.dtype), _cabi.stream_ptr()))
    return y


class Mamba2(nn.Module):
    def __init__(self, m, width, eps, load, extra=None):
        super().__init__()
        self.heads, self.vdim, self.state, self.groups = m["heads"], m["vdim"], m["state"], m["groups"]
        self.norm_groups, self.taps, self.eps = m["norm_groups"], m["conv"], eps
        if self.heads % self.groups or (self.heads * self.vdim) % self.norm_groups:
            raise ValueError("mamba2: heads must divide by groups, and their width by norm_groups")
        inner, gn = self.heads * self.vdim, self.groups * self.state
        self.inner, self.channels = inner, inner + 2 * gn
        w_in = load("in", (inner + self.channels + self.heads, width))
        z, xbc, dt = w_in.split([inner, self.channels, self.heads])
        self.stacked = StackedLinear({"z": z, "xbc": xbc, "dt": dt, **(extra or {})})
        param = lambda t: nn.Parameter(t, requires_grad=False)
        self.conv_w, self.conv_b = param(load("conv", (self.channels, self.taps))), param(load("conv.b", (self.channels,)))
        self.dt_bias, self.A_log, self.D = (param(load(n, (self.heads,))) for n in ("dt_bias", "A_log", "D"))
        self.norm_w, self.o_w = param(load("norm", (inner,))), param(load("o", (width, inner)))
        self.slot_state = None          # assigned by the model runner

    def slot_state_spec(self, dtype):
        """Per-sequence state: name -> (shape, dtype)."""
        return {"conv": ((self.taps - 1, self.channels), dtype),
                "ssm": ((self.heads, self.state, self.vdim), torch.float32)}

    def forward(self, h):
        """h (tokens, width) -> (mixer output (tokens, width), {extra parts of the stacked projection})."""
        ctx = get_context()
        p = self.stacked(h)
        slots, starts, nd = ctx.state_slots, ctx.state_starts, ctx.num_decode
        conv, ssm = self.slot_state["conv"], self.slot_state["ssm"]
        u, dt = p["xbc"], p["dt"]
        y = torch.empty((h.shape[0], self.inner), dtype=h.dtype, device=h.device)
        if nd:                           # sequences with one token come first
            w = (self.conv_w, self.conv_b)
            par = (self.dt_bias, self.A_log, self.D)
            dims = (self.heads, self.vdim, self.state, self.groups)
            if self.vdim % 4 == 0 and self.state % 4 == 0:
                ssm_step(u[:nd], *w, conv, dt[:nd], *par, slots[:nd], starts[:nd], ssm, *dims, out=y[:nd])
            else:
                xbc = conv_silu(u[:nd], *w, None, slots[:nd], starts[:nd], conv)
                ssm_scan(xbc, dt[:nd], *par, None, slots[:nd], starts[:nd], ssm, *dims, out=y[:nd])
        if h.shape[0] > nd:
            cu = ctx.portion_cu_q
            xbc = conv_silu(u[nd:], self.conv_w, self.conv_b, cu, slots[nd:], starts[nd:], conv)
            ssm_scan(xbc, dt[nd:], self.dt_bias, self.A_log, self.D, cu, slots[nd:], starts[nd:], ssm, self.heads,
                     self.vdim, self.state, self.groups, out=y[nd:])
        conv_state_update(conv, u, self.taps, ctx.cu_seqlens_q, slots, starts)
        y = gated_group_norm(y, p["z"], self.norm_w, self.norm_groups, self.eps)
        return F.linear(y, self.o_w), p
