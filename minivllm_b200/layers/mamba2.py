"""State-space mixer (Mamba-2 / SSD): stacked input projection, causal depthwise convolution with silu, the
selective recurrence, gated group norm and output projection (csrc/mamba2.cu).

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


def conv_silu(u, weight, bias, cu, slots, starts, state):
    """u (tokens, channels) any row stride -> (tokens, channels); see mv_conv_silu."""
    _cabi.require_cuda(u, weight, slots, starts)
    tokens, channels = u.shape
    out = torch.empty((tokens, channels), dtype=u.dtype, device=u.device)
    _cabi.check(_cabi.lib().mv_conv_silu(
        out.data_ptr(), u.data_ptr(), u.stride(0), weight.data_ptr(), bias.data_ptr(), weight.shape[1], channels,
        cu.data_ptr() if cu is not None else None, slots.numel(), tokens, slots.data_ptr(), starts.data_ptr(),
        state.data_ptr(), state.shape[0], _cabi.layer_dtype_code(u.dtype), _cabi.stream_ptr()))
    return out


def conv_state_update(state, u, taps, cu, slots, starts):
    _cabi.check(_cabi.lib().mv_conv_state_update(
        state.data_ptr(), u.data_ptr(), u.stride(0), taps, u.shape[1], cu.data_ptr() if cu is not None else None,
        slots.numel(), slots.data_ptr(), starts.data_ptr(), state.shape[0], _cabi.layer_dtype_code(u.dtype),
        _cabi.stream_ptr()))


def ssm_scan(xbc, dt, dt_bias, A_log, D, cu, slots, starts, state, heads, vdim, state_dim, groups):
    """xbc (tokens, heads*vdim + 2*groups*state_dim) contiguous, dt (tokens, heads); returns y (tokens, heads*vdim)
    and advances `state` (slots, heads, state_dim, vdim) fp32."""
    _cabi.require_cuda(xbc, dt, state)
    y = torch.empty((xbc.shape[0], heads * vdim), dtype=xbc.dtype, device=xbc.device)
    _cabi.check(_cabi.lib().mv_ssm_scan(
        y.data_ptr(), xbc.data_ptr(), dt.data_ptr(), dt.stride(0), dt_bias.data_ptr(), A_log.data_ptr(), D.data_ptr(),
        cu.data_ptr() if cu is not None else None, slots.numel(), slots.data_ptr(), starts.data_ptr(),
        state.data_ptr(), state.shape[0], heads, vdim, state_dim, groups, _cabi.layer_dtype_code(xbc.dtype),
        _cabi.stream_ptr()))
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
        cu, slots, starts = ctx.cu_seqlens_q, ctx.state_slots, ctx.state_starts
        conv, ssm = self.slot_state["conv"], self.slot_state["ssm"]
        xbc = conv_silu(p["xbc"], self.conv_w, self.conv_b, cu, slots, starts, conv)
        y = ssm_scan(xbc, p["dt"], self.dt_bias, self.A_log, self.D, cu, slots, starts, ssm, self.heads, self.vdim,
                     self.state, self.groups)
        conv_state_update(conv, p["xbc"], self.taps, cu, slots, starts)
        y = gated_group_norm(y, p["z"], self.norm_w, self.norm_groups, self.eps)
        return F.linear(y, self.o_w), p
