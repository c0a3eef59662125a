"""Short causal depthwise convolution, followed by silu or added to its own input, its last inputs kept per sequence
(csrc/short_conv.cu)."""
import torch

from .. import _cabi


def _conv(entry, u, weight, bias, cu, slots, starts, state, out):
    _cabi.require_cuda(u, weight, slots, starts)
    tokens, channels = u.shape
    if out is None:
        out = torch.empty((tokens, channels), dtype=u.dtype, device=u.device)
    _cabi.check(getattr(_cabi.lib(), entry)(
        out.data_ptr(), u.data_ptr(), u.stride(0), weight.data_ptr(),
        bias.data_ptr() if bias is not None else None, weight.shape[1], channels,
        cu.data_ptr() if cu is not None else None, slots.numel(), tokens, slots.data_ptr(), starts.data_ptr(),
        state.data_ptr(), state.shape[0], _cabi.layer_dtype_code(u.dtype), _cabi.stream_ptr()))
    return out


def conv_silu(u, weight, bias, cu, slots, starts, state, out=None):
    """silu of the convolution of u (tokens, channels; any row stride) -> (tokens, channels); see mv_conv_silu.  bias may be
    None."""
    return _conv("mv_conv_silu", u, weight, bias, cu, slots, starts, state, out)


def conv_add(u, weight, bias, cu, slots, starts, state, out=None):
    """u plus its convolution."""
    return _conv("mv_conv_add", u, weight, bias, cu, slots, starts, state, out)


def conv_state_update(state, u, taps, cu, slots, starts):
    _cabi.check(_cabi.lib().mv_conv_state_update(
        state.data_ptr(), u.data_ptr(), u.stride(0), taps, u.shape[1], cu.data_ptr() if cu is not None else None,
        slots.numel(), slots.data_ptr(), starts.data_ptr(), state.shape[0], _cabi.layer_dtype_code(u.dtype),
        _cabi.stream_ptr()))
