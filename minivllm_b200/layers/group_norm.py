"""Steps between sublayers for decoders with an fp32 residual stream, (grouped) RMS norms, a norm on one or both sides
of every sublayer and perhaps an element-wise gate on its result.  One launch each (csrc/norms.cu); bf16 or fp32
activations.  Without a norm in front of the next sublayer (`w_next` None) that sublayer reads the stream itself, rounded
to the activation type.
"""
import torch

from .. import _cabi


def _rows(t, name):
    if t.dim() != 2 or (t.shape[1] > 1 and t.stride(1) != 1):
        raise ValueError(f"{name} must be (rows, columns) with dense rows")
    return t.data_ptr(), t.stride(0)


ACTS = {"sigmoid": 0, "silu": 1, "gelu_tanh": 2, "clamped": 3, "relu": 4}      # enum mv_act


def _ptr(t):
    return t.data_ptr() if t is not None else None


def embed_norm(ids, embed, w_next, groups, eps, w_post=None):
    """Residual stream x (rows, width) fp32 from the embedding rows (their norm, with `w_post`), and its norm: (x, h)."""
    _cabi.require_cuda(ids, embed, w_next, w_post)
    rows, width = ids.numel(), embed.shape[1]
    x = torch.empty((rows, width), dtype=torch.float32, device=embed.device)
    h = torch.empty((rows, width), dtype=embed.dtype, device=embed.device)
    _cabi.check(_cabi.lib().mv_embed_norm(h.data_ptr(), x.data_ptr(), ids.data_ptr(), embed.data_ptr(), embed.shape[0],
                                          _ptr(w_post), _ptr(w_next), rows, width, groups, eps,
                                          _cabi.layer_dtype_code(embed.dtype), _cabi.stream_ptr()))
    return x, h


def gated_residual_norm(x, y, gate, gate_bias, w_post, w_next, mult, groups, eps):
    """x += mult * norm(y * sigmoid(gate + gate_bias)) * w_post in place; returns norm(x) * w_next.
    gate (rows, width) may be None."""
    _cabi.require_cuda(x, y, gate, w_post, w_next)
    rows, width = x.shape
    yp, ys = _rows(y, "y")
    gp, gs = _rows(gate, "gate") if gate is not None else (None, 0)
    out = torch.empty((rows, width), dtype=y.dtype, device=y.device)
    _cabi.check(_cabi.lib().mv_gated_residual_norm(
        out.data_ptr(), x.data_ptr(), yp, ys, gp, gs, gate_bias.data_ptr() if gate is not None else None,
        w_post.data_ptr(), _ptr(w_next), mult, rows, width, groups, eps, _cabi.layer_dtype_code(y.dtype),
        _cabi.stream_ptr()))
    return out


def pair_residual_norm(x, a, w_a, b, w_b, w_post, w_next, mult, groups, eps):
    """gated_residual_norm whose y is half the sum of norm(a) * w_a and norm(b) * w_b, without a gate."""
    _cabi.require_cuda(x, a, w_a, b, w_b, w_post, w_next)
    rows, width = x.shape
    ap, as_ = _rows(a, "a")
    bp, bs = _rows(b, "b")
    out = torch.empty((rows, width), dtype=a.dtype, device=a.device)
    _cabi.check(_cabi.lib().mv_pair_residual_norm(
        out.data_ptr(), x.data_ptr(), ap, as_, w_a.data_ptr(), bp, bs, w_b.data_ptr(), w_post.data_ptr(), _ptr(w_next),
        mult, rows, width, groups, eps, _cabi.layer_dtype_code(a.dtype), _cabi.stream_ptr()))
    return out


def moe_residual_norm(x, expert_rows, pos, top_weights, shared, shared_gate, gate, gate_bias, w_post, w_next, mult,
                      groups, eps):
    """gated_residual_norm whose y is the mixture: sum_k top_weights[t, k] * expert_rows[pos[t, k]], plus
    sigmoid(shared_gate[t]) * shared[t] (shared[t] without a gate) when there is a shared expert."""
    _cabi.require_cuda(x, expert_rows, pos, top_weights, shared, w_post, w_next)
    rows, width = x.shape
    gp, gs = _rows(gate, "gate") if gate is not None else (None, 0)
    sp, ss = _rows(shared, "shared") if shared is not None else (None, 0)
    out = torch.empty((rows, width), dtype=expert_rows.dtype, device=x.device)
    _cabi.check(_cabi.lib().mv_moe_residual_norm(
        out.data_ptr(), x.data_ptr(), expert_rows.data_ptr(), pos.data_ptr(), top_weights.data_ptr(),
        top_weights.shape[1], sp, ss, shared_gate.data_ptr() if shared_gate is not None else None,
        shared_gate.stride(0) if shared_gate is not None else 0, gp, gs,
        gate_bias.data_ptr() if gate is not None else None, w_post.data_ptr(), _ptr(w_next), mult, rows, width,
        groups, eps, _cabi.layer_dtype_code(expert_rows.dtype), _cabi.stream_ptr()))
    return out


def gated_group_norm(y, z, weight, groups, eps):
    """norm(y * silu(z)) * weight, rows in `groups` runs of channels."""
    _cabi.require_cuda(y, z, weight)
    yp, ys = _rows(y, "y")
    zp, zs = _rows(z, "z")
    out = torch.empty(y.shape, dtype=y.dtype, device=y.device)
    _cabi.check(_cabi.lib().mv_gated_group_norm(out.data_ptr(), yp, ys, zp, zs, weight.data_ptr(), y.shape[0],
                                                y.shape[1], groups, eps, _cabi.layer_dtype_code(y.dtype),
                                                _cabi.stream_ptr()))
    return out


def head_norm_gate(y, z, weight, heads, eps, out=None, den=None, act="silu", mult=1.0):
    """norm(y / den) * weight * act(z) * mult, rows in `heads` runs of channels; den (rows, heads) fp32 or None; weight has one
    run's length, or a row's; act silu or sigmoid; out may have any row stride."""
    _cabi.require_cuda(y, z, weight, den)
    yp, ys = _rows(y, "y")
    zp, zs = _rows(z, "z")
    if out is None:
        out = torch.empty(y.shape, dtype=y.dtype, device=y.device)
    full = weight.numel() == y.shape[1]
    if not full and weight.numel() * heads != y.shape[1]:
        raise ValueError("the norm's weight has neither a head's nor a row's length")
    _cabi.check(_cabi.lib().mv_head_norm_gate(
        *_rows(out, "out"), yp, ys, _ptr(den), zp, zs, weight.data_ptr(), int(full), ACTS[act], mult, y.shape[0], y.shape[1], heads, eps,
        _cabi.layer_dtype_code(y.dtype), _cabi.stream_ptr()))
    return out


def gate_mul(y, gate, act="sigmoid", out=None, limit=0.0):
    """A gate applied to y: y * act(gate) for sigmoid, silu, gelu_tanh and relu; "clamped" with `limit` see enum mv_act.  y (rows, cols), or (rows, heads, cols / heads) with any row and head
    stride; gate (rows, cols).  Returns (rows, cols)."""
    _cabi.require_cuda(y, gate)
    rows, cols = gate.shape
    if y.dim() == 3:
        heads, row_stride, head_stride = y.shape[1], y.stride(0), y.stride(1)
        if y.stride(2) != 1 and y.shape[2] > 1:
            raise ValueError("y must have dense pieces")
    else:
        heads, head_stride = 1, 0
        row_stride = _rows(y, "y")[1]
    if out is None:
        out = torch.empty((rows, cols), dtype=y.dtype, device=y.device)
    gp, gs = _rows(gate, "gate")
    _cabi.check(_cabi.lib().mv_gate_mul(out.data_ptr(), y.data_ptr(), row_stride, head_stride, heads, gp, gs,
                                        ACTS[act], limit, rows, cols, _cabi.layer_dtype_code(y.dtype),
                                        _cabi.stream_ptr()))
    return out
