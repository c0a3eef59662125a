"""Gated delta rule: short convolutions on q, k and v, unit-length q and k per head, a scalar decay and a step size per
head, the recurrence on a matrix state in 32-bit, a norm per head and an output gate (csrc/gated_delta.cu; portions of
prompts in chunks on tensor cores, csrc/gated_delta_chunk.cu).
"""
import torch
import torch.nn as nn
import torch.nn.functional as F

from .. import _cabi
from ..utils.context import get_context
from .gla import CHUNK_FROM
from .group_norm import head_norm_gate
from .linear import StackedLinear
from .short_conv import conv_silu, conv_state_update


def delta_scan(qkv, beta, a, A_log, dt_bias, cu, slots, starts, state, heads, kv_heads, dim, vdim, conv_w=None,
               conv_state=None, gate=None, norm_w=None, eps=0.0, out=None, chunked=None):
    """qkv (tokens, 2 * kv_heads * dim + heads * vdim), beta and a (tokens, heads) with one row stride.  Advances `state`
    (slots, heads, dim, vdim) fp32 and returns (tokens, heads * vdim): the read-outs of packed portions (cu; qkv after
    its convolution), or with cu None (one token per sequence) the normed and gated rows, the convolution included
    (conv_state is only read).  See mv_delta_scan.  bf16 portions take the chunked kernels when those have the sizes."""
    _cabi.require_cuda(qkv, beta, a, state, gate, norm_w, conv_w, conv_state)
    if beta.stride(0) != a.stride(0):
        raise ValueError("beta and a must share a row stride")
    out = torch.empty((qkv.shape[0], heads * vdim), dtype=qkv.dtype, device=qkv.device) if out is None else out
    L, tokens = _cabi.lib(), qkv.shape[0]
    need = L.mv_delta_chunk_workspace_bytes(tokens, slots.numel(), heads, dim, vdim) if cu is not None else -1
    if chunked is None:
        chunked = need >= 0 and qkv.dtype == torch.bfloat16 and tokens >= CHUNK_FROM * slots.numel()
    if chunked:
        ws = torch.empty(max(need, 1), dtype=torch.uint8, device=qkv.device)
        _cabi.check(L.mv_delta_chunk_scan(
            out.data_ptr(), out.stride(0), qkv.data_ptr(), qkv.stride(0), beta.data_ptr(), a.data_ptr(), a.stride(0),
            A_log.data_ptr(), dt_bias.data_ptr(), cu.data_ptr(), slots.numel(), tokens, slots.data_ptr(), starts.data_ptr(),
            state.data_ptr(), state.shape[0], heads, kv_heads, dim, vdim, dim ** -0.5, ws.data_ptr(), ws.numel(),
            _cabi.stream_ptr()))
        return out
    ptr = lambda t: t.data_ptr() if t is not None else None
    _cabi.check(L.mv_delta_scan(
        out.data_ptr(), out.stride(0), qkv.data_ptr(), qkv.stride(0), beta.data_ptr(), a.data_ptr(), a.stride(0),
        A_log.data_ptr(), dt_bias.data_ptr(), ptr(cu), slots.numel(), slots.data_ptr(), starts.data_ptr(),
        state.data_ptr(), state.shape[0], heads, kv_heads, dim, vdim, dim ** -0.5, ptr(conv_w),
        conv_w.shape[1] if conv_w is not None else 0, ptr(conv_state), ptr(gate), gate.stride(0) if gate is not None else 0,
        ptr(norm_w), eps, _cabi.layer_dtype_code(qkv.dtype), _cabi.stream_ptr()))
    return out


class GatedDeltaRule(nn.Module):
    """With `stack` False the caller computes the products of `parts` (one stacked product for several mixers) and hands
    them to `mix`."""

    def __init__(self, m, width, eps, load, stack=True):
        super().__init__()
        self.heads, self.kv_heads, self.dim, self.vdim, self.taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
        self.eps = eps
        if self.heads % self.kv_heads or self.taps < 1:
            raise ValueError("gated delta rule: heads must be a multiple of kv_heads, and the convolution have a tap")
        H, qk, vs = self.heads, self.kv_heads * self.dim, self.heads * self.vdim
        self.channels = 2 * qk + vs
        self.parts = {"qkv": torch.cat([load("q", (qk, width)), load("k", (qk, width)), load("v", (vs, width))]),
                      "g": load("g", (vs, width)), "ba": torch.cat([load("b", (H, width)), load("a", (H, width))])}
        self.stacked = None
        if stack:
            self.stacked, self.parts = StackedLinear(self.parts), None
        param = lambda t: nn.Parameter(t, requires_grad=False)
        self.conv_w = param(torch.cat([load(n + ".conv", (c, self.taps)) for n, c in (("q", qk), ("k", qk), ("v", vs))]))
        self.A_log, self.dt_bias = param(load("A_log", (H,))), param(load("dt_bias", (H,)))
        self.norm_w, self.o_w = param(load("norm", (self.vdim,))), param(load("o", (width, vs)))
        self.slot_state = None          # assigned by the model runner

    def slot_state_spec(self, dtype):
        """Per-sequence state: name -> (shape, dtype)."""
        return {"conv": ((self.taps - 1, self.channels), dtype),
                "S": ((self.heads, self.dim, self.vdim), torch.float32)}

    def forward(self, h):
        return self.mix(self.stacked(h))

    def mix(self, p):
        """p: {name: (tokens, rows)} of the parts' products -> (tokens, width)."""
        ctx = get_context()
        u, g, beta, a = p["qkv"], p["g"], p["ba"][:, :self.heads], p["ba"][:, self.heads:]
        slots, starts, nd = ctx.state_slots, ctx.state_starts, ctx.num_decode
        conv, S = self.slot_state["conv"], self.slot_state["S"]
        dims, gates = (self.heads, self.kv_heads, self.dim, self.vdim), (self.A_log, self.dt_bias)
        y = torch.empty((u.shape[0], self.heads * self.vdim), dtype=u.dtype, device=u.device)
        if nd:                           # sequences with one token come first
            delta_scan(u[:nd], beta[:nd], a[:nd], *gates, None, slots[:nd], starts[:nd], S, *dims, conv_w=self.conv_w,
                       conv_state=conv, gate=g[:nd], norm_w=self.norm_w, eps=self.eps, out=y[:nd])
        if u.shape[0] > nd:
            cu = ctx.portion_cu_q
            x = conv_silu(u[nd:], self.conv_w, None, cu, slots[nd:], starts[nd:], conv)
            o = delta_scan(x, beta[nd:], a[nd:], *gates, cu, slots[nd:], starts[nd:], S, *dims)
            head_norm_gate(o, g[nd:], self.norm_w, self.heads, self.eps, out=y[nd:])
        conv_state_update(conv, u, self.taps, ctx.cu_seqlens_q, slots, starts)
        return F.linear(y, self.o_w)
