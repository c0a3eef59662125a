"""Matrix memory with exponential input gates, capped gate logits and a running maximum (mLSTM): the recurrence on a matrix
and a vector per head in 32-bit, a norm per head and a sigmoid output gate (csrc/mlstm.cu; portions of prompts in chunks on
tensor cores, csrc/mlstm_chunk.cu).
"""
import torch
import torch.nn as nn
import torch.nn.functional as F

from .. import _cabi
from ..utils.context import get_context
from .gla import CHUNK_FROM
from .group_norm import head_norm_gate
from .linear import StackedLinear, router_logits


def mlstm_gates(gates, i_b, f_b, cap, cu, slots, starts, m, heads):
    """gates (tokens, 2 * heads) fp32 logits of packed portions -> the chain (tokens, heads, 4) fp32: log input gate, log
    forget gate, running maximum before and after the token.  Advances m (slots, heads).  See mv_mlstm_gates."""
    _cabi.require_cuda(gates, i_b, f_b, m)
    chain = torch.empty((gates.shape[0], heads, 4), dtype=torch.float32, device=gates.device)
    _cabi.check(_cabi.lib().mv_mlstm_gates(
        chain.data_ptr(), gates.data_ptr(), gates.stride(0), i_b.data_ptr(), f_b.data_ptr(), cap, cu.data_ptr(), slots.numel(),
        slots.data_ptr(), starts.data_ptr(), m.data_ptr(), m.shape[0], heads, _cabi.layer_dtype_code(i_b.dtype),
        _cabi.stream_ptr()))
    return chain


def mlstm_scan(q, k, v, chain, cu, slots, starts, S, n, heads, dim, vdim, chunked=None):
    """q, k, v: views of one row-major product, packed portions.  Advances S (slots, heads, dim, vdim) and n (slots, heads,
    dim), fp32; returns the read-outs (tokens, heads * vdim) and their denominators (tokens, heads) fp32.  bf16 portions take
    the chunked kernels when those have the sizes."""
    _cabi.require_cuda(q, k, v, chain, S, n)
    if not q.stride(0) == k.stride(0) == v.stride(0):
        raise ValueError("q, k and v must share a row stride")
    L, tokens = _cabi.lib(), q.shape[0]
    out = torch.empty((tokens, heads * vdim), dtype=q.dtype, device=q.device)
    den = torch.empty((tokens, heads), dtype=torch.float32, device=q.device)
    need = L.mv_mlstm_chunk_workspace_bytes(tokens, slots.numel(), heads, dim, vdim)
    if chunked is None:
        chunked = need >= 0 and q.dtype == torch.bfloat16 and tokens >= CHUNK_FROM * slots.numel()
    head = (out.data_ptr(), out.stride(0), den.data_ptr(), q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0), chain.data_ptr(),
            cu.data_ptr(), slots.numel())
    state = (slots.data_ptr(), starts.data_ptr(), S.data_ptr(), n.data_ptr(), S.shape[0], heads, dim, vdim, dim ** -0.5)
    if chunked:
        ws = torch.empty(max(need, 1), dtype=torch.uint8, device=q.device)
        _cabi.check(L.mv_mlstm_chunk_scan(*head, tokens, *state, ws.data_ptr(), ws.numel(), _cabi.stream_ptr()))
    else:
        _cabi.check(L.mv_mlstm_scan(*head, *state, _cabi.layer_dtype_code(q.dtype), _cabi.stream_ptr()))
    return out, den


def mlstm_step(q, k, v, x, gates_w, i_b, f_b, cap, slots, starts, S, n, m, heads, dim, vdim, gate, norm_w, eps, out=None):
    """One token per sequence: the normed and gated rows (tokens, heads * vdim).  The gates' logits are formed here, from x
    (tokens, width) and gates_w (2 * heads, width).  See mv_mlstm_step."""
    _cabi.require_cuda(q, k, v, x, gates_w, S, n, m, gate, norm_w)
    if not q.stride(0) == k.stride(0) == v.stride(0):
        raise ValueError("q, k and v must share a row stride")
    out = torch.empty((q.shape[0], heads * vdim), dtype=q.dtype, device=q.device) if out is None else out
    _cabi.check(_cabi.lib().mv_mlstm_step(
        out.data_ptr(), out.stride(0), q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0), x.data_ptr(), x.stride(0),
        gates_w.data_ptr(), x.shape[1], i_b.data_ptr(), f_b.data_ptr(), cap, slots.numel(), slots.data_ptr(), starts.data_ptr(), S.data_ptr(), n.data_ptr(),
        m.data_ptr(), S.shape[0], heads, dim, vdim, dim ** -0.5, gate.data_ptr(), gate.stride(0), norm_w.data_ptr(), eps,
        _cabi.layer_dtype_code(q.dtype), _cabi.stream_ptr()))
    return out


class MatrixMemory(nn.Module):
    def __init__(self, m, width, eps, load):
        super().__init__()
        self.heads, self.dim, self.vdim, self.cap, self.eps = m["heads"], m["dim"], m["vdim"], float(m["gate_cap"]), eps
        if self.cap <= 0:
            raise ValueError("mlstm: gate_cap must be positive")
        H, K, V = self.heads, self.dim, self.vdim
        self.stacked = StackedLinear({"q": load("q", (H * K, width)), "k": load("k", (H * K, width)),
                                      "v": load("v", (H * V, width)), "g": load("g", (H * V, width))})
        param = lambda t: nn.Parameter(t, requires_grad=False)
        self.gates_w = param(torch.cat([load("i", (H, width)), load("f", (H, width))]))
        self.i_b, self.f_b = param(load("i.b", (H,))), param(load("f.b", (H,)))
        self.norm_w, self.o_w = param(load("norm", (H * V,))), param(load("o", (width, H * V)))
        self.slot_state = None          # assigned by the model runner

    def slot_state_spec(self, dtype):
        """Per-sequence state: name -> (shape, dtype)."""
        return {"S": ((self.heads, self.dim, self.vdim), torch.float32), "n": ((self.heads, self.dim), torch.float32),
                "m": ((self.heads,), torch.float32)}

    def forward(self, h):
        """h (tokens, width) -> (tokens, width)."""
        ctx = get_context()
        p = self.stacked(h)
        q, k, v, g = p["q"], p["k"], p["v"], p["g"]
        slots, starts, nd = ctx.state_slots, ctx.state_starts, ctx.num_decode
        S, n, m = (self.slot_state[name] for name in ("S", "n", "m"))
        dims = (self.heads, self.dim, self.vdim)
        y = torch.empty((h.shape[0], self.heads * self.vdim), dtype=h.dtype, device=h.device)
        if nd:                           # sequences with one token come first
            mlstm_step(q[:nd], k[:nd], v[:nd], h[:nd], self.gates_w, self.i_b, self.f_b, self.cap, slots[:nd], starts[:nd], S, n, m, *dims,
                       g[:nd], self.norm_w, self.eps, out=y[:nd])
        if h.shape[0] > nd:
            cu, at = ctx.portion_cu_q, (slots[nd:], starts[nd:])
            z = router_logits(h[nd:], self.gates_w)          # the gates' logits stay in 32-bit
            chain = mlstm_gates(z, self.i_b, self.f_b, self.cap, cu, *at, m, self.heads)
            o, den = mlstm_scan(q[nd:], k[nd:], v[nd:], chain, cu, *at, S, n, *dims)
            head_norm_gate(o, g[nd:], self.norm_w, self.heads, self.eps, out=y[nd:], den=den, act="sigmoid")
        return F.linear(y, self.o_w)
