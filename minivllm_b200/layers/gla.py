"""Gated linear attention: a decay per key channel from a low-rank projection, the recurrence on a matrix state in
32-bit, a norm per head and an output gate (csrc/gla.cu; portions of prompts in chunks on tensor cores, csrc/gla_chunk.cu).
"""
import torch
import torch.nn as nn
import torch.nn.functional as F

from .. import _cabi
from ..utils.context import get_context
from .group_norm import head_norm_gate
from .linear import StackedLinear

CHUNK_FROM = 16          # mean tokens per portion from which the chunked kernels are used
DEFAULT_RANK = 16        # of seeded weights; a checkpoint's tensors have their own


def gla_scan(q, k, v, z, tau, cu, slots, starts, state, heads, dim, vdim, gate=None, norm_w=None, eps=0.0, out=None,
             chunked=None):
    """q, k, v, gate: views of one row-major product; z (tokens, heads * dim).  Advances `state` (slots, heads, dim,
    vdim) fp32 and returns (tokens, heads * vdim): the read-outs of packed portions (cu), or with cu None (one token per
    sequence) the normed and gated rows.  See mv_gla_scan.  bf16 portions take the chunked kernels when those have the
    sizes."""
    _cabi.require_cuda(q, k, v, z, state, gate, norm_w)
    if not q.stride(0) == k.stride(0) == v.stride(0):
        raise ValueError("q, k and v must share a row stride")
    out = torch.empty((q.shape[0], heads * vdim), dtype=q.dtype, device=q.device) if out is None else out
    L, tokens = _cabi.lib(), q.shape[0]
    need = L.mv_gla_chunk_workspace_bytes(tokens, slots.numel(), heads, dim, vdim) if cu is not None else -1
    if chunked is None:
        chunked = need >= 0 and q.dtype == torch.bfloat16 and tokens >= CHUNK_FROM * slots.numel()
    if chunked:
        ws = torch.empty(max(need, 1), dtype=torch.uint8, device=q.device)
        _cabi.check(L.mv_gla_chunk_scan(
            out.data_ptr(), out.stride(0), q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0), z.data_ptr(), z.stride(0),
            tau, cu.data_ptr(), slots.numel(), tokens, slots.data_ptr(), starts.data_ptr(), state.data_ptr(), state.shape[0],
            heads, dim, vdim, dim ** -0.5, ws.data_ptr(), ws.numel(), _cabi.stream_ptr()))
        return out
    _cabi.check(L.mv_gla_scan(
        out.data_ptr(), out.stride(0), q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0), z.data_ptr(), z.stride(0),
        tau, cu.data_ptr() if cu is not None else None, slots.numel(), slots.data_ptr(), starts.data_ptr(),
        state.data_ptr(), state.shape[0], heads, dim, vdim, dim ** -0.5, gate.data_ptr() if gate is not None else None,
        gate.stride(0) if gate is not None else 0, norm_w.data_ptr() if norm_w is not None else None, eps,
        _cabi.layer_dtype_code(q.dtype), _cabi.stream_ptr()))
    return out


class GatedLinearAttention(nn.Module):
    def __init__(self, m, width, eps, load):
        super().__init__()
        self.heads, self.dim, self.vdim, self.tau, self.eps = m["heads"], m["dim"], m["vdim"], float(m["tau"]), eps
        if self.tau <= 0:
            raise ValueError("gla: tau must be positive")
        H, K, V = self.heads, self.dim, self.vdim
        rank = load.shape("a1", (DEFAULT_RANK, width))[0]
        self.stacked = StackedLinear({"q": load("q", (H * K, width)), "k": load("k", (H * K, width)),
                                      "v": load("v", (H * V, width)), "g": load("g", (H * V, width)),
                                      "a1": load("a1", (rank, width))})
        param = lambda t: nn.Parameter(t, requires_grad=False)
        self.a2_w, self.a2_b = param(load("a2", (H * K, rank))), param(load("a2.b", (H * K,)))
        self.norm_w, self.o_w = param(load("norm", (V,))), param(load("o", (width, H * V)))
        self.slot_state = None          # assigned by the model runner

    def slot_state_spec(self, dtype):
        """Per-sequence state: name -> (shape, dtype)."""
        return {"S": ((self.heads, self.dim, self.vdim), torch.float32)}

    def forward(self, h):
        """h (tokens, width) -> (tokens, width)."""
        ctx = get_context()
        p = self.stacked(h)
        q, k, v, g = p["q"], p["k"], p["v"], p["g"]
        z = F.linear(p["a1"], self.a2_w, self.a2_b)
        slots, starts, nd, S = ctx.state_slots, ctx.state_starts, ctx.num_decode, self.slot_state["S"]
        dims = (self.heads, self.dim, self.vdim)
        y = torch.empty((h.shape[0], self.heads * self.vdim), dtype=h.dtype, device=h.device)
        if nd:                           # sequences with one token come first
            gla_scan(q[:nd], k[:nd], v[:nd], z[:nd], self.tau, None, slots[:nd], starts[:nd], S, *dims, gate=g[:nd],
                     norm_w=self.norm_w, eps=self.eps, out=y[:nd])
        if h.shape[0] > nd:
            o = gla_scan(q[nd:], k[nd:], v[nd:], z[nd:], self.tau, ctx.portion_cu_q, slots[nd:], starts[nd:], S, *dims)
            head_norm_gate(o, g[nd:], self.norm_w, self.heads, self.eps, out=y[nd:])
        return F.linear(y, self.o_w)
