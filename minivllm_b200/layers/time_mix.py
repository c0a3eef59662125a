"""Time mixing (RWKV): projections of mixtures with the token before, a decay per key channel from a low-rank product, the
recurrence on a matrix state in 32-bit with a bonus for the token's own entry, a norm per head and an output gate
(csrc/time_mix.cu; portions of prompts in chunks on tensor cores, csrc/gla_chunk.cu).
"""
import torch
import torch.nn as nn
import torch.nn.functional as F

from .. import _cabi
from ..utils.context import get_context
from .gla import CHUNK_FROM, DEFAULT_RANK
from .group_norm import head_norm_gate
from .linear import router_logits
from .tanh_norm import TokenShift


def tanh_rows(y, dtype):
    """tanh of y (rows, cols) fp32, in `dtype`."""
    _cabi.require_cuda(y)
    out = torch.empty(y.shape, dtype=dtype, device=y.device)
    _cabi.check(_cabi.lib().mv_tanh_rows(out.data_ptr(), y.data_ptr(), y.stride(0), y.shape[0], y.shape[1],
                                         _cabi.layer_dtype_code(dtype), _cabi.stream_ptr()))
    return out


def time_scan(r, k, v, z, w0, bonus, cu, slots, starts, state, heads, dim, vdim, gate=None, norm_w=None, eps=0.0, out_scale=1.0,
              out=None, chunked=None):
    """r, k, v: rows of one stride; z (tokens, heads * dim) fp32.  Advances `state` (slots, heads, dim, vdim) fp32 and returns
    (tokens, heads * vdim): the read-outs of packed portions (cu), or with cu None (one token per sequence) the normed and
    gated rows times out_scale.  See mv_time_scan.  bf16 portions take the chunked kernels when those have the sizes."""
    _cabi.require_cuda(r, k, v, z, w0, bonus, state, gate, norm_w)
    if not r.stride(0) == k.stride(0) == v.stride(0):
        raise ValueError("r, k and v must share a row stride")
    out = torch.empty((r.shape[0], heads * vdim), dtype=r.dtype, device=r.device) if out is None else out
    L, tokens = _cabi.lib(), r.shape[0]
    need = L.mv_gla_chunk_workspace_bytes(tokens, slots.numel(), heads, dim, vdim) if cu is not None else -1
    if chunked is None:
        chunked = need >= 0 and r.dtype == torch.bfloat16 and tokens >= CHUNK_FROM * slots.numel()
    head = (out.data_ptr(), out.stride(0), r.data_ptr(), k.data_ptr(), v.data_ptr(), r.stride(0), z.data_ptr(), z.stride(0),
            w0.data_ptr(), bonus.data_ptr(), cu.data_ptr() if cu is not None else None, slots.numel())
    tail = (slots.data_ptr(), starts.data_ptr(), state.data_ptr(), state.shape[0], heads, dim, vdim)
    if chunked:
        ws = torch.empty(max(need, 1), dtype=torch.uint8, device=r.device)
        _cabi.check(L.mv_time_chunk_scan(*head, tokens, *tail, ws.data_ptr(), ws.numel(), _cabi.stream_ptr()))
        return out
    ptr = lambda t: t.data_ptr() if t is not None else None
    _cabi.check(L.mv_time_scan(*head, *tail, ptr(gate), gate.stride(0) if gate is not None else 0, ptr(norm_w), eps, out_scale,
                               _cabi.layer_dtype_code(r.dtype), _cabi.stream_ptr()))
    return out


class TimeMixing(nn.Module):
    """The caller makes the mixtures in front of it (`shift`) and the output product (`o_w`)."""
    MIXTURES = ("r", "k", "v", "g", "w")

    def __init__(self, m, width, eps, load):
        super().__init__()
        self.heads, self.dim, self.eps = m["heads"], m["dim"], eps
        n = self.heads * self.dim
        param = lambda t: nn.Parameter(t, requires_grad=False)
        self.shift = TokenShift(torch.stack([load("mu." + x, (width,)) for x in self.MIXTURES]))
        self.rkvg_w = param(torch.stack([load(x, (n, width)) for x in "rkvg"]))
        rank = load.shape("w1", (DEFAULT_RANK, width))[0]
        pad = -rank % 8                  # rows of whole 16-byte pieces
        self.w1_w = param(F.pad(load("w1", (rank, width)), (0, 0, 0, pad)))
        self.w2_w = param(F.pad(load("w2", (n, rank)), (0, pad)))
        self.w0, self.bonus = param(load("w0", (n,))), param(load("u", (self.heads, self.dim)))
        self.norm_w, self.o_w = param(load("norm", (n,))), param(load("o", (width, n)))
        self.slot_state = None          # assigned by the model runner

    @property
    def columns(self):
        return self.heads * self.dim

    def slot_state_spec(self, dtype):
        """Per-sequence state: name -> (shape, dtype)."""
        return {"S": ((self.heads, self.dim, self.dim), torch.float32)}

    def results(self, inputs, out, scale):
        """inputs (h, mixtures (5, tokens, width)); the heads' results times `scale` go to out (tokens, columns), any row
        stride."""
        ctx, (_, x) = get_context(), inputs
        r, k, v, g = torch.bmm(x[:4], self.rkvg_w.transpose(1, 2)).unbind(0)
        z = router_logits(tanh_rows(router_logits(x[4], self.w1_w), x.dtype), self.w2_w)
        slots, starts, nd, S = ctx.state_slots, ctx.state_starts, ctx.num_decode, self.slot_state["S"]
        dims, decay = (self.heads, self.dim, self.dim), (self.w0, self.bonus)
        if nd:                           # sequences with one token come first
            time_scan(r[:nd], k[:nd], v[:nd], z[:nd], *decay, None, slots[:nd], starts[:nd], S, *dims, gate=g[:nd],
                      norm_w=self.norm_w, eps=self.eps, out_scale=scale, out=out[:nd])
        if r.shape[0] > nd:
            o = time_scan(r[nd:], k[nd:], v[nd:], z[nd:], *decay, ctx.portion_cu_q, slots[nd:], starts[nd:], S, *dims)
            head_norm_gate(o, g[nd:], self.norm_w, self.heads, self.eps, out=out[nd:], mult=scale)
