"""Mixture-of-experts feed-forward: fp32 router with softmax over the chosen experts (perhaps chosen within the best
groups of experts), grouped products over the experts' row ranges, an optional shared expert, perhaps with a scalar gate
per token (csrc/moe.cu).

The step's h feeds everything at once: one stacked product gives the shared expert's gate and up projections, its
scalar gate, and whatever the caller adds (`extra`, e.g. the gate of the residual); the expert sum itself is formed
by the kernel that adds the result to the residual stream (layers/group_norm.py).
"""
import torch
import torch.nn as nn
import torch.nn.functional as F

from .. import _cabi
from .attention import _error_word
from .group_norm import ACTS, gate_mul, moe_residual_norm
from .linear import StackedLinear, router_logits


def route(logits, bias, top, groups=1, keep=1, over_all=False, scale=1.0):
    """fp32 logits (tokens, experts) -> (idx int32, weight fp32), both (tokens, top), best first.  Of `groups` equal runs
    of experts only the `keep` with the largest maxima are chosen from.  Weights are `scale` times a softmax over the chosen
    experts, or with `over_all` over all."""
    _cabi.require_cuda(logits)
    tokens, experts = logits.shape
    idx = torch.empty((tokens, top), dtype=torch.int32, device=logits.device)
    weight = torch.empty((tokens, top), dtype=torch.float32, device=logits.device)
    _cabi.check(_cabi.lib().mv_moe_route(idx.data_ptr(), weight.data_ptr(), logits.data_ptr(), logits.stride(0),
                                         bias.data_ptr() if bias is not None else None, tokens, experts, top, groups,
                                         keep, int(over_all), scale, _cabi.stream_ptr()))
    return idx, weight


def sort_by_expert(idx, experts):
    """(pos (tokens, top), row_token (tokens * top), offsets (experts + 1)), int32: see mv_moe_sort."""
    tokens, top = idx.shape
    dev = idx.device
    pos = torch.empty((tokens, top), dtype=torch.int32, device=dev)
    row_token = torch.empty(tokens * top, dtype=torch.int32, device=dev)
    offsets = torch.empty(experts + 1, dtype=torch.int32, device=dev)
    L = _cabi.lib()
    need = L.mv_moe_sort_workspace_bytes(tokens, experts, top)
    ws = torch.empty(max(need, 1), dtype=torch.uint8, device=dev)
    _cabi.check(L.mv_moe_sort(pos.data_ptr(), row_token.data_ptr(), offsets.data_ptr(), idx.data_ptr(), tokens,
                              experts, top, ws.data_ptr(), need, _cabi.stream_ptr()))
    return pos, row_token, offsets


def gather_rows(x, row_token):
    out = torch.empty((row_token.numel(), x.shape[1]), dtype=x.dtype, device=x.device)
    _cabi.check(_cabi.lib().mv_gather_rows(out.data_ptr(), x.data_ptr(), x.stride(0), row_token.data_ptr(),
                                           row_token.numel(), x.shape[1], _cabi.layer_dtype_code(x.dtype),
                                           _cabi.stream_ptr()))
    return out


def grouped_linear(x, weight, offsets, gated=False, tensor_cores=None, act="silu", limit=0.0):
    """x (rows, in) sorted by expert, weight (experts, out, in) -> (rows, out).  With `gated`, weight is
    (experts, 2 * out, in), gate rows first, and the result the gate applied to up (`act`).  bf16 runs on the tensor cores when the rows
    are whole 16-byte pieces."""
    _cabi.require_cuda(x, weight, offsets)
    experts, out_dim, in_dim = weight.shape
    if gated:
        out_dim //= 2
    rows, code = x.shape[0], ACTS[act] if gated else -1
    out = torch.empty((rows, out_dim), dtype=x.dtype, device=x.device)
    if tensor_cores is None:
        tensor_cores = x.dtype == torch.bfloat16 and in_dim % 8 == 0
    if tensor_cores:
        _cabi.check(_cabi.lib().mv_grouped_gemm(out.data_ptr(), x.data_ptr(), weight.data_ptr(), offsets.data_ptr(),
                                                experts, rows, in_dim, out_dim, code, limit,
                                                _error_word(x.device).data_ptr(), _cabi.stream_ptr()))
        return out
    _cabi.check(_cabi.lib().mv_grouped_rows(out.data_ptr(), x.data_ptr(), weight.data_ptr(), offsets.data_ptr(),
                                            experts, rows, in_dim, out_dim, code, limit,
                                            _cabi.layer_dtype_code(x.dtype), _cabi.stream_ptr()))
    return out


class MixtureOfExperts(nn.Module):
    """spec: {'router': {'experts', 'top', 'groups': {'count', 'keep'} or absent, 'scale' of the weights or absent}, 'expert':
    {'ff', 'limit' with the clamped activation}, 'shared': the same or absent}; `load(name, shape)` returns a tensor of the
    layer's feed-forward.  `over_all`: weights are probabilities among all experts, not among the chosen."""

    def __init__(self, spec, width, load, extra=None, act="silu", router_bias=True, shared_gate=True,
                 over_all=False):
        super().__init__()
        self.experts, self.top = spec["router"]["experts"], spec["router"]["top"]
        groups = spec["router"].get("groups") or {"count": 1, "keep": 1}
        self.groups, self.keep = groups["count"], groups["keep"]
        if self.experts % self.groups or not 0 < self.keep <= self.groups or \
                not 0 < self.top <= self.experts // self.groups * self.keep:
            raise ValueError(f"moe: top {self.top} of {self.experts} experts in {self.groups} groups, {self.keep} kept")
        self.over_all, self.scale = over_all, float(spec["router"].get("scale", 1.0))
        ff = spec["expert"]["ff"]
        self.act, self.limit = act, float(spec["expert"].get("limit", 0.0))
        param = lambda t: nn.Parameter(t, requires_grad=False)
        self.router_w = param(load("router", (self.experts, width)))
        self.router_b = param(load("router.b", (self.experts,)).float()) if router_bias else None
        first = load("e0.gate", (ff, width))
        gate_up = torch.empty((self.experts, 2 * ff, width), dtype=first.dtype, device=first.device)
        down = torch.empty((self.experts, width, ff), dtype=first.dtype, device=first.device)
        for e in range(self.experts):
            gate_up[e, :ff] = first if e == 0 else load(f"e{e}.gate", (ff, width))
            gate_up[e, ff:] = load(f"e{e}.up", (ff, width))
            down[e] = load(f"e{e}.down", (width, ff))
        self.gate_up_w, self.down_w = param(gate_up), param(down)
        parts = dict(extra or {})
        self.shared_down = None
        if spec.get("shared"):
            sff = spec["shared"]["ff"]
            parts["shared_gate"] = load("shared.gate", (sff, width))
            parts["shared_up"] = load("shared.up", (sff, width))
            if shared_gate:
                parts["sg"] = load("shared.sg", (1, width))
            self.shared_limit = float(spec["shared"].get("limit", 0.0))
            self.shared_down = param(load("shared.down", (width, sff)))
        self.stacked = StackedLinear(parts) if parts else None

    def routed(self, h):
        """h (tokens, width) -> (rows, pos, weight): token t's experts' results are rows[pos[t, k]], to be summed with
        weight[t, k]."""
        idx, weight = route(router_logits(h, self.router_w), self.router_b, self.top, self.groups, self.keep, self.over_all,
                            self.scale)
        pos, row_token, offsets = sort_by_expert(idx, self.experts)
        act = grouped_linear(gather_rows(h, row_token), self.gate_up_w, offsets, gated=True, act=self.act,
                             limit=self.limit)
        return grouped_linear(act, self.down_w, offsets), pos, weight

    def forward(self, h, x, gate_bias, w_post, w_next, mult, groups, eps):
        """h: the sublayer's input, x: residual stream (updated in place).  Returns the next sublayer's input.  The
        residual gate, if any, is the stacked part 'residual_gate'."""
        p = self.stacked(h) if self.stacked is not None else {}
        rows, pos, weight = self.routed(h)
        shared = None
        if self.shared_down is not None:
            shared = F.linear(gate_mul(p["shared_up"], p["shared_gate"], self.act, limit=self.shared_limit),
                              self.shared_down)
        return moe_residual_norm(x, rows, pos, weight, shared, p.get("sg"), p.get("residual_gate"), gate_bias, w_post,
                                 w_next, mult, groups, eps)
