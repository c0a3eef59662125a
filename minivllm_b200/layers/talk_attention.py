"""Grouped-query attention with capped scores, a bias that grows with the logarithm of the distance, and softmax weights that
are mixed across the heads (csrc/talk_attention.cu, csrc/talk_prefill.cu).

The cache holds one row [keys of all KV heads | values of all KV heads] per token.  Decoded tokens leave every head's weights
in scratch and mix them where they meet the values.  The mixture is linear, so portions of prompts take it afterwards: the
tcgen05 kernel applies every head's weights to the values of every value head, and a second launch combines the results.
Sizes those kernels do not take, and 32-bit models, run on a kernel for any sizes, with the same second launch.
"""
import torch
import torch.nn as nn

from .. import _cabi
from ..utils.context import get_context
from .attention import _error_word
from .latent_attention import latent_gather
from .linear import StackedLinear
from .rotary_attention import qkv_rope_store
from .window_attention import UNBOUNDED, window_keys


def talk_attention_rows(q, cache, block_tables, cu_q, positions, kv_heads, dim, vdim, scale, r1, r2, cap):
    """q (tokens, heads * dim) -> (tokens, heads, kv_heads, vdim) fp32: every head's weights over every value head; cu_q None:
    one token per row of block_tables."""
    _cabi.require_cuda(q, cache, block_tables, positions, r1, r2)
    tokens, heads = q.shape[0], q.shape[1] // dim
    a = torch.empty((tokens, heads, kv_heads, vdim), dtype=torch.float32, device=q.device)
    _cabi.check(_cabi.lib().mv_talk_attention_rows(
        a.data_ptr(), q.data_ptr(), q.stride(0), cache.data_ptr(), block_tables.data_ptr(), block_tables.stride(0),
        block_tables.shape[1], cache.shape[1], cache.shape[0], cu_q.data_ptr() if cu_q is not None else None,
        block_tables.shape[0], positions.data_ptr(), r1.data_ptr(), r2.data_ptr(), cap, tokens, heads, kv_heads, dim, vdim, scale,
        _cabi.layer_dtype_code(q.dtype), _cabi.stream_ptr()))
    return a


def talk_decode(q, cache, block_tables, positions, kv_heads, dim, vdim, scale, r1, r2, cap, talk, out, out_scale=1.0):
    """One token per sequence; out (batch, heads * vdim), any row stride.  False when the kernels do not take the sizes."""
    _cabi.require_cuda(q, cache, block_tables, positions, r1, r2, talk, out)
    batch, heads = q.shape[0], q.shape[1] // dim
    L = _cabi.lib()
    need = L.mv_talk_decode_workspace_bytes(batch, heads, kv_heads, dim, vdim, cap, block_tables.shape[1] * cache.shape[1])
    if need < 0 or q.dtype != torch.bfloat16 or out.stride(0) % 2 or out.data_ptr() % 4:
        return False
    ws = torch.empty(max(need, 16), dtype=torch.uint8, device=q.device)
    _cabi.check(L.mv_talk_decode(
        out.data_ptr(), out.stride(0), q.data_ptr(), q.stride(0), cache.data_ptr(), block_tables.data_ptr(), block_tables.stride(0),
        block_tables.shape[1], cache.shape[1], cache.shape[0], positions.data_ptr(), r1.data_ptr(), r2.data_ptr(), talk.data_ptr(),
        cap, batch, heads, kv_heads, dim, vdim, scale, out_scale, ws.data_ptr(), ws.numel(), _cabi.stream_ptr()))
    return True


def talk_prefill(q, k, v, cu_q, cu_k, kv_heads, dim, vdim, scale, r1, r2, cap):
    """q (tokens, heads * dim), k (keys, kv_heads * dim), v (keys, kv_heads * vdim), packed, any row strides -> (tokens, heads,
    kv_heads, vdim)."""
    _cabi.require_cuda(q, k, v, cu_q, cu_k, r1, r2)
    heads = q.shape[1] // dim
    a = torch.empty((q.shape[0], heads, kv_heads, vdim), dtype=q.dtype, device=q.device)
    _cabi.check(_cabi.lib().mv_talk_prefill(
        a.data_ptr(), q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), cu_q.data_ptr(),
        cu_k.data_ptr(), cu_q.numel() - 1, q.shape[0], k.shape[0], r1.data_ptr(), r2.data_ptr(), cap, heads, kv_heads, dim, vdim,
        scale, _error_word(q.device).data_ptr(), _cabi.stream_ptr()))
    return a


def head_mix(a, talk, out, out_scale=1.0):
    """a (tokens, heads, kv_heads, vdim), fp32 or out's type; out (tokens, heads * vdim), any row stride: head h gets out_scale
    times the sum of talk[h, g] a[g, value head of h]."""
    _cabi.require_cuda(a, talk, out)
    tokens, heads, kv_heads, vdim = a.shape
    _cabi.check(_cabi.lib().mv_head_mix(
        out.data_ptr(), out.stride(0), a.data_ptr(), _cabi.layer_dtype_code(a.dtype), talk.data_ptr(), out_scale, tokens, heads,
        kv_heads, vdim, _cabi.layer_dtype_code(out.dtype), _cabi.stream_ptr()))
    return out


class TalkingAttention(nn.Module):
    """The caller makes the output product (`o_w`)."""
    shift = None

    def __init__(self, m, width, eps, load):
        super().__init__()
        self.heads, self.kv_heads, self.dim, self.vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        self.scale, self.cap = float(m["scale"]), float(m["softcap"])
        if self.heads % self.kv_heads or not self.cap > 0:
            raise ValueError("attention: heads must be a multiple of kv_heads, and softcap positive")
        H, G, d, vd = self.heads, self.kv_heads, self.dim, self.vdim
        self.stacked = StackedLinear({"q": load("q", (H * d, width)), "k": load("k", (G * d, width)), "v": load("v", (G * vd, width))})
        param = lambda t: nn.Parameter(t, requires_grad=False)
        self.r1, self.r2, self.talk = (param(load(n, s).float()) for n, s in (("r1", (H,)), ("r2", (H,)), ("talk", (H, H))))
        self.o_w = param(load("o", (width, H * vd)))
        self.paged_cache = None         # (blocks, block_size, paged_row), assigned by the model runner

    @property
    def columns(self):
        return self.heads * self.vdim

    @property
    def paged_row(self):
        return self.kv_heads * (self.dim + self.vdim)

    def _tiles(self, dtype):
        """Does the tensor-core prefill kernel take this layer's sizes?"""
        return dtype == torch.bfloat16 and bool(_cabi.lib().mv_talk_prefill_takes(self.dim, self.vdim, self.cap))

    def results(self, inputs, out, scale):
        """inputs: h (tokens, width), or a tuple that begins with it; the heads' results times `scale` go to out (tokens,
        columns), any row stride."""
        ctx, p = get_context(), self.stacked(inputs[0] if isinstance(inputs, tuple) else inputs)
        q, k, v, nd, cache = p["q"], p["k"], p["v"], ctx.num_decode, self.paged_cache
        tokens, G, d = q.shape[0], self.kv_heads, self.dim
        qkv_rope_store(None, k, v, None, None, None, 0.0, ctx.positions, None, 0, None, 0, G, cache, ctx.slot_mapping)
        sizes = (G, d, self.vdim, self.scale, self.r1, self.r2, self.cap)
        if nd:                           # sequences with one token come first
            args = (q[:nd], cache, ctx.block_tables[:nd])
            if not talk_decode(*args, ctx.positions[:nd], *sizes, self.talk, out[:nd], scale):
                head_mix(talk_attention_rows(*args, None, ctx.positions[:nd], *sizes), self.talk, out[:nd], scale)
        if tokens > nd:
            tables, cu_q = ctx.block_tables[nd:], ctx.portion_cu_q
            if not self._tiles(q.dtype):
                a = talk_attention_rows(q[nd:], cache, tables, cu_q, ctx.positions[nd:], *sizes)
            elif ctx.portion_fresh:
                a = talk_prefill(q[nd:], k[nd:], v[nd:], cu_q, cu_q, *sizes)
            else:
                cu_k, first, keys = window_keys(ctx, UNBOUNDED, q.device)
                rows = latent_gather(cache, cu_k, keys, tables, first)
                a = talk_prefill(q[nd:], rows[:, :G * d], rows[:, G * d:], cu_q, cu_k, *sizes)
            head_mix(a, self.talk, out[nd:], scale)
