"""Differential attention in chunks of the sequence: every head has two maps with queries and keys of their own over the same
values; the second one's result, times one learned factor per layer, is taken off the first's, and the difference is normed per
head and gated (csrc/window_attention.cu, csrc/latent_prefill.cu).  Its keys and values may be an earlier layer's.

The cache holds one row [keys of all KV heads, two maps each | values of all KV heads] per token, keys after their norm.
"""
import torch
import torch.nn as nn
import torch.nn.functional as F

from .. import _cabi
from ..utils.context import get_context
from .attention import _error_word
from .latent_attention import latent_gather
from .linear import StackedLinear
from .rotary_attention import qkv_rope_store
from .window_attention import chunk_keys

MAPS = 2


def diff_attention_rows(q, cache, block_tables, cu_q, positions, chunk, gate, lam, mult, eps, heads, kv_heads, dim, vdim, scale, out):
    """q (tokens, heads * 2 * dim), gate (tokens, heads * vdim); out (tokens, heads * vdim), dense.  cu_q None: one token per
    row of block_tables."""
    _cabi.require_cuda(q, cache, block_tables, positions, gate, out)
    tokens = q.shape[0]
    a = torch.empty((tokens, heads, MAPS, vdim), dtype=torch.float32, device=q.device)
    _cabi.check(_cabi.lib().mv_diff_attention_rows(
        a.data_ptr(), q.data_ptr(), q.stride(0), cache.data_ptr(), block_tables.data_ptr(), block_tables.stride(0),
        block_tables.shape[1], cache.shape[1], cache.shape[0], cu_q.data_ptr() if cu_q is not None else None,
        block_tables.shape[0], positions.data_ptr(), chunk, tokens, heads, kv_heads, dim, vdim, scale,
        _cabi.layer_dtype_code(q.dtype), _cabi.stream_ptr()))
    _cabi.check(_cabi.lib().mv_diff_norm_gate(out.data_ptr(), a.data_ptr(), gate.data_ptr(), gate.stride(0), lam, mult, eps, tokens,
                                              heads, vdim, _cabi.layer_dtype_code(q.dtype), _cabi.stream_ptr()))
    return out


def diff_decode(q, cache, block_tables, positions, chunk, gate, lam, mult, eps, heads, kv_heads, dim, vdim, scale, out):
    """diff_attention_rows for one row per sequence on tensor cores; None when the kernel does not take the sizes."""
    _cabi.require_cuda(q, cache, block_tables, positions, gate, out)
    batch, L = q.shape[0], _cabi.lib()
    need = L.mv_diff_decode_workspace_bytes(batch, heads, kv_heads, dim, vdim, max(1, min(chunk, block_tables.shape[1] * cache.shape[1])))
    if need < 0 or q.dtype != torch.bfloat16:
        return None
    ws = torch.empty(max(need, 16), dtype=torch.uint8, device=q.device)
    _cabi.check(L.mv_diff_decode(
        out.data_ptr(), q.data_ptr(), q.stride(0), cache.data_ptr(), block_tables.data_ptr(), block_tables.stride(0),
        block_tables.shape[1], cache.shape[1], cache.shape[0], positions.data_ptr(), chunk, gate.data_ptr(), gate.stride(0), lam, mult,
        eps, batch, heads, kv_heads, dim, vdim, scale, ws.data_ptr(), ws.numel(), _cabi.stream_ptr()))
    return out


def diff_prefill(q, kv, cu_q, cu_k, chunk, gate, lam, mult, eps, heads, kv_heads, dim, vdim, scale, out):
    """q (tokens, heads * 2 * dim), kv (keys, kv_heads * (2 * dim + vdim)) packed rows, a sequence's first at the beginning of a
    chunk; out (tokens, heads * vdim), dense."""
    _cabi.require_cuda(q, kv, cu_q, cu_k, gate, out)
    v = kv[:, kv_heads * MAPS * dim:]
    _cabi.check(_cabi.lib().mv_diff_prefill(
        out.data_ptr(), q.data_ptr(), q.stride(0), kv.data_ptr(), kv.stride(0), v.data_ptr(), v.stride(0), cu_q.data_ptr(),
        cu_k.data_ptr(), cu_q.numel() - 1, q.shape[0], kv.shape[0], chunk, gate.data_ptr(), gate.stride(0), lam, mult, eps, heads,
        kv_heads, dim, vdim, scale, _error_word(q.device).data_ptr(), _cabi.stream_ptr()))
    return out


class DifferentialAttention(nn.Module):
    """`source`: the earlier layer of this class whose keys and values this one uses, or None."""
    shift = None

    def __init__(self, m, width, eps, load, source=None):
        super().__init__()
        self.heads, self.kv_heads, self.dim, self.vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        self.scale, self.eps, self.chunk = float(m["scale"]), eps, int(m["mask"]["size"])
        if self.heads % self.kv_heads or self.chunk < 1:
            raise ValueError("attention: heads must be a multiple of kv_heads, and a chunk hold a token")
        H, G, d, vd = self.heads, self.kv_heads, self.dim, self.vdim
        parts = {"q": load("q", (H * MAPS * d, width)), "g": load("g", (H * vd, width))}
        param = lambda t: nn.Parameter(t, requires_grad=False)
        self.q_norm, self.k_norm = param(load("q.norm", (d,))), None
        lq1, lk1, lq2, lk2 = (load(n, (d,)).float() for n in ("lq1", "lk1", "lq2", "lk2"))
        self.lam = float(torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + m["diff"])
        self.mult = 1.0 - float(m["diff"])
        self.o_w = param(load("o", (width, H * vd)))
        self._source = (source,)        # in a tuple: not a module of this one
        self.lends = False              # does a later layer use these keys and values?
        if source is None:
            parts.update(k=load("k", (G * MAPS * d, width)), v=load("v", (G * vd, width)))
            self.k_norm = param(load("k.norm", (d,)))
            self.paged_cache = None     # (blocks, block_size, paged_row), assigned by the model runner
        else:
            mine, its = ([getattr(x, n) for n in ("kv_heads", "dim", "vdim")] for x in (self, source))
            if mine != its or source._source[0] is not None:
                raise ValueError("attention: kv_from must name an earlier layer with keys and values of its own, and the same "
                                 "KV heads and sizes")
            source.lends = True
        self.stacked = StackedLinear(parts)

    @property
    def paged_row(self):
        return self.kv_heads * (MAPS * self.dim + self.vdim)

    def _tiles(self, dtype):
        """Does the tensor-core prefill kernel take this layer's sizes?"""
        return dtype == torch.bfloat16 and self.scale > 0 and bool(_cabi.lib().mv_diff_prefill_takes(self.dim, self.vdim))

    def _portion_rows(self, ctx, owner, fresh, tables):
        """The packed rows that the portions of this step can see through this layer's chunks, and their cu_k.  A layer that uses
        this one's finds them here too."""
        if fresh is not None:
            return fresh, ctx.portion_cu_q
        cu_k, first, keys = chunk_keys(ctx, self.chunk, owner.paged_cache.device)
        key = ("chunk_rows", id(owner), self.chunk)
        if key in ctx.memo:
            return ctx.memo[key], cu_k
        gathered = latent_gather(owner.paged_cache, cu_k, keys, tables, first)
        if owner.lends:
            ctx.memo[key] = gathered
        return gathered, cu_k

    def forward(self, h):
        """h (tokens, width) -> (tokens, width)."""
        ctx, p = get_context(), self.stacked(h)
        owner = self._source[0] or self
        q, g, nd, cache = p["q"], p["g"], ctx.num_decode, owner.paged_cache
        tokens, H, G = q.shape[0], self.heads, self.kv_heads
        tiles = tokens > nd and self._tiles(q.dtype)
        fresh = tiles and ctx.portion_fresh
        kv = qkv_rope_store(q, p.get("k"), p.get("v"), self.q_norm, self.k_norm, None, self.eps, ctx.positions, None, 0, None,
                            MAPS * H, MAPS * G, cache, ctx.slot_mapping, packed=fresh and owner is self, v_heads=G)
        if fresh and owner.lends:        # the step's own rows, for the layers that share them
            kv = ctx.memo.setdefault(("fresh_rows", id(owner)), kv)
        sizes = (H, G, self.dim, self.vdim, self.scale)
        end = lambda a, b: (self.chunk, g[a:b], self.lam, self.mult, self.eps, *sizes, o[a:b])
        o = torch.empty((tokens, H * self.vdim), dtype=q.dtype, device=q.device)
        if nd:                           # sequences with one token come first
            args = (q[:nd], cache, ctx.block_tables[:nd])
            if diff_decode(*args, ctx.positions[:nd], *end(0, nd)) is None:
                diff_attention_rows(*args, None, ctx.positions[:nd], *end(0, nd))
        if tokens > nd:
            tables, cu_q = ctx.block_tables[nd:], ctx.portion_cu_q
            if not tiles:
                diff_attention_rows(q[nd:], cache, tables, cu_q, ctx.positions[nd:], *end(nd, tokens))
            else:
                rows, cu_k = self._portion_rows(ctx, owner, kv[nd:] if fresh else None, tables)
                diff_prefill(q[nd:], rows, cu_q, cu_k, *end(nd, tokens))
        return F.linear(o, self.o_w)
