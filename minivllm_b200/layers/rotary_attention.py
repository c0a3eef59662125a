"""Grouped-query attention with a sliding window, norms per query and key head, rotary positions on keys and values, and a
learned factor per head (csrc/window_attention.cu, csrc/latent_prefill.cu); its keys and values may be an earlier layer's.

A value is turned by its own position before it is cached, and a head's result is turned back by the query's, so that only
their distance is left.  The cache holds one row [keys of all KV heads | values of all KV heads] per token.  Inside the
kernels rotated pairs are neighbouring columns: the weights' rows and columns are put into that order when they are loaded.
The kernels are those of WindowAttention.
"""
import torch
import torch.nn as nn
import torch.nn.functional as F

from .. import _cabi
from ..utils.context import get_context
from .latent_attention import latent_gather, rope_table
from .linear import StackedLinear
from .window_attention import UNBOUNDED, window_attention_rows, window_decode, window_keys, window_prefill


def pair_order(size, dims):
    """Order of a head's `size` columns in which the pairs (i, i + dims / 2) of the first `dims` are neighbours."""
    return [i // 2 + (i % 2) * (dims // 2) for i in range(dims)] + list(range(dims, size))


_turn_tables = {}


def turn_table(base, dims, max_position, device):
    """(dims / 2, max_position, 2) fp32: cos and sin of position * base^(-2i / dims), positions side by side."""
    key = (float(base), int(dims), int(max_position), str(device))
    if key not in _turn_tables:
        _turn_tables[key] = torch.stack([t.t() for t in rope_table(base, dims, max_position, device)], 2).contiguous()
    return _turn_tables[key]


def _reorder(w, heads, order, dim=0):
    """Puts the columns of every head, along dimension `dim` of w, into `order`."""
    if order == list(range(len(order))):
        return w
    at = torch.tensor([h * len(order) + i for h in range(heads) for i in order], device=w.device)
    return w.index_select(dim, at).contiguous()


def qkv_rope_store(q, k, v, q_weight, k_weight, temp, eps, positions, table, dims, vtable, heads, kv_heads, cache=None,
                   slot_mapping=None, packed=False, v_heads=None):
    """Norms and rotates q in place; [k | v], normed and rotated, goes to the cache and, with `packed`, to the returned
    (tokens, row) tensor.  k and v None: queries only; q None: keys and values only; k_weight None: keys without a norm; v_heads:
    value heads, when they are not as many as the key heads.  table, vtable: (cos, sin) or None.  See mv_qkv_rope_store."""
    _cabi.require_cuda(q, k, v, q_weight, k_weight, temp, cache, positions)
    if len({t.stride(0) for t in (q, k, v) if t is not None}) > 1:
        raise ValueError("q, k and v must share a row stride")
    any_, G = q if q is not None else k, kv_heads if k is not None else 0
    VG = (v_heads or G) if G else 0
    heads = heads if q is not None else 0
    tokens, dim = any_.shape[0], any_.shape[1] // (heads or G)
    vdim = v.shape[1] // VG if G else 0
    out = torch.empty((tokens, G * dim + VG * vdim), dtype=any_.dtype, device=any_.device) if packed else None
    ptr = lambda t: t.data_ptr() if t is not None else None
    cos, sin = table if table is not None else (None, None)
    vcos, vsin = vtable if vtable is not None and G else (None, None)
    rows = [t.shape[0] for t in (cos, vcos) if t is not None]
    if not G:
        cache = None
    _cabi.check(_cabi.lib().mv_qkv_rope_store(
        ptr(q), ptr(k), ptr(v), any_.stride(0), ptr(q_weight), ptr(k_weight) if G else None, ptr(temp), ptr(cos), ptr(sin),
        dims, ptr(vcos), ptr(vsin), min(rows) if rows else 1, positions.data_ptr(), ptr(out), ptr(cache),
        slot_mapping.data_ptr() if cache is not None else None, cache.shape[0] * cache.shape[1] if cache is not None else 0,
        tokens, heads, G, VG, dim, vdim, eps, _cabi.layer_dtype_code(any_.dtype), _cabi.stream_ptr()))
    return out


class RotaryWindowAttention(nn.Module):
    """`source`: the earlier layer of this class whose keys and values this one uses, or None."""

    def __init__(self, m, width, eps, load, max_position, source=None):
        super().__init__()
        self.heads, self.kv_heads, self.dim, self.vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        self.scale, self.eps, self.max_position = float(m["scale"]), eps, max_position
        self.base, self.dims = float(m["rot"]["base"]), m["rot"]["dims"]
        self.window = int((m.get("mask") or {}).get("size", UNBOUNDED))
        if self.heads % self.kv_heads or self.window < 1:
            raise ValueError("attention: heads must be a multiple of kv_heads, and the window hold a token")
        if not 0 <= self.dims <= self.dim or self.dims % 2 or self.vdim % 2:
            raise ValueError("attention: rotated sizes must be even, and rot.dims at most dim")
        H, G, d, vd = self.heads, self.kv_heads, self.dim, self.vdim
        order, vorder = pair_order(d, self.dims), pair_order(vd, vd)
        parts = {"q": _reorder(load("q", (H * d, width)), H, order)}
        param = lambda t: nn.Parameter(t, requires_grad=False)
        self.q_norm, self.k_norm = param(_reorder(load("q.norm", (d,)), 1, order)), None
        self.temp = param(load("temp", (H,)))
        self.o_w = param(_reorder(load("o", (width, H * vd)), H, vorder, dim=1))
        self._source = (source,)        # in a tuple: not a module of this one
        self.lends = False              # does a later layer use these keys and values?
        if source is None:
            parts["k"] = _reorder(load("k", (G * d, width)), G, order)
            parts["v"] = _reorder(load("v", (G * vd, width)), G, vorder)
            self.k_norm = param(_reorder(load("k.norm", (d,)), 1, order))
            self.paged_cache = None     # (blocks, block_size, paged_row), assigned by the model runner
        else:
            mine, its = ([getattr(x, n) for n in ("kv_heads", "dim", "vdim", "base", "dims")] for x in (self, source))
            if mine != its or source._source[0] is not None:
                raise ValueError("attention: kv_from must name an earlier layer with keys and values of its own, and the "
                                 "same KV heads, sizes and rotation")
            source.lends = True
        self.stacked = StackedLinear(parts)

    @property
    def paged_row(self):
        return self.kv_heads * (self.dim + self.vdim)

    def _tiles(self, dtype):
        """Does the tensor-core prefill kernel take this layer's sizes?"""
        return dtype == torch.bfloat16 and _cabi.lib().mv_window_prefill_distances(self.dim, self.vdim) >= 1

    def _portion_rows(self, ctx, fresh, rows, tables):
        """The packed [k | v] rows that the portions of this step can see through this layer's window, and their cu_k.  A
        layer that uses this one's finds them here too."""
        if fresh:
            return rows, ctx.portion_cu_q
        owner = self._source[0] or self
        cu_k, first, keys = window_keys(ctx, self.window, owner.paged_cache.device)
        key = ("window_rows", id(owner), self.window)
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
        q, nd, cache = p["q"], ctx.num_decode, owner.paged_cache
        tokens = q.shape[0]
        table = rope_table(self.base, self.dims, self.max_position, h.device) if self.dims else None
        vtable = rope_table(self.base, self.vdim, self.max_position, h.device)
        turn = turn_table(self.base, self.vdim, self.max_position, h.device)
        tiles = tokens > nd and self._tiles(q.dtype)
        fresh = tiles and ctx.portion_fresh
        kv = qkv_rope_store(q, p.get("k"), p.get("v"), self.q_norm, self.k_norm, self.temp, self.eps, ctx.positions, table, self.dims,
                            vtable, self.heads, self.kv_heads, cache, ctx.slot_mapping, packed=fresh and owner is self)
        if fresh and owner.lends:        # the step's own rows, for the layers that share them
            kv = ctx.memo.setdefault(("fresh_rows", id(owner)), kv)
        sizes = (self.kv_heads, self.dim, self.vdim, self.window, self.scale)
        o = torch.empty((tokens, self.heads * self.vdim), dtype=q.dtype, device=q.device)
        if nd:                           # sequences with one token come first
            args = (q[:nd], cache, ctx.block_tables[:nd])
            if window_decode(*args, ctx.positions[:nd], *sizes, out=o[:nd], turn=turn) is None:
                window_attention_rows(*args, None, ctx.positions[:nd], *sizes, out=o[:nd], turn=turn)
        if tokens > nd:
            tables, cu_q, pos = ctx.block_tables[nd:], ctx.portion_cu_q, ctx.positions[nd:]
            if not tiles:
                window_attention_rows(q[nd:], cache, tables, cu_q, pos, *sizes, out=o[nd:], turn=turn)
            else:
                rows, cu_k = self._portion_rows(ctx, fresh, kv[nd:] if fresh else None, tables)
                window_prefill(q[nd:], rows, cu_q, cu_k, *sizes, out=o[nd:], turn=turn, positions=pos)
        return F.linear(o, self.o_w)
