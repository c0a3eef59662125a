"""Grouped-query attention with a sliding window, a learned bias per distance bucket, a sink per head and norms over the
whole query and key projections (csrc/window_attention.cu, csrc/latent_prefill.cu).

The cache holds one row [keys of all KV heads | values of all KV heads] per token.  Decoded tokens take a split kernel
over the rows inside the window.  Portions of prompts take the tcgen05 prefill kernel on packed rows: the step's own, or,
when a sequence has tokens behind it, those that its window reaches, gathered from the cache.  Sizes those kernels do not
take, and 32-bit models, run on a kernel for any sizes.
"""
import math

import torch
import torch.nn as nn
import torch.nn.functional as F

from .. import _cabi
from ..utils.context import get_context
from .attention import _error_word
from .latent_attention import latent_gather
from .linear import StackedLinear

UNBOUNDED = 1 << 30
DEFAULT_BUCKETS = 32     # of seeded weights; a checkpoint's tensors have their own


def distance_buckets(count, buckets, bias_max):
    """Bucket of the distances 0 .. count - 1: the first half of the buckets one each, then geometrically up to
    bias_max."""
    half = buckets // 2
    if half < 1 or (count > half and bias_max <= half):
        raise ValueError(f"distance bias: {buckets} buckets up to {bias_max}")
    far = lambda n: half + math.floor(math.log(n / half) / math.log(bias_max / half) * (buckets - half))
    return [n if n < half else min(buckets - 1, far(n)) for n in range(count)]


def distance_bias(rel, bias_max, window):
    """rel (buckets, heads) -> (heads, distances) fp32; larger distances have the last one's bias."""
    count = min(window, max(math.ceil(bias_max), rel.shape[0] // 2) + 1)
    idx = torch.tensor(distance_buckets(count, rel.shape[0], bias_max), device=rel.device)
    return rel.float()[idx].t().contiguous()


def kv_norm_store(q, k, v, q_weight, k_weight, eps, cache=None, slot_mapping=None, packed=False):
    """Norms q in place; [normed k | v] goes to the cache and, with `packed`, to the returned (tokens, row) tensor."""
    _cabi.require_cuda(q, k, v, q_weight, k_weight, cache)
    if not q.stride(0) == k.stride(0) == v.stride(0):
        raise ValueError("q, k and v must share a row stride")
    tokens, row = q.shape[0], k.shape[1] + v.shape[1]
    out = torch.empty((tokens, row), dtype=q.dtype, device=q.device) if packed else None
    _cabi.check(_cabi.lib().mv_kv_norm_store(
        q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0), q_weight.data_ptr(), k_weight.data_ptr(),
        out.data_ptr() if packed else None, cache.data_ptr() if cache is not None else None,
        slot_mapping.data_ptr() if cache is not None else None, cache.shape[0] * cache.shape[1] if cache is not None else 0,
        tokens, q.shape[1], k.shape[1], v.shape[1], eps, _cabi.layer_dtype_code(q.dtype), _cabi.stream_ptr()))
    return out


def _bias_args(bias):
    return (bias.data_ptr(), bias.stride(0), bias.shape[1]) if bias is not None else (None, 0, 1)


def _turn_args(turn):
    """turn: (vdim / 2, positions, 2) fp32 (cos, sin) of the angles by which results are turned back, or None."""
    return (turn.data_ptr(), turn.shape[1]) if turn is not None else (None, 0)


def window_attention_rows(q, cache, block_tables, cu_q, positions, kv_heads, dim, vdim, window, scale, bias=None, sink=None,
                          out=None, turn=None):
    """q (tokens, heads * dim) -> (tokens, heads * vdim); cu_q None: one token per row of block_tables."""
    _cabi.require_cuda(q, cache, block_tables, positions, bias, sink)
    tokens, heads = q.shape[0], q.shape[1] // dim
    out = torch.empty((tokens, heads * vdim), dtype=q.dtype, device=q.device) if out is None else out
    _cabi.check(_cabi.lib().mv_window_attention_rows(
        out.data_ptr(), q.data_ptr(), q.stride(0), cache.data_ptr(), block_tables.data_ptr(), block_tables.stride(0),
        block_tables.shape[1], cache.shape[1], cache.shape[0], cu_q.data_ptr() if cu_q is not None else None,
        block_tables.shape[0], positions.data_ptr(), *_bias_args(bias), sink.data_ptr() if sink is not None else None, *_turn_args(turn),
        tokens, heads, kv_heads, dim, vdim, window, scale, _cabi.layer_dtype_code(q.dtype), _cabi.stream_ptr()))
    return out


def window_decode(q, cache, block_tables, positions, kv_heads, dim, vdim, window, scale, bias=None, sink=None, out=None,
                  turn=None):
    """window_attention_rows for one row per sequence on tensor cores; None when the kernel does not take the sizes."""
    _cabi.require_cuda(q, cache, block_tables, positions, bias, sink)
    batch, heads = q.shape[0], q.shape[1] // dim
    L = _cabi.lib()
    need = L.mv_window_decode_workspace_bytes(batch, heads, kv_heads, dim, vdim,
                                              max(1, min(window, block_tables.shape[1] * cache.shape[1])))
    if need < 0 or q.dtype != torch.bfloat16:
        return None
    ws = torch.empty(max(need, 4), dtype=torch.uint8, device=q.device)
    out = torch.empty((batch, heads * vdim), dtype=q.dtype, device=q.device) if out is None else out
    _cabi.check(L.mv_window_decode(
        out.data_ptr(), q.data_ptr(), q.stride(0), cache.data_ptr(), block_tables.data_ptr(), block_tables.stride(0),
        block_tables.shape[1], cache.shape[1], cache.shape[0], positions.data_ptr(), *_bias_args(bias),
        sink.data_ptr() if sink is not None else None, *_turn_args(turn), batch, heads, kv_heads, dim, vdim, window, scale, ws.data_ptr(),
        ws.numel(), _cabi.stream_ptr()))
    return out


def window_prefill(q, kv, cu_q, cu_k, kv_heads, dim, vdim, window, scale, bias=None, sink=None, out=None, turn=None,
                   positions=None):
    """q (tokens, heads * dim), kv (keys, kv_heads * (dim + vdim)) packed rows -> (tokens, heads * vdim).  `turn` wants the
    queries' positions."""
    _cabi.require_cuda(q, kv, cu_q, cu_k, bias, sink)
    heads = q.shape[1] // dim
    out = torch.empty((q.shape[0], heads * vdim), dtype=q.dtype, device=q.device) if out is None else out
    v = kv[:, kv_heads * dim:]
    _cabi.check(_cabi.lib().mv_window_prefill(
        out.data_ptr(), out.stride(0), q.data_ptr(), q.stride(0), kv.data_ptr(), kv.stride(0), v.data_ptr(), v.stride(0),
        cu_q.data_ptr(), cu_k.data_ptr(), cu_q.numel() - 1, q.shape[0], kv.shape[0], heads, kv_heads, dim, vdim, window, scale,
        *_bias_args(bias), sink.data_ptr() if sink is not None else None, *_turn_args(turn),
        positions.data_ptr() if turn is not None else None, _error_word(q.device).data_ptr(),
        _cabi.stream_ptr()))
    return out


def window_keys(ctx, window, device):
    """Keys that the portions of a step can see through a window: (cu_k, first position of each sequence, total)."""
    return _portion_keys(ctx, ("window_keys", window), lambda behind: max(0, behind - window + 1), device)


def chunk_keys(ctx, size, device):
    """The same for positions that see their own chunk of the sequence."""
    return _portion_keys(ctx, ("chunk_keys", size), lambda behind: behind // size * size, device)


def _portion_keys(ctx, key, first_of, device):
    if key not in ctx.memo:
        first = [first_of(behind) for behind, _ in ctx.portion_spans]
        cu = [0]
        for f, (behind, n) in zip(first, ctx.portion_spans):
            cu.append(cu[-1] + behind + n - f)
        host = torch.tensor(cu + first, dtype=torch.int32).pin_memory()
        dev = host.to(device, non_blocking=True)
        ctx.memo[key] = (dev[:len(cu)], dev[len(cu):], cu[-1], host)
    return ctx.memo[key][:3]


class WindowAttention(nn.Module):
    """With `stack` False the caller computes the products of `parts` (and adds `biases`) and hands them to `mix`."""

    def __init__(self, m, width, eps, load, stack=True):
        super().__init__()
        self.heads, self.kv_heads, self.dim, self.vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        self.scale, self.eps = float(m["scale"]), eps
        self.window = int((m.get("mask") or {}).get("size", UNBOUNDED))
        if self.heads % self.kv_heads or self.window < 1:
            raise ValueError("window attention: heads must be a multiple of kv_heads, and the window hold a token")
        H, G, d, vd = self.heads, self.kv_heads, self.dim, self.vdim
        sizes = {"q": H * d, "k": G * d, "v": G * vd}
        self.parts = {n: load(n, (r, width)) for n, r in sizes.items()}
        self.biases = {n: load(n + ".b", (r,)) for n, r in sizes.items()}
        self.stacked = None
        if stack:
            self.stacked, self.parts, self.biases = StackedLinear(self.parts, self.biases), None, None
        param = lambda t: nn.Parameter(t, requires_grad=False)
        self.q_norm, self.k_norm = param(load("q.norm", (H * d,))), param(load("k.norm", (G * d,)))
        buckets = load.shape("rel", (DEFAULT_BUCKETS, H))[0]
        self.bias = param(distance_bias(load("rel", (buckets, H)), m["bias_max"], self.window))
        self.sink, self.o_w = param(load("sink", (H,))), param(load("o", (width, H * vd)))
        self.paged_cache = None         # (blocks, block_size, paged_row), assigned by the model runner

    @property
    def paged_row(self):
        return self.kv_heads * (self.dim + self.vdim)

    def _tiles(self, dtype):
        """Does the tensor-core prefill kernel take this layer's sizes?"""
        return dtype == torch.bfloat16 and \
            self.bias.shape[1] <= _cabi.lib().mv_window_prefill_distances(self.dim, self.vdim)

    def forward(self, h):
        return self.mix(self.stacked(h))

    def mix(self, p):
        """p: {name: (tokens, rows)} of the parts' products -> (tokens, width).  The queries are overwritten."""
        ctx = get_context()
        q, nd = p["q"], ctx.num_decode
        tokens, cache = q.shape[0], self.paged_cache
        tiles = tokens > nd and self._tiles(q.dtype)
        fresh = tiles and ctx.portion_fresh
        kv = kv_norm_store(q, p["k"], p["v"], self.q_norm, self.k_norm, self.eps, cache, ctx.slot_mapping, packed=fresh)
        sizes = (self.kv_heads, self.dim, self.vdim, self.window, self.scale, self.bias, self.sink)
        o = torch.empty((tokens, self.heads * self.vdim), dtype=q.dtype, device=q.device)
        if nd:                           # sequences with one token come first
            args = (q[:nd], cache, ctx.block_tables[:nd])
            if window_decode(*args, ctx.positions[:nd], *sizes, out=o[:nd]) is None:
                window_attention_rows(*args, None, ctx.positions[:nd], *sizes, out=o[:nd])
        if tokens > nd:
            tables, cu_q = ctx.block_tables[nd:], ctx.portion_cu_q
            if not tiles:
                window_attention_rows(q[nd:], cache, tables, cu_q, ctx.positions[nd:], *sizes, out=o[nd:])
            elif fresh:
                window_prefill(q[nd:], kv[nd:], cu_q, cu_q, *sizes, out=o[nd:])
            else:
                cu_k, first, keys = window_keys(ctx, self.window, q.device)
                window_prefill(q[nd:], latent_gather(cache, cu_k, keys, tables, first), cu_q, cu_k, *sizes, out=o[nd:])
        return F.linear(o, self.o_w)
