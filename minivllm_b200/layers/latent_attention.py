"""Latent attention: low-rank key/value rows in a paged cache, one rotated key part shared by all heads, a learned
sink per head and a sigmoid gate on the heads (csrc/latent_attention.cu).

The cache holds one row [c | rotated key part] per token.  Decoded tokens run in the absorbed form: the key
up-projection is applied to the queries, the value up-projection to the weighted sum of the c's.  Portions of
prompts expand keys and values per head (one product over the packed latent rows, gathered from the cache when a
sequence has tokens behind it) and run tcgen05 prefill attention.  Sizes those kernels do not take, and 32-bit
models, use the absorbed form with a kernel for any sizes.
"""
import torch
import torch.nn as nn
import torch.nn.functional as F

from .. import _cabi
from ..utils.context import get_context
from .attention import _error_word
from .group_norm import gate_mul
from .linear import StackedLinear

_rope_tables = {}


def rope_table(base, dims, max_position, device):
    """(cos, sin), each (max_position, dims / 2) fp32, of position * base^(-2i / dims); angles formed in double."""
    key = (float(base), int(dims), int(max_position), str(device))
    if key not in _rope_tables:
        inv = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64, device=device)
        ang = torch.arange(max_position, dtype=torch.float64, device=device)[:, None] * inv[None, :]
        _rope_tables[key] = (ang.cos().float().contiguous(), ang.sin().float().contiguous())
    return _rope_tables[key]


def latent_prep(q, down, c_weight, positions, cos_t, sin_t, heads, dim, rot_dim, rope_dims, rank, eps, cache=None,
                slot_mapping=None):
    """Rotates q in place, returns the step's latent rows (tokens, rank + rot_dim) and scatters them into `cache`."""
    _cabi.require_cuda(q, down, positions)
    tokens = q.shape[0]
    lat = torch.empty((tokens, rank + rot_dim), dtype=q.dtype, device=q.device)
    slots = cache.shape[0] * cache.shape[1] if cache is not None else 0
    _cabi.check(_cabi.lib().mv_latent_prep(
        q.data_ptr(), q.stride(0), down.data_ptr(), down.stride(0), c_weight.data_ptr(), positions.data_ptr(),
        cos_t.data_ptr(), sin_t.data_ptr(), cos_t.shape[0], lat.data_ptr(),
        cache.data_ptr() if cache is not None else None, slot_mapping.data_ptr() if cache is not None else None, slots,
        tokens, heads, dim, rot_dim, rope_dims, rank, eps, _cabi.layer_dtype_code(q.dtype), _cabi.stream_ptr()))
    return lat


def latent_attention_rows(q_lat, q_rot, cache, block_tables, cu_q, positions, sink, scale, out=None):
    """q_lat (tokens, heads, rank), q_rot (tokens, heads, rot_dim), any token and head strides; cache (blocks,
    block_size, rank + rot_dim).  Returns (tokens, heads, rank), laid out head by head."""
    _cabi.require_cuda(q_lat, q_rot, cache, block_tables, positions)
    tokens, heads, rank = q_lat.shape
    rot = q_rot.shape[2]
    if out is None:
        out = torch.empty((heads, tokens, rank), dtype=q_lat.dtype, device=q_lat.device).transpose(0, 1)
    _cabi.check(_cabi.lib().mv_latent_attention_rows(
        out.data_ptr(), out.stride(0), out.stride(1), q_lat.data_ptr(), q_lat.stride(0), q_lat.stride(1),
        q_rot.data_ptr(), q_rot.stride(0), q_rot.stride(1), cache.data_ptr(), block_tables.data_ptr(),
        block_tables.stride(0), block_tables.shape[1], cache.shape[1], cache.shape[0],
        cu_q.data_ptr() if cu_q is not None else None, block_tables.shape[0], positions.data_ptr(),
        sink.data_ptr() if sink is not None else None, tokens, heads, rank, rot, scale,
        _cabi.layer_dtype_code(q_lat.dtype), _cabi.stream_ptr()))
    return out


def latent_decode(q_lat, q_rot, cache, block_tables, positions, sink, scale, workspace=None):
    """latent_attention_rows for one row per sequence on tensor cores; None when the kernel does not take the sizes."""
    _cabi.require_cuda(q_lat, q_rot, cache, block_tables, positions)
    batch, heads, rank = q_lat.shape
    rot = q_rot.shape[2]
    L = _cabi.lib()
    need = L.mv_latent_decode_workspace_bytes(batch, heads, rank, rot)
    bs = cache.shape[1]
    pieces = [t.data_ptr() // 2 | t.stride(0) | t.stride(1) for t in (q_lat, q_rot) if t.numel()]
    if any(x % 8 for x in pieces):          # rows that are not whole 16-byte pieces
        return None
    if need < 0 or q_lat.dtype != torch.bfloat16 or (bs % 64 and bs not in (8, 16, 32)):
        return None
    if workspace is None:
        workspace = torch.empty(need, dtype=torch.uint8, device=q_lat.device)
    out = torch.empty((heads, batch, rank), dtype=q_lat.dtype, device=q_lat.device).transpose(0, 1)
    _cabi.check(L.mv_latent_decode(
        out.data_ptr(), out.stride(0), out.stride(1), q_lat.data_ptr(), q_lat.stride(0), q_lat.stride(1),
        q_rot.data_ptr(), q_rot.stride(0), q_rot.stride(1), cache.data_ptr(), block_tables.data_ptr(),
        block_tables.stride(0), block_tables.shape[1], cache.shape[1], cache.shape[0], positions.data_ptr(), None,
        sink.data_ptr() if sink is not None else None, batch, heads, rank, rot, scale, workspace.data_ptr(),
        workspace.numel(), _error_word(q_lat.device).data_ptr(), _cabi.stream_ptr()))
    return out


def latent_gather(cache, cu_k, keys, block_tables, first=None):
    """Packed rows (keys, row) of the sequences of cu_k, from position `first` of each (0), out of the paged cache."""
    row = cache.shape[2]
    out = torch.empty((keys, row), dtype=cache.dtype, device=cache.device)
    _cabi.check(_cabi.lib().mv_latent_gather(
        out.data_ptr(), cache.data_ptr(), cu_k.data_ptr(), first.data_ptr() if first is not None else None,
        cu_k.numel() - 1, keys, block_tables.data_ptr(),
        block_tables.stride(0), block_tables.shape[1], cache.shape[1], cache.shape[0], row,
        _cabi.layer_dtype_code(cache.dtype), _cabi.stream_ptr()))
    return out


def latent_prefill(q, kv, k_rot, cu_q, cu_k, heads, dim, rot_dim, vdim, scale, sink):
    """q (tokens, heads * (dim + rot_dim)), kv (keys, heads * (dim + vdim)): all keys, then all values; k_rot (keys,
    rot_dim).  Returns (tokens, heads * vdim)."""
    _cabi.require_cuda(q, kv, k_rot, cu_q, cu_k)
    out = torch.empty((q.shape[0], heads * vdim), dtype=q.dtype, device=q.device)
    v = kv[:, heads * dim:]
    _cabi.check(_cabi.lib().mv_latent_prefill(
        out.data_ptr(), out.stride(0), q.data_ptr(), q.stride(0), kv.data_ptr(), kv.stride(0), k_rot.data_ptr(),
        k_rot.stride(0), v.data_ptr(), v.stride(0), cu_q.data_ptr(), cu_k.data_ptr(), cu_q.numel() - 1, q.shape[0],
        kv.shape[0], heads, dim, rot_dim, vdim, scale, sink.data_ptr() if sink is not None else None,
        _error_word(q.device).data_ptr(), _cabi.stream_ptr()))
    return out


class LatentAttention(nn.Module):
    def __init__(self, m, width, eps, load, extra=None, max_position=4096):
        super().__init__()
        self.heads, self.dim, self.rot_dim, self.vdim, self.rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        self.scale, self.eps = float(m["scale"]), eps
        self.rope_dims = int(m["rot"]["dims"])
        H, d, r, vd, rank = self.heads, self.dim, self.rot_dim, self.vdim, self.rank
        self.stacked = StackedLinear({"q": load("q", (H * (d + r), width)), "dkv": load("dkv", (rank + r, width)),
                                      "g": load("g", (H * vd, width)), **(extra or {})})
        param = lambda t: nn.Parameter(t, requires_grad=False)
        self.c_norm, self.sink = param(load("dkv.norm", (rank,))), param(load("sink", (H,)))
        self.ukv_w = param(torch.cat([load("uk", (H * d, rank)), load("uv", (H * vd, rank))]))
        self.o_w = param(load("o", (width, H * vd)))
        self.cos_t, self.sin_t = rope_table(m["rot"]["base"], self.rope_dims, max_position, self.o_w.device)
        self.paged_cache = None        # (blocks, block_size, rank + rot_dim), assigned by the model runner

    @property
    def paged_row(self):
        return self.rank + self.rot_dim

    @property
    def uk_w(self):
        return self.ukv_w[:self.heads * self.dim].view(self.heads, self.dim, self.rank)

    @property
    def uv_w(self):
        return self.ukv_w[self.heads * self.dim:].view(self.heads, self.vdim, self.rank)

    def _expands(self, dtype):
        """Does the tensor-core prefill kernel take this layer's sizes?"""
        d, r, vd = self.dim, self.rot_dim, self.vdim
        return dtype == torch.bfloat16 and d % 8 == 0 and r % 8 == 0 and vd % 8 == 0 and self.rank % 8 == 0 and \
            -(-d // 64) - (-r // 64) <= 3 and vd <= 128 and self.scale > 0

    def _absorbed(self, q, block_tables, cu_q, positions):
        """q (tokens, heads, dim + rot_dim) -> (tokens, heads, vdim) view of a head-major tensor.  cu_q None: one
        token per row of block_tables."""
        d = self.dim
        q_lat = torch.bmm(q[:, :, :d].transpose(0, 1), self.uk_w).transpose(0, 1)            # (tokens, heads, rank)
        o = None
        if cu_q is None:
            o = latent_decode(q_lat, q[:, :, d:], self.paged_cache, block_tables, positions, self.sink, self.scale)
        if o is None:
            o = latent_attention_rows(q_lat, q[:, :, d:], self.paged_cache, block_tables, cu_q, positions, self.sink,
                                      self.scale)
        return torch.bmm(o.transpose(0, 1), self.uv_w.transpose(1, 2)).transpose(0, 1)

    def _portions(self, ctx, q2, lat, nd):
        """The rows behind the decoded ones -> (tokens, heads * vdim) or (tokens, heads, vdim)."""
        H, d, r, rank = self.heads, self.dim, self.rot_dim, self.rank
        tokens, tables, positions = q2.shape[0], ctx.block_tables[nd:], ctx.positions[nd:]
        q = q2.unflatten(1, (H, d + r))
        if not self._expands(q2.dtype):
            return self._absorbed(q, tables, ctx.portion_cu_q, positions)
        if tokens <= 16 and ctx.portion_keys >= 2048:
            # a few tokens far into a sequence: expanding every key would cost more than decoding them
            at = torch.arange(tokens, device=q.device, dtype=torch.int32)
            seq = torch.bucketize(at, ctx.portion_cu_q[1:], right=True)
            return self._absorbed(q, tables.index_select(0, seq), None, positions)
        if ctx.portion_fresh:
            cu_k = ctx.portion_cu_q
        else:
            cu_k = ctx.portion_cu_k
            lat = latent_gather(self.paged_cache, cu_k, ctx.portion_keys, tables)
        kv = F.linear(lat[:, :rank], self.ukv_w)
        return latent_prefill(q2, kv, lat[:, rank:], ctx.portion_cu_q, cu_k, H, d, r, self.vdim, self.scale, self.sink)

    def forward(self, h):
        """h (tokens, width) -> (mixer output (tokens, width), {extra parts of the stacked projection})."""
        ctx = get_context()
        p = self.stacked(h)
        H, d, r = self.heads, self.dim, self.rot_dim
        q, g, nd = p["q"], p["g"], ctx.num_decode
        lat = latent_prep(q, p["dkv"], self.c_norm, ctx.positions, self.cos_t, self.sin_t, H, d, r, self.rope_dims,
                          self.rank, self.eps, self.paged_cache, ctx.slot_mapping)
        o = torch.empty((h.shape[0], H * self.vdim), dtype=h.dtype, device=h.device)
        if nd:
            y = self._absorbed(q[:nd].unflatten(1, (H, d + r)), ctx.block_tables[:nd], None, ctx.positions[:nd])
            gate_mul(y, g[:nd], out=o[:nd])
        if h.shape[0] > nd:
            gate_mul(self._portions(ctx, q[nd:], lat[nd:], nd), g[nd:], out=o[nd:])
        return F.linear(o, self.o_w), p
