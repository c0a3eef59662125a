"""Latent attention: low-rank key/value rows in a paged cache, one rotated key part shared by all heads, a learned
sink per head and a sigmoid gate on the heads (csrc/latent_attention.cu).

The cache holds one row [c | rotated key part] per token.  Attention runs in the absorbed form: the key
up-projection is applied to the queries, the value up-projection to the weighted sum of the c's.
"""
import torch
import torch.nn as nn
import torch.nn.functional as F

from .. import _cabi
from ..utils.context import get_context
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
        self.uk_w = param(load("uk", (H * d, rank)))                    # (heads * dim, rank)
        self.uv_w = param(load("uv", (H * vd, rank)))                   # (heads * vdim, rank)
        self.o_w = param(load("o", (width, H * vd)))
        self.cos_t, self.sin_t = rope_table(m["rot"]["base"], self.rope_dims, max_position, self.o_w.device)
        self.latent_cache = None        # (blocks, block_size, rank + rot_dim), assigned by the model runner

    @property
    def latent_row(self):
        return self.rank + self.rot_dim

    def _absorbed(self, q, block_tables, cu_q, positions):
        """q (tokens, heads, dim + rot_dim) -> (tokens, heads, vdim) view of a head-major tensor."""
        H, d = self.heads, self.dim
        q_lat = torch.bmm(q[:, :, :d].transpose(0, 1), self.uk_w.view(H, d, self.rank))      # (heads, tokens, rank)
        o = latent_attention_rows(q_lat.transpose(0, 1), q[:, :, d:], self.latent_cache, block_tables, cu_q, positions,
                                  self.sink, self.scale)
        return torch.bmm(o.transpose(0, 1), self.uv_w.view(H, self.vdim, self.rank).transpose(1, 2)).transpose(0, 1)

    def forward(self, h):
        """h (tokens, width) -> (mixer output (tokens, width), {extra parts of the stacked projection})."""
        ctx = get_context()
        p = self.stacked(h)
        H, d, r = self.heads, self.dim, self.rot_dim
        latent_prep(p["q"], p["dkv"], self.c_norm, ctx.positions, self.cos_t, self.sin_t, H, d, r, self.rope_dims,
                    self.rank, self.eps, self.latent_cache, ctx.slot_mapping)
        q = p["q"].unflatten(1, (H, d + r))
        o = self._absorbed(q, ctx.block_tables, ctx.cu_seqlens_q, ctx.positions)
        return F.linear(gate_mul(o, p["g"]), self.o_w), p
