"""Device memory that outlives a step, for modules other than the K/V attention layers.

Two kinds, found on the model's modules by attribute, as the K/V caches are:
  * paged rows: `paged_row` (elements per token) and `paged_cache`, which becomes the layer's
    (blocks, block_size, paged_row) slice of one pool addressed by the block tables;
  * per-sequence state: `slot_state_spec(dtype)` (name -> shape, dtype) and `slot_state`, which becomes a dict of
    (slots, *shape) tensors indexed by the sequence's slot.  Slots are not cleared when they change hands: a kernel
    takes the contents as zero for a sequence that starts.
"""
import math

import torch


def paged_modules(model):
    return [m for m in model.modules() if hasattr(m, "paged_cache")]


def state_modules(model):
    return [m for m in model.modules() if hasattr(m, "slot_state_spec")]


def paged_block_bytes(model, block_size, dtype):
    return sum(m.paged_row for m in paged_modules(model)) * block_size * dtype.itemsize


def slot_bytes(model, dtype):
    return sum(math.prod(shape) * dt.itemsize for m in state_modules(model)
               for shape, dt in m.slot_state_spec(dtype).values())


def bind(model, num_blocks, block_size, num_slots, dtype, device):
    """Allocates and assigns both kinds; returns the list of pools (for whoever must keep or inspect them)."""
    pools = []
    for m in paged_modules(model):
        m.paged_cache = torch.zeros(num_blocks, block_size, m.paged_row, dtype=dtype, device=device)
        pools.append(m.paged_cache)
    for m in state_modules(model):
        m.slot_state = {name: torch.zeros(num_slots, *shape, dtype=dt, device=device)
                        for name, (shape, dt) in m.slot_state_spec(dtype).items()}
        pools.extend(m.slot_state.values())
    return pools
