"""Small Dafotar configurations and helpers shared by the tests."""
import functools

import torch

from oracle import dafotar_oracle as oracle
from tests.sipazen_cases import check, error  # noqa: F401  (re-exported)


def _mem(heads, dim, vdim, cap):
    return "mlstm", {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def _att(heads, kv, dim, vdim, window, dims, base=1e4, scale=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": window}, "rot": {"base": base, "dims": dims},
         "scale": scale if scale is not None else dim ** -0.5}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return "attention", m


def _config(vocab, width, streams, taps, layers, eps=1e-5):
    return {"architecture": "Dafotar", "vocab": vocab, "width": width, "streams": streams, "canon": {"taps": taps},
            "norm": {"eps": eps},
            "layers": [{"type": t, "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None} for (t, m), ff in layers]}


def odd():
    """No size is a multiple of eight, no two sizes agree; every mixer with and without a feed-forward; a layer that uses an
    earlier one's keys through a longer window, and one through a shorter."""
    return _config(131, 90, 3, 4, [
        (_att(6, 2, 19, 14, 11, 12, base=300.0), 46),
        (_mem(3, 14, 10, 5.0), 21),
        (_att(6, 2, 19, 14, 37, 12, base=300.0, scale=0.4, kv_from=0), None),
        (_mem(2, 37, 41, 2.5), None),
        (_att(6, 2, 19, 14, 6, 12, base=300.0, kv_from=0), 35)], eps=1e-4)


def even():
    """Sizes that the tensor-core kernels take, windows shorter and longer than a tile of keys."""
    return _config(320, 192, 4, 2, [
        (_mem(2, 128, 64, 15.0), None),
        (_att(8, 2, 64, 128, 33, 32), 256),
        (_att(8, 2, 64, 128, 150, 32, kv_from=1), None),
        (_mem(4, 32, 96, 9.0), 136),
        (_att(4, 1, 128, 64, 70, 128, base=5e5), 72),
        (_att(4, 1, 128, 64, 70, 128, base=5e5, scale=0.1, kv_from=4), 64)])


def between():
    """Sizes that some of the tensor-core kernels take and others do not; wide heads, many streams, long convolution."""
    return _config(257, 136, 5, 6, [
        (_att(3, 1, 40, 24, 57, 16), 44),
        (_mem(1, 200, 52, 12.0), None),
        (_att(4, 2, 136, 96, 24, 100, scale=0.05), None),
        (_mem(2, 72, 36, 4.0), 30),
        (_att(2, 2, 200, 160, 9, 200, scale=0.05), 19),
        (_mem(1, 130, 20, 7.0), None)])


def ones():
    """Sizes of one: a single stream, head, tap, or key per window."""
    return _config(67, 40, 1, 1, [
        (_att(1, 1, 8, 16, 1, 8), 24),
        (_mem(1, 8, 8, 1.0), 8),
        (_att(16, 1, 16, 8, 5, 2), None),
        (_mem(1, 1, 3, 3.0), None)])


def memory_only():
    return _config(200, 64, 2, 3, [(_mem(2, 32, 32, 10.0), 96), (_mem(2, 32, 32, 10.0), None)])


def attention_only():
    return _config(200, 64, 2, 5, [(_att(4, 2, 32, 32, 20, 32), 64), (_att(4, 4, 32, 48, 1 << 20, 24), None)])


CONFIGS = {f.__name__: f for f in (odd, even, between, ones, memory_only, attention_only)}


@functools.lru_cache(maxsize=None)
def model(name):
    cfg = CONFIGS[name]()
    return cfg, oracle.random_weights(cfg, seed=len(name))


def tokens(name, n, seed=0):
    g = torch.Generator().manual_seed(1000 * seed + n)
    return torch.randint(0, model(name)[0]["vocab"], (n,), generator=g).tolist()


@functools.lru_cache(maxsize=None)
def expected(name, n, seed=0):
    """Oracle logits (n, vocab) in float64."""
    cfg, w = model(name)
    return oracle.forward(cfg, w, tokens(name, n, seed))


def engine(name, dtype, **over):
    from minivllm_b200.engine.llm_engine import LLMEngine
    from minivllm_b200.engine.weights import DictWeights
    cfg, w = model(name)
    c = {**cfg, "dtype": dtype, "weights": DictWeights(w, dtype, "cuda"), "block_size": 16, "num_kv_blocks": 40,
         "max_num_seqs": 4, "max_model_length": 512, "max_num_batched_tokens": 512, "chunked_prefill": True,
         "greedy": True, "keep_logits": True}
    c.update(over)
    return LLMEngine(c)
